"""A plain, slow implementation of the Pazatar decoder, written from its equations: one function per
mechanism, tensors in, tensors out, no kernels, no cache manager, no code shared with the library.
Everything runs in the dtype of the weights it is given (float64 in the tests), on the CPU, over a
whole sequence at once (position p counts from 0, T tokens, W the width).

    rms(x) = x / sqrt(mean(x^2) + eps);   norm(x, w) = rms(x) * w
    embedding     x_p = E[t_p]
    layer         x += norm(mixer(norm(x, w1)), w1b);  x += norm(ff(norm(x, w2)), w2b)   (ff optional)
    loop          layers [start, stop) run `times` times with the same weights (each pass with keys and
                  states of its own); right before pass t: x += L[t]
    attention     q, k = Wq y, Wk y, v = k;  q <- norm(q, wq) over all heads at once, k likewise; the
                  first R dims of each head rotated, pairs (2i, 2i + 1), YaRN frequencies and magnitude;
                  s_ij = (q_i . k_j) scale;  j visible from i iff j <= i and i // c == j // c;  softmax;  Wo
    parallel      (norm(left(y), wl) + norm(right(y), wr)) / 2
      left        q, k, v = Wq y, Wk y, Wv y, each through a causal convolution per channel;
                  q <- norm(q, wq) per head, k likewise;  rotation in pairs (i, i + R/2) with frequencies
                  slowed by bands of wavelength;  s <- cap tanh((q . k) scale / cap);  the chunk mask;
                  w_ij = exp(s_ij) / (1 + sum_j' exp(s_ij'));  Wo
      right       q = Wq y D^(-1/2), k = Wk y (heads of D), v = Wv y (heads of Dv);
                  decay d = sigmoid(Wa2 (Wa1 y) + b)^(1/tau);  S_p = diag(d_p) S_(p-1) + k_p v_p^T;
                  o = S_p^T q;  Wo (norm(o, wn) per head * silu(Wg y))
    feed-forward  Wd max(Wu y, 0)^2
    output        logits = E norm(x, wf)
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional, Tuple

import torch


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_unit(x, eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ---- rotations ---------------------------------------------------------------------------------
def plain_frequencies(dims: int, base: float) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims: int, base: float, scaling: Optional[Mapping]) -> Tuple[List[float], float]:
    """(frequencies, factor on cosine and sine)."""
    freqs = plain_frequencies(dims, base)
    if scaling is None:
        return freqs, 1.0

    def at(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def banded_frequencies(dims: int, base: float, scaling: Optional[Mapping]) -> List[float]:
    """Short wavelengths as they are, long ones slowed by `factor`, a blend between."""
    freqs = plain_frequencies(dims, base)
    if scaling is None:
        return freqs
    out = []
    for f in freqs:
        wave = 2 * math.pi / f
        if wave < scaling["original"] / scaling["high"]:
            out.append(f)
        elif wave > scaling["original"] / scaling["low"]:
            out.append(f / scaling["factor"])
        else:
            s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
            out.append((1 - s) * f / scaling["factor"] + s * f)
    return out


def angles(T: int, freqs: List[float], dtype) -> torch.Tensor:
    return torch.arange(T, dtype=dtype)[:, None] * torch.tensor(freqs, dtype=dtype)[None, :]


def rotate_half(x: torch.Tensor, freqs: List[float]) -> torch.Tensor:
    """x [T, heads, D]: pairs (i, i + R/2) of the first R = 2 len(freqs) dimensions."""
    half = len(freqs)
    if half == 0:
        return x
    a = angles(x.shape[0], freqs, x.dtype)
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def rotate_interleaved(x: torch.Tensor, freqs: List[float], magnitude: float) -> torch.Tensor:
    """x [T, heads, D]: pairs (2i, 2i + 1) of the first 2 len(freqs) dimensions."""
    n = len(freqs)
    if n == 0:
        return x
    a = angles(x.shape[0], freqs, x.dtype)
    c, s = magnitude * torch.cos(a)[:, None, :], magnitude * torch.sin(a)[:, None, :]
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out = x.clone()
    out[..., 0:2 * n:2] = u * c - v * s
    out[..., 1:2 * n:2] = v * c + u * s
    return out


# ---- attention ---------------------------------------------------------------------------------
def chunk_mask(T: int, size: int) -> torch.Tensor:
    """[T, T] bool: may query i see key j (size 0: causal only)."""
    p = torch.arange(T)
    see = p[:, None] >= p[None, :]
    return see if size == 0 else see & (p[:, None] // size == p[None, :] // size)


def weigh(s: torch.Tensor, see: torch.Tensor, sink: bool) -> torch.Tensor:
    """Softmax over the visible keys, with a key of score 0 and no value in the sum (``sink``)."""
    s = s.masked_fill(~see, float("-inf"))
    top = s.max(dim=-1, keepdim=True).values
    if sink:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    return e / (total + torch.exp(-top) if sink else total)


def grouped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, chunk: int,
                      softcap: float, sink: bool) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    see = chunk_mask(T, chunk)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // per
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        out[:, h] = weigh(s, see, sink) @ v[:, g]
    return out


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, taps]: the last tap on the current token, zeros before the first."""
    T, taps = u.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], dim=0)
    return sum(w[:, j] * padded[j:j + T] for j in range(taps))


def attention_mixer(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    T, H, G, D = y.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = y @ w[p + "q"].T, y @ w[p + "k"].T
    v = k.view(T, G, D)
    q = norm(q, w[p + "q.norm"], eps).view(T, H, D)
    k = norm(k, w[p + "k.norm"], eps).view(T, G, D)
    if m.get("rot"):
        freqs, mag = yarn_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q, k = rotate_interleaved(q, freqs, mag), rotate_interleaved(k, freqs, mag)
    chunk = m["mask"]["size"] if m.get("mask") else 0
    o = grouped_attention(q, k, v, m["scale"], chunk, 0.0, False)
    return o.reshape(T, H * D) @ w[p + "o"].T


def conv_attention(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    T, H, G, D = y.shape[0], m["heads"], m["kv_heads"], m["dim"]
    Dv = m.get("vdim", D)
    q, k, v = (causal_conv(y @ w[p + n].T, w[f"{p}{n}.conv"]) if f"{p}{n}.conv" in w else y @ w[p + n].T
               for n in "qkv")
    q = norm(q.view(T, H, D), w[p + "q.norm"], eps)
    k = norm(k.view(T, G, D), w[p + "k.norm"], eps)
    if m.get("rot"):
        freqs = banded_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q, k = rotate_half(q, freqs), rotate_half(k, freqs)
    chunk = m["mask"]["size"] if m.get("mask") else 0
    o = grouped_attention(q, k, v.view(T, G, Dv), m["scale"], chunk, m.get("softcap", 0.0), True)
    return o.reshape(T, H * Dv) @ w[p + "o"].T


# ---- gated linear attention ----------------------------------------------------------------------
def gla_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor,
                   S: Optional[torch.Tensor] = None):
    """q (scaled), k, decay [T, H, D], v [T, H, Dv] -> (o [T, H, Dv], the state [H, D, Dv] after)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hd,hdj->hj", q[t], S)
    return out, S


def gla_decay(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, tau: float) -> torch.Tensor:
    z = (y @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    log_sigmoid = torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))
    return torch.exp(log_sigmoid / tau)


def gated_linear_attention(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping,
                           eps: float) -> torch.Tensor:
    T, H, D = y.shape[0], m["heads"], m["dim"]
    Dv = m.get("vdim", D)
    q = (y @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (y @ w[p + "k"].T).view(T, H, D)
    v = (y @ w[p + "v"].T).view(T, H, Dv)
    o, _ = gla_recurrence(q, k, v, gla_decay(y, w, p, m["tau"]).view(T, H, D))
    o = norm(o, w[p + "norm"], eps).reshape(T, H * Dv)
    return (o * silu(y @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(left: torch.Tensor, right: torch.Tensor, wl: torch.Tensor, wr: torch.Tensor,
                 eps: float) -> torch.Tensor:
    return 0.5 * (norm(left, wl, eps) + norm(right, wr, eps))


def parallel_mixer(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    return side_by_side(conv_attention(y, w, p + "left.", m["left"], eps),
                        gated_linear_attention(y, w, p + "right.", m["right"], eps),
                        w[p + "left.out"], w[p + "right.out"], eps)


MIXERS = {"attention": attention_mixer, "parallel": parallel_mixer}


# ---- feed-forward and model ----------------------------------------------------------------------
def squared_relu_ff(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str) -> torch.Tensor:
    return torch.clamp(y @ w[p + "up"].T, min=0) ** 2 @ w[p + "down"].T


def run_order(cfg: Mapping) -> List[Tuple[int, Optional[int]]]:
    """(layer, pass that starts here or None) in the order in which the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    order: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg: Mapping, w: Mapping[str, torch.Tensor], tokens, streams: Optional[List] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``streams`` collects x after every layer run."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, start in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if start is not None:
            x = x + w["loop.step"][start]
        y = norm(x, w[p + "norm1"], eps)
        x = x + norm(MIXERS[layer["type"]](y, w, p + "mix.", layer["mixer"], eps), w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = norm(x, w[p + "norm2"], eps)
            x = x + norm(squared_relu_ff(y, w, p + "mlp."), w[p + "norm2b"], eps)
        if streams is not None:
            streams.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["embed"].T


def generate_greedy(cfg: Mapping, w: Mapping[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    ids, out = list(prompt), []
    for _ in range(n_new):
        tok = int(torch.argmax(forward(cfg, w, ids)[-1]))
        out.append(tok)
        ids.append(tok)
    return out


def load_folder(folder: str, dtype: torch.dtype = torch.float64):
    """(config.json as a dict, every tensor of model.safetensors in ``dtype``)."""
    import json
    import os
    from safetensors import safe_open
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    weights: Dict[str, torch.Tensor] = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            t = f.get_tensor(name)
            weights[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, weights
