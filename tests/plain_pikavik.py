"""A plain, slow implementation of the Pikavik decoder, written from its equations: one function per
mechanism, tensors in, tensors out, no kernels, no cache manager, no code shared with the library.
Everything runs in the dtype of the weights it is given (float64 in the tests), on the CPU, over a
whole sequence at once (position p counts from 0, T tokens, W the width).

    rms(x) = x / sqrt(mean(x^2) + eps)
    embedding     x_p = E[t_p]
    layer i       y = rms(x) * (1 + w1);  x += a1 * mixer(y) + a2 * ff(y)   (a1, a2 vectors of W; ff
                  optional)
    wkv           y' = y of the token before (zeros for the first);  m_s = y + (y' - y) * mu_s for
                  s = r, k, v, g, w;  r, k, v = W_s m_s (heads of D);  gate = silu(Wg m_g);
                  decay d = exp(-exp(W2 tanh(W1 m_w) + w0));  per head
                  o_p = S_(p-1)^T r_p + (sum_c r_p[c] u[c] k_p[c]) v_p;  S_p = diag(d_p) S_(p-1) + k_p v_p^T;
                  Wo (rms(o) per head * wn * gate)
    mlstm         q = Wq y D^(-1/2), k = Wk y (heads of D), v = Wv y (heads of Dv);
                  i = c tanh((Wi y + bi) / c);  f = log sigmoid(c tanh((Wf y + bf) / c));
                  m_p = max(f + m_(p-1), i), m from 0;  S_p = e^(f + m_(p-1) - m_p) S_(p-1) + e^(i - m_p) k v^T;
                  n_p likewise with k alone;  o = S^T q / (max(|n . q|, e^(-m)) + 1e-6);
                  Wo (rms(o) per head * wn * sigmoid(Wg y))
    latent        q = Wuq (rms(Wdq y) * wq), per head [D plain | R rotated];  [c' | kr] = Wdkv y,
    attention     c = rms(c') * wc;  per head k = [Wuk c | kr], v = Wuv c;  the first `dims` of the R
                  rotated dimensions turned (pairs (i, i + dims/2), angle p base^(-2i/dims));
                  s_ij = (q_i . k_j) scale, j <= i;  w_ij = e^s_ij / (e^sink + sum_j' e^s_ij');  Wo
    experts       s = sigmoid(Wr y);  groups of neighbours, a group's score the sum of its two largest
                  s;  the `top` largest s within the `keep` best groups;  weights
                  s / (sum of the chosen s + 1e-20) * scale;  expert: Wd (g sigmoid(1.702 g) (u + 1)),
                  g = min(Wg y, L), u = clamp(Wu y, -L, L);  plus sigmoid(Ws y) * shared(y)
    output        logits = H (rms(x) * (1 + wf))
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional

import torch


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def zero_centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_unit(x, eps) * (1.0 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


# ---- rotation ----------------------------------------------------------------------------------
def rotate_half(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, R]: the first ``dims`` of every head rotated, pair (i, i + dims/2) at position p
    by the angle p * base^(-2i/dims)."""
    if dims == 0:
        return x
    half = dims // 2
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    ang = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


# ---- mixers ------------------------------------------------------------------------------------
def shifted(y: torch.Tensor) -> torch.Tensor:
    return torch.cat([torch.zeros_like(y[:1]), y[:-1]], dim=0)


def wkv_recurrence(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor,
                   u: torch.Tensor, S: Optional[torch.Tensor] = None):
    """r, k, decay [T, H, D], v [T, H, Dv], u [H, D] -> (o [T, H, Dv], the state [H, D, Dv] after)."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[2], dtype=r.dtype) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=r.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hd,hdj->hj", r[t], S + u[:, :, None] * kv)
        S = decay[t][:, :, None] * S + kv
    return out, S


def wkv_mixer(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    T = y.shape[0]
    H, D = m["heads"], m["dim"]
    before = shifted(y)
    mix = {s: y + (before - y) * w[f"{p}mu.{s}"] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].T).view(T, H, D) for s in "rkv")
    gate = silu(mix["g"] @ w[p + "g"].T)
    raw = torch.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]
    decay = torch.exp(-torch.exp(raw)).view(T, H, D)
    o, _ = wkv_recurrence(r, k, v, decay, w[p + "u"].view(H, D))
    o = rms_unit(o, eps).reshape(T, H * D)
    return (o * w[p + "norm"] * gate) @ w[p + "o"].T


def mlstm_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor,
                     f: torch.Tensor, state=None):
    """q (scaled), k [T, H, D], v [T, H, Dv], log gates i, f [T, H] -> (o [T, H, Dv], (S, n, m))."""
    T, H, D = q.shape
    if state is None:
        S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
        n = torch.zeros(H, D, dtype=q.dtype)
        mx = torch.zeros(H, dtype=q.dtype)
    else:
        S, n, mx = (x.clone() for x in state)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        new = torch.maximum(f[t] + mx, i[t])
        keep, add = torch.exp(f[t] + mx - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        mx = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-mx)) + 1e-6
        out[t] = torch.einsum("hd,hdj->hj", q[t], S) / den[:, None]
    return out, (S, n, mx)


def mlstm_mixer(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    T = y.shape[0]
    H, D = m["heads"], m["dim"]
    Dv, cap = m.get("vdim", D), m["gate_cap"]
    q = (y @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k = (y @ w[p + "k"].T).view(T, H, D)
    v = (y @ w[p + "v"].T).view(T, H, Dv)
    i = cap * torch.tanh((y @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((y @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o, _ = mlstm_recurrence(q, k, v, i, f)
    o = rms_unit(o, eps).reshape(T, H * Dv)
    return (o * w[p + "norm"] * torch.sigmoid(y @ w[p + "g"].T)) @ w[p + "o"].T


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float,
                   sink: torch.Tensor) -> torch.Tensor:
    """q, k [T, H, D], v [T, H, Dv] of one sequence, causal -> [T, H, Dv]."""
    T, H = q.shape[0], q.shape[1]
    see = torch.arange(T)[:, None] >= torch.arange(T)[None, :]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = ((q[:, h] @ k[:, h].T) * scale).masked_fill(~see, float("-inf"))
        s = torch.cat([s, sink[h].expand(T, 1)], dim=1)
        out[:, h] = torch.softmax(s, dim=-1)[:, :T] @ v[:, h]
    return out


def latent_attention_mixer(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, m: Mapping,
                           eps: float) -> torch.Tensor:
    T = y.shape[0]
    H, D, R, Dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_unit(y @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, D + R)
    ckr = y @ w[p + "dkv"].T
    c = rms_unit(ckr[:, :rank], eps) * w[p + "dkv.norm"]
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    kr = rotate_half(ckr[:, None, rank:], dims, base).expand(T, H, R)
    q = torch.cat([q[..., :D], rotate_half(q[..., D:], dims, base)], dim=-1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, D), kr], dim=-1)
    v = (c @ w[p + "uv"].T).view(T, H, Dv)
    o = sink_attention(q, k, v, m["scale"], w[p + "sink"])
    return o.reshape(T, H * Dv) @ w[p + "o"].T


MIXERS = {"wkv": wkv_mixer, "mlstm": mlstm_mixer, "latent_attention": latent_attention_mixer}


# ---- feed-forward ------------------------------------------------------------------------------
def clamped_expert(x: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(x @ w[p + "gate"].T, max=limit)
    u = torch.clamp(x @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(z: torch.Tensor, top: int, groups: int, keep: int, scale: float):
    """From router outputs z [T, experts]: (chosen [T, top], weights [T, top], margin [T]).  The margin
    says how far the closest of the two choices (groups, experts) was: the relative change of a token's
    z that it takes, to first order, to turn it."""
    s = torch.sigmoid(z)
    T, E = s.shape
    # what s moves by when every z moves by its typical size
    moves = s * (1.0 - s) * (z * z).mean(dim=-1, keepdim=True).sqrt().clamp(min=0.1)
    margin = torch.full((T,), float("inf"), dtype=s.dtype)
    allowed = torch.ones(T, E, dtype=torch.bool)
    if groups > 1 and keep < groups:
        size = E // groups
        two = torch.topk(s.view(T, groups, size), min(2, size), dim=-1)
        best = two.values.sum(-1)
        give = torch.gather(moves.view(T, groups, size), 2, two.indices).sum(-1)
        order = torch.argsort(best, dim=-1, descending=True, stable=True)
        ranked, give = torch.gather(best, 1, order), torch.gather(give, 1, order)
        margin = (ranked[:, keep - 1] - ranked[:, keep]) / (give[:, keep - 1] + give[:, keep]).clamp(min=1e-30)
        ok = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, order[:, :keep], True)
        allowed = ok.repeat_interleave(size, dim=1)
    masked = s.masked_fill(~allowed, float("-inf"))
    order = torch.argsort(masked, dim=-1, descending=True, stable=True)
    ranked, give = torch.gather(masked, 1, order), torch.gather(moves, 1, order)
    if top < int(allowed[0].sum()):
        margin = torch.minimum(margin, (ranked[:, top - 1] - ranked[:, top])
                               / (give[:, top - 1] + give[:, top]).clamp(min=1e-30))
    chosen = order[:, :top]
    picked = torch.gather(s, 1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20) * scale, margin


def routed_ff(y: torch.Tensor, w: Mapping[str, torch.Tensor], p: str, mlp: Mapping,
              margins: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    chosen, weight, margin = choose(y @ w[p + "router"].T, r["top"], g["count"], g["keep"], r.get("scale", 1.0))
    if margins is not None:
        margins.append(margin)
    out = torch.zeros_like(y)
    for e in range(r["experts"]):
        t, k = (chosen == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += weight[t, k][:, None] * clamped_expert(y[t], w, f"{p}e{e}.", mlp["expert"]["limit"])
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(y @ w[p + "shared.sg"].T) * clamped_expert(y, w, p + "shared.",
                                                                             mlp["shared"]["limit"])
    return out


# ---- the model ---------------------------------------------------------------------------------
def forward(cfg: Mapping, w: Mapping[str, torch.Tensor], tokens, streams: Optional[List] = None,
            margins: Optional[List] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``streams`` collects x after every layer, ``margins`` the
    routers' margins (a small one means a router's choice is a close call)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = zero_centred_norm(x, w[p + "norm1"], eps)
        add = MIXERS[layer["type"]](y, w, p + "mix.", layer["mixer"], eps) * w[p + "ls1"]
        if layer.get("mlp") is not None:
            add = add + routed_ff(y, w, p + "mlp.", layer["mlp"], margins) * w[p + "ls2"]
        x = x + add
        if streams is not None:
            streams.append(x.clone())
    return zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T


def forward_marked(cfg: Mapping, w: Mapping[str, torch.Tensor], tokens, least_margin: float):
    """(logits, sure): ``sure[t]`` is False where some router's choice at token t is a close call."""
    margins: List[torch.Tensor] = []
    logits = forward(cfg, w, tokens, None, margins)
    sure = torch.ones(logits.shape[0], dtype=torch.bool)
    for m in margins:
        sure &= m >= least_margin
    return logits, sure


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
