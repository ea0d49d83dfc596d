"""Grouped-query attention whose queries and keys are normed as a whole and whose scores are
soft-capped, as a mixer.

    q, k, v = Wq u + bq, Wk u + bk, Wv u + bv          (``bias``; v of its own width ``value_dim``;
        ``values`` "keys": there is no Wv, v is k as it is before norm and rotation)
    q, k, v <- a causal convolution per channel, ``conv`` taps, the last on the current token, zeros
        before the start, no bias, no activation                               (``conv`` > 0)
    q <- q / sqrt(mean(q^2) + eps) * wq over ALL heads of q at once, k likewise    (``qk_norm``;
        with ``norm_scope`` "head": over each head by itself, one weight of the head's width)
    a rotation of the first ``rotary_dim`` dimensions of every head of q and k      (``position``)
    s_ij = (q_i . k_j) * scale;  s_ij <- softcap * tanh(s_ij / softcap)              (``softcap`` > 0)
    j visible from i iff j <= i and (i - j < window or j < keep_first)   (``window`` > 0; with
        ``keep_first`` the first tokens of a sequence stay visible, at their true positions)
        and floor(i / chunk) == floor(j / chunk), counted from position 0          (``chunk`` > 0)
    o = concat_h(softmax_j(s_ij) v_j), with one added to the softmax's sum         (``sink``)
    o <- o * sigmoid(Wg u)                                                         (``gate``)
    out = Wo (o * out_scale)

Every size, constant and switch is a parameter, and so are the tensors' names (behind ``prefix +
tensor_prefix``: ``q``, ``k``, ``v``, ``o``, biases ``<name>.b``, norm weights ``q.norm``,
``k.norm``, the convolutions ``<name>.conv`` [channels, taps], the gate ``g``).  One packed product
gives q|k|v(|g) in float32 (bias added by the product); one kernel norms, rotates and writes the step's keys and values and the cache's pages; the attention is
``parts.sink_attention.scored_attention``; Wo adds into the residual stream.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..config.base import PartSpec
from ..kernels import api as K
from ..weights.spec import MATRIX, VECTOR, Init, TensorSpec
from .base import CacheRequest, CallBinding, Mixer, StateRequest, StepContext
from .linear import Linear
from .sink_attention import ScoreSpec, project_out, scored_attention


CONV_STATE = "attention.conv"


class QkNormAttention(Mixer):
    capturable = True      # launches kernels only; safe inside a CUDA graph capture
    stores_fresh_output = True     # its last product goes through ``project_out``

    def libraries(self, dtype: torch.dtype) -> List[str]:
        libs = ["ops", "mixer_prep", "attention_sink"]
        libs.append("gemm_tc" if dtype == torch.bfloat16 else "gemm_simt")
        if self.conv:
            libs.append("recurrent")
        if K.sink_attention_tc_supported(dtype, self.head_dim, self.value_dim):
            libs.append("attention_prefill_tc")
        return libs

    def __init__(self, hidden_size: int, n_heads: int, n_kv_heads: int, head_dim: int,
                 value_dim: int, scale: float, norm_eps: float, softcap: float = 0.0,
                 window: int = 0, qk_norm: bool = True, bias: bool = True,
                 position: Optional[PartSpec] = None, tensor_prefix: str = "mix.",
                 init_std: float = 0.02, norm_scope: str = "all", keep_first: int = 0,
                 gate: bool = False, out_scale: float = 1.0, chunk: int = 0, sink: bool = False,
                 values: str = "own", conv: int = 0):
        from ..registry import build_part
        if n_kv_heads < 1 or n_heads % n_kv_heads != 0:
            raise ValueError(f"{n_heads} heads do not divide into {n_kv_heads} key/value heads")
        for what, d in (("key", head_dim), ("value", value_dim)):
            if not 1 <= d <= 640:
                raise ValueError(f"{what} size {d} is not supported: the kernels take 1 to 640")
        if min(softcap, window, keep_first, chunk) < 0:
            raise ValueError("softcap, window, chunk and keep_first must not be negative")
        if values not in ("own", "keys") or (values == "keys" and value_dim != head_dim):
            raise ValueError("values are \"own\" or \"keys\" (then of the keys' size)")
        if not 0 <= conv <= 8:
            raise ValueError(f"the convolution's kernel takes up to 8 taps, got {conv}")
        if norm_scope not in ("all", "head"):
            raise ValueError(f"norm_scope is \"all\" or \"head\", got {norm_scope!r}")
        self.hidden_size = int(hidden_size)
        self.n_heads = int(n_heads)
        self.n_kv_heads = int(n_kv_heads)
        self.head_dim = int(head_dim)
        self.value_dim = int(value_dim)
        self.scale = float(scale)
        self.norm_eps = float(norm_eps)
        self.softcap = float(softcap)
        self.window = int(window)
        self.qk_norm = bool(qk_norm)
        self.bias = bool(bias)
        self.norm_scope = norm_scope
        self.keep_first = int(keep_first) if window > 0 else 0
        self.gate = bool(gate)
        self.chunk = int(chunk)
        self.sink = bool(sink)
        self.values = values
        self.conv = int(conv)
        self.conv_w: Optional[torch.Tensor] = None         # [channels, taps]: q | k | v
        self.conv_wt: Optional[torch.Tensor] = None        # the same as [taps, channels]
        self.names = "qk" if values == "keys" else "qkv"   # the projections' tensors
        self.out_scale = float(out_scale)
        self.tensor_prefix = tensor_prefix
        self.init_std = float(init_std)
        self.position = build_part("position", position) if position is not None else None
        self.qkv: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.q_norm: Optional[torch.Tensor] = None
        self.k_norm: Optional[torch.Tensor] = None

    def _widths(self):
        """Columns of q, k and v in the packed projection (v: none if the values are the keys)."""
        return (self.n_heads * self.head_dim, self.n_kv_heads * self.head_dim,
                self.n_kv_heads * self.value_dim if self.values == "own" else 0)

    # ---- weights ----------------------------------------------------------------------
    def tensor_specs(self, prefix: str) -> List[TensorSpec]:
        p = f"{prefix}{self.tensor_prefix}"
        nq, nk, nv = self._widths()
        init = Init(0.0, self.init_std)
        widths = dict(zip("qkv", (nq, nk, nv)))
        specs = [TensorSpec(f"{p}{n}", (widths[n], self.hidden_size), MATRIX, init) for n in self.names]
        specs.append(TensorSpec(f"{p}o", (self.hidden_size, self.n_heads * self.value_dim), MATRIX, init))
        if self.bias:
            specs += [TensorSpec(f"{p}{n}.b", (widths[n],), VECTOR, init) for n in self.names]
        if self.conv:
            specs += [TensorSpec(f"{p}{n}.conv", (widths[n], self.conv), VECTOR, Init(0.0, 0.3)) for n in self.names]
        if self.qk_norm:
            per_head = self.norm_scope == "head"
            specs += [TensorSpec(f"{p}q.norm", (self.head_dim if per_head else nq,), VECTOR, Init(1.0, 0.0)),
                      TensorSpec(f"{p}k.norm", (self.head_dim if per_head else nk,), VECTOR, Init(1.0, 0.0))]
        if self.gate:
            specs.append(TensorSpec(f"{p}g", (self.n_heads * self.value_dim, self.hidden_size), MATRIX, init))
        return specs

    def load(self, prefix: str, weights: Dict[str, torch.Tensor]) -> None:
        p = f"{prefix}{self.tensor_prefix}"
        parts = [weights[f"{p}{n}"] for n in self.names + ("g" if self.gate else "")]
        if len({t.dtype for t in parts}) != 1:
            parts = [t.to(torch.float32) for t in parts]
        b = None
        if self.bias:
            biases = [weights[f"{p}{n}.b"] for n in self.names]
            if self.gate:          # the gate has no bias of its own
                biases.append(torch.zeros(self.n_heads * self.value_dim, dtype=biases[0].dtype,
                                          device=biases[0].device))
            b = torch.cat(biases).contiguous()
        self.qkv = Linear(torch.cat(parts, dim=0).contiguous(), b)
        self.out = Linear(weights[f"{p}o"])
        if self.conv:
            self.conv_w = torch.cat([weights[f"{p}{n}.conv"] for n in self.names], dim=0).contiguous()
            self.conv_wt = self.conv_w.t().contiguous()
        if self.qk_norm:
            self.q_norm, self.k_norm = weights[f"{p}q.norm"], weights[f"{p}k.norm"]
        # the projection of q|k|v can apply a norm's 1/rms itself (bfloat16 on tensor cores)
        self.accepts_row_scale = self.qkv.takes_row_scale()

    def export(self, prefix: str) -> Dict[str, torch.Tensor]:
        p = f"{prefix}{self.tensor_prefix}"
        nq, nk, nv = self._widths()
        out = {f"{p}o": self.out.weight}
        for name, lo, hi in (("q", 0, nq), ("k", nq, nq + nk), ("v", nq + nk, nq + nk + nv))[:len(self.names)]:
            out[f"{p}{name}"] = self.qkv.weight[lo:hi]
            if self.conv:
                out[f"{p}{name}.conv"] = self.conv_w[lo:hi]
            if self.bias:
                out[f"{p}{name}.b"] = self.qkv.bias[lo:hi]
        if self.qk_norm:
            out[f"{p}q.norm"], out[f"{p}k.norm"] = self.q_norm, self.k_norm
        if self.gate:
            out[f"{p}g"] = self.qkv.weight[nq + nk + nv:]
        return out

    # ---- what it keeps per sequence -----------------------------------------------------
    def cache_request(self) -> Optional[CacheRequest]:
        # kept first tokens stay visible for ever: such a layer keeps every position, not a ring
        return CacheRequest(self.n_kv_heads, self.head_dim, self.scores().reach(),
                            self.value_dim if self.value_dim != self.head_dim else 0)

    def state_request(self) -> Sequence[StateRequest]:
        # the projections' outputs of a sequence's last taps - 1 tokens
        if self.conv < 2:
            return ()
        return (StateRequest(CONV_STATE, (sum(self._widths()), self.conv - 1), torch.float32),)

    def scores(self) -> ScoreSpec:
        return ScoreSpec(n_heads=self.n_heads, n_kv_heads=self.n_kv_heads, head_dim=self.head_dim,
                         value_dim=self.value_dim, scale=self.scale, window=self.window,
                         softcap=self.softcap, keep_first=self.keep_first, chunk=self.chunk, sink=self.sink)

    # ---- the step -----------------------------------------------------------------------
    def forward_add(self, x: torch.Tensor, ctx: StepContext, binding: CallBinding,
                    residual: torch.Tensor) -> None:
        qkv = self.qkv.forward(x, torch.float32, row_scale=ctx.input_scale)
        project_out(self.out, self.run(qkv, 0, ctx, binding), ctx, residual)

    @property
    def in_proj(self) -> Linear:
        return self.qkv

    def run(self, qkv: torch.Tensor, off: int, ctx: StepContext, binding: CallBinding) -> torch.Tensor:
        """The operand of the output product, from the packed projection's columns in ``qkv`` (float32
        rows, this mixer's columns from ``off`` on)."""
        n = qkv.shape[0]
        nh, nk, hd, vd = self.n_heads, self.n_kv_heads, self.head_dim, self.value_dim
        nq_w, nk_w, nv_w = self._widths()
        dev, act = qkv.device, ctx.act_dtype
        cache = binding.cache
        if cache is None:
            raise K.KernelError("the attention mixer was given no cache entry")
        if cache.k.dtype != act:
            raise K.KernelError("the cache and the activations must share one dtype")
        heads, q_off = qkv, off      # the rows and the column that q, k and v are taken from
        conv = None
        if self.conv:
            channels = nq_w + nk_w + nv_w
            state = binding.state.get(CONV_STATE)
            if state is None:        # one tap: nothing is kept
                state = torch.empty((1, channels, 0), dtype=torch.float32, device=dev)
            conv = (self.conv_w, self.conv_wt, state, ctx.cu_seqlens, ctx.slots, ctx.n_rows, ctx.single_token)
            if self.norm_scope == "all" or self.values == "keys":
                # the kernel that prepares head by head convolves as it reads; here it comes first
                heads = torch.empty((n, channels), dtype=torch.float32, device=dev)
                q_off = 0
                K.conv_silu(qkv, off, channels, self.conv_w, None, state, ctx.token_row, ctx.cu_seqlens,
                            ctx.slots, heads, ctx.n_rows, single=ctx.single_token, activation="none")
                conv = None
        k_off = q_off + nq_w
        v_off = k_off if self.values == "keys" else k_off + nk_w
        inv_freq, rot_dims, style, magnitude = None, 0, 0, 1.0
        if self.position is not None and getattr(self.position, "rotary_dim", 0) > 0:
            inv_freq, rot_dims, style = self.position.tables(dev)
            magnitude = self.position.magnitude()
        q = torch.empty((n, nh, hd), dtype=act, device=dev)
        write = binding.writes_cache
        own_kv = ctx.from_start
        k_step = v_step = None
        if own_kv and write:
            k_step = torch.empty((n, nk, hd), dtype=act, device=dev)
            v_step = torch.empty((n, nk, vd), dtype=act, device=dev)
            if binding.has_readers:
                ctx.extras[("step_kv", binding.entry)] = (k_step, v_step)
        elif own_kv:
            k_step, v_step = ctx.extras[("step_kv", binding.entry)]
        if self.norm_scope == "head":
            K.head_prepare(heads, ctx.positions, ctx.token_row, ctx.seq_end, q,
                           k_step if write else None, v_step if write else None,
                           cache.k if write else None, cache.v if write else None,
                           cache.page_table if write else None, cache.table_stride, cache.ring,
                           q_off=q_off, n_heads=nh, q_width=hd, k_off=k_off, n_kv=nk, k_width=hd,
                           v_off=v_off, v_width=vd, q_norm=self.q_norm, k_norm=self.k_norm,
                           eps=self.norm_eps, inv_freq=inv_freq, rot_dims=rot_dims, rot_style=style,
                           rot_magnitude=magnitude, q_mul=1.0, k_mul=1.0, status=ctx.status, conv=conv)
        else:
            K.qk_prepare(heads, ctx.positions, ctx.token_row, ctx.seq_end, q,
                         k_step if write else None, v_step if write else None,
                         cache.k if write else None, cache.v if write else None,
                         cache.page_table if write else None, cache.table_stride, cache.ring,
                         q_off=q_off, n_heads=nh, q_width=hd, k_off=k_off, n_kv=nk, k_width=hd,
                         v_off=v_off, v_width=vd, v_from_k=False,
                         q_norm=self.q_norm, k_norm=self.k_norm, eps=self.norm_eps,
                         inv_freq=inv_freq, rot_dims=rot_dims, rot_style=style,
                         rot_magnitude=magnitude, q_rot_off=0, k_rot_off=0, status=ctx.status)
        o = torch.empty((n, nh * vd), dtype=act, device=dev)
        scored_attention(self.scores(), q, k_step, v_step, cache, ctx, o)
        if self.gate:
            K.gate_mul(o, qkv, off + nq_w + nk_w + nv_w, self.out_scale)
        elif self.out_scale != 1.0:
            raise K.KernelError("an output scale rides on the output gate; this attention has none")
        return o
