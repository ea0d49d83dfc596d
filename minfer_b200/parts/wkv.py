"""WKV, the recurrence of the RWKV models, as a mixer: linear attention with a data-dependent decay per key channel, a
bonus for the current token, and inputs that are each mixed with the token before.

    u' = the u of the sequence's token before (zeros for the first)
    m_s = u + (u' - u) * mu_s,   s = r, k, v, g, w
    r, k, v = W_s m_s  (heads of ``head_dim``),   gate = silu(Wg m_g)
    decay d = exp(-exp(W2 tanh(W1 m_w) + w0))      per head and key channel, W1 and W2 through ``rank``
    per head:  o_t = S_(t-1)^T r_t + (sum_c r_t[c] bonus[c] k_t[c]) v_t
               S_t = diag(d_t) S_(t-1) + k_t v_t^T
    o <- o / sqrt(mean(o^2) + eps) per head, times a weight over all heads, times the gate;  Wo

State per sequence (float32, zeroed when a slot is handed out): S of every head and the last u.  A
step may bring any number of tokens per sequence; the recurrence walks them in order, so the result
does not depend on how a sequence is cut.  One kernel forms the five mixes; r, k, v and g come from
one grouped product (float32 out); decays, recurrence, norm and gate are float32 in both engines.
Tensor names behind ``prefix + tensor_prefix``: ``mu.{r,k,v,g,w}``, ``r``, ``k``, ``v``, ``g``, ``w1``,
``w2``, ``w0``, ``u``, ``norm``, ``o``.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..kernels import api as K
from ..weights.spec import MATRIX, VECTOR, Init, TensorSpec
from .base import CallBinding, Mixer, StateRequest, StepContext
from .linear import GroupedLinear, Linear
from .sink_attention import project_out

WKV_STATE = "wkv.state"
WKV_PREVIOUS = "wkv.previous"
MIXES = "rkvgw"


class Wkv(Mixer):
    capturable = True      # launches kernels only; safe inside a CUDA graph capture
    stores_fresh_output = True     # its last product goes through ``project_out``

    def libraries(self, dtype: torch.dtype) -> List[str]:
        return ["ops", "outer_scan", "retention", "gemm_tc" if dtype == torch.bfloat16 else "gemm_simt"]

    def __init__(self, hidden_size: int, n_heads: int, head_dim: int, rank: int, norm_eps: float,
                 tensor_prefix: str = "mix.", init_std: float = 0.02):
        if min(n_heads, head_dim, rank) < 1:
            raise ValueError("wkv: every size must be at least 1")
        if head_dim > 256 or rank > 768:
            raise ValueError("wkv: the kernels take keys up to 256 wide and a decay rank up to 768")
        self.hidden_size = int(hidden_size)
        self.n_heads, self.head_dim, self.rank = int(n_heads), int(head_dim), int(rank)
        self.norm_eps = float(norm_eps)
        self.tensor_prefix = tensor_prefix
        self.init_std = float(init_std)
        self.rkvg: Optional[GroupedLinear] = None
        self.decay_in: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.mu: Optional[torch.Tensor] = None            # [5, width]: r, k, v, g, w
        self.w2: Optional[torch.Tensor] = None            # as the checkpoint holds it
        self.w2t: Optional[torch.Tensor] = None           # float32 [rank, heads * head_dim]
        self.w: Dict[str, torch.Tensor] = {}

    # ---- weights ----------------------------------------------------------------------
    def tensor_specs(self, prefix: str) -> List[TensorSpec]:
        p = f"{prefix}{self.tensor_prefix}"
        n, w = self.n_heads * self.head_dim, self.hidden_size
        init = Init(0.0, self.init_std)
        specs = [TensorSpec(f"{p}mu.{s}", (w,), VECTOR, Init(0.5, 0.2)) for s in MIXES]
        specs += [TensorSpec(f"{p}{s}", (n, w), MATRIX, init) for s in "rkvg"]
        # the decay's second matrix takes part in a 32-bit product: held in float32
        specs += [TensorSpec(f"{p}w1", (self.rank, w), MATRIX, init),
                  TensorSpec(f"{p}w2", (n, self.rank), VECTOR, Init(0.0, 0.1)),
                  TensorSpec(f"{p}w0", (n,), VECTOR, Init(-2.0, 1.0)),
                  TensorSpec(f"{p}u", (self.n_heads, self.head_dim), VECTOR, Init(0.0, 0.5)),
                  TensorSpec(f"{p}norm", (n,), VECTOR, Init(1.0, 0.0)),
                  TensorSpec(f"{p}o", (w, n), MATRIX, init)]
        return specs

    def load(self, prefix: str, weights: Dict[str, torch.Tensor]) -> None:
        p = f"{prefix}{self.tensor_prefix}"
        self.mu = torch.stack([weights[f"{p}mu.{s}"] for s in MIXES]).contiguous()
        self.rkvg = GroupedLinear([weights[f"{p}{s}"] for s in "rkvg"])
        self.decay_in = Linear(weights[f"{p}w1"])
        self.w2 = weights[f"{p}w2"]
        self.w2t = self.w2.to(torch.float32).t().contiguous()
        self.w = {n: weights[f"{p}{n}"] for n in ("w0", "u", "norm")}
        self.out = Linear(weights[f"{p}o"])

    def export(self, prefix: str) -> Dict[str, torch.Tensor]:
        p = f"{prefix}{self.tensor_prefix}"
        out = {f"{p}mu.{s}": self.mu[i] for i, s in enumerate(MIXES)}
        out.update({f"{p}{s}": self.rkvg.weight[i] for i, s in enumerate("rkvg")})
        out.update({f"{p}w1": self.decay_in.weight, f"{p}w2": self.w2, f"{p}o": self.out.weight})
        out.update({f"{p}{n}": t for n, t in self.w.items()})
        return out

    # ---- what it keeps per sequence -----------------------------------------------------
    def state_request(self) -> Sequence[StateRequest]:
        return (StateRequest(WKV_STATE, (self.n_heads, self.head_dim, self.head_dim), torch.float32),
                StateRequest(WKV_PREVIOUS, (self.hidden_size,), torch.float32))

    # ---- the step -----------------------------------------------------------------------
    def forward_add(self, x: torch.Tensor, ctx: StepContext, binding: CallBinding,
                    residual: torch.Tensor) -> None:
        n, dev = x.shape[0], x.device
        width = self.n_heads * self.head_dim
        mixes = torch.empty((len(MIXES), n, self.hidden_size), dtype=x.dtype, device=dev)
        K.shift_mix(x, self.mu, ctx.token_row, ctx.cu_seqlens, ctx.slots, binding.state[WKV_PREVIOUS],
                    mixes, ctx.n_rows, ctx.single_token)
        rkvg = self.rkvg.forward(mixes[:4])                        # float32 [4, tokens, width]
        t1 = self.decay_in.forward(mixes[4], torch.float32)
        decay = torch.empty((n, width), dtype=torch.float32, device=dev)
        K.wkv_decay(t1, self.w2t, self.w["w0"], decay)
        o = torch.empty((n, width), dtype=torch.float32, device=dev)
        K.wkv_scan(rkvg[0], rkvg[1], rkvg[2], decay, self.w["u"], binding.state[WKV_STATE],
                   ctx.cu_seqlens, ctx.slots, o, ctx.n_rows, ctx.max_row_tokens)
        gated = torch.empty((n, width), dtype=ctx.act_dtype, device=dev)
        K.unit_norm_gate(o, rkvg[3], 0, gated, self.n_heads, self.norm_eps, "silu",
                         weight=self.w["norm"])
        project_out(self.out, gated, ctx, residual)
