"""Gated linear attention as a mixer: a matrix state per head with a data-dependent decay per key channel.

    q = Wq u * head_dim^(-1/2),  k = Wk u  (heads of ``head_dim``),  v = Wv u  (heads of ``value_dim``)
    decay d = sigmoid(Wa2 (Wa1 u) + b)^(1 / tau)   per head and key channel, Wa1 and Wa2 through ``rank``
    per head:  S_t = diag(d_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
    o <- o / sqrt(mean(o^2) + eps) per head, times a weight [value_dim] shared by the heads, times
    silu(Wg u);  out = Wo o

State per sequence (float32, zeroed when a slot is handed out): S of every head.  A step may bring any
number of tokens per sequence; the recurrence walks them in order, so the result does not depend on
how a sequence is cut.  One packed product gives q | k | v | g | a1 in float32; decays (the second
product of their pair included), recurrence, norm and gate are float32 in both engines.  Tensor names
behind ``prefix + tensor_prefix``: ``q``, ``k``, ``v``, ``g``, ``a1``, ``a2``, ``a2.b``, ``norm``, ``o``.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..kernels import api as K
from ..weights.spec import MATRIX, VECTOR, Init, TensorSpec
from .base import CallBinding, Mixer, StateRequest, StepContext
from .linear import Linear
from .sink_attention import project_out

GLA_STATE = "gla.state"


class GatedLinearAttention(Mixer):
    capturable = True      # launches kernels only; safe inside a CUDA graph capture
    stores_fresh_output = True     # its last product goes through ``project_out``

    def libraries(self, dtype: torch.dtype) -> List[str]:
        return ["ops", "outer_scan", "retention", "gemm_tc" if dtype == torch.bfloat16 else "gemm_simt"]

    def __init__(self, hidden_size: int, n_heads: int, head_dim: int, value_dim: int, rank: int, tau: float,
                 norm_eps: float, tensor_prefix: str = "mix.", init_std: float = 0.02):
        if min(n_heads, head_dim, value_dim, rank) < 1 or not tau > 0.0:
            raise ValueError("gated linear attention: every size must be at least 1 and tau positive")
        if head_dim > 256 or rank > 765:
            raise ValueError("gated linear attention: the kernels take keys up to 256 wide and a decay rank up to 765")
        self.hidden_size = int(hidden_size)
        self.n_heads, self.head_dim, self.value_dim = int(n_heads), int(head_dim), int(value_dim)
        self.rank, self.tau = int(rank), float(tau)
        self.norm_eps = float(norm_eps)
        self.tensor_prefix = tensor_prefix
        self.init_std = float(init_std)
        self.in_proj: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.a2t: Optional[torch.Tensor] = None           # float32 [rank, heads * head_dim]
        self.norm_all: Optional[torch.Tensor] = None      # the norm's weight, once per head
        self.w: Dict[str, torch.Tensor] = {}

    # ---- the packed projection's columns --------------------------------------------------
    def _segments(self):
        """(name of the tensor, rows) in the order of the packed projection."""
        nk, nv = self.n_heads * self.head_dim, self.n_heads * self.value_dim
        return [("q", nk), ("k", nk), ("v", nv), ("g", nv), ("a1", self.rank)]

    # ---- weights ----------------------------------------------------------------------
    def tensor_specs(self, prefix: str) -> List[TensorSpec]:
        p = f"{prefix}{self.tensor_prefix}"
        init = Init(0.0, self.init_std)
        nk = self.n_heads * self.head_dim
        specs = [TensorSpec(f"{p}{n}", (rows, self.hidden_size), MATRIX, init) for n, rows in self._segments()]
        # the decay's second matrix takes part in a 32-bit product: held in float32
        return specs + [TensorSpec(f"{p}a2", (nk, self.rank), VECTOR, Init(0.0, 0.1)),
                        TensorSpec(f"{p}a2.b", (nk,), VECTOR, Init(1.0, 1.0)),
                        TensorSpec(f"{p}norm", (self.value_dim,), VECTOR, Init(1.0, 0.0)),
                        TensorSpec(f"{p}o", (self.hidden_size, self.n_heads * self.value_dim), MATRIX, init)]

    def load(self, prefix: str, weights: Dict[str, torch.Tensor]) -> None:
        p = f"{prefix}{self.tensor_prefix}"
        parts = [weights[f"{p}{n}"] for n, _ in self._segments()]
        if len({t.dtype for t in parts}) != 1:
            parts = [t.to(torch.float32) for t in parts]
        self.in_proj = Linear(torch.cat(parts, dim=0).contiguous())
        self.out = Linear(weights[f"{p}o"])
        self.w = {n: weights[f"{p}{n}"] for n in ("a2", "a2.b", "norm")}
        self.a2t = self.w["a2"].to(torch.float32).t().contiguous()
        self.norm_all = self.w["norm"].repeat(self.n_heads).contiguous()
        self.accepts_row_scale = self.in_proj.takes_row_scale()

    def export(self, prefix: str) -> Dict[str, torch.Tensor]:
        p = f"{prefix}{self.tensor_prefix}"
        out, at = {f"{p}o": self.out.weight}, 0
        for n, rows in self._segments():
            out[f"{p}{n}"] = self.in_proj.weight[at:at + rows]
            at += rows
        out.update({f"{p}{n}": t for n, t in self.w.items()})
        return out

    # ---- what it keeps per sequence -----------------------------------------------------
    def state_request(self) -> Sequence[StateRequest]:
        # a column of S (one value channel, all key channels) is contiguous: the lanes of the
        # recurrence's kernel keep stretches of it in registers
        return (StateRequest(GLA_STATE, (self.n_heads, self.value_dim, self.head_dim), torch.float32),)

    # ---- the step -----------------------------------------------------------------------
    def forward_add(self, x: torch.Tensor, ctx: StepContext, binding: CallBinding,
                    residual: torch.Tensor) -> None:
        proj = self.in_proj.forward(x, torch.float32, row_scale=ctx.input_scale)
        project_out(self.out, self.run(proj, 0, ctx, binding), ctx, residual)

    def run(self, proj: torch.Tensor, off: int, ctx: StepContext, binding: CallBinding) -> torch.Tensor:
        """The operand of the output product, from the packed projection's columns in ``proj`` (float32
        rows, this mixer's columns from ``off`` on)."""
        n, dev = proj.shape[0], proj.device
        nk, nv = self.n_heads * self.head_dim, self.n_heads * self.value_dim
        q_off, k_off, v_off = off, off + nk, off + 2 * nk
        g_off = v_off + nv
        a_off = g_off + nv
        decay = torch.empty((n, nk), dtype=torch.float32, device=dev)
        K.sigmoid_decay(proj[:, a_off:a_off + self.rank], self.a2t, self.w["a2.b"], self.tau, decay)
        o = torch.empty((n, nv), dtype=torch.float32, device=dev)
        K.gla_scan(proj, q_off, k_off, v_off, decay, self.head_dim ** -0.5, binding.state[GLA_STATE],
                   ctx.cu_seqlens, ctx.slots, o, ctx.n_rows, ctx.max_row_tokens)
        gated = torch.empty((n, nv), dtype=ctx.act_dtype, device=dev)
        K.unit_norm_gate(o, proj, g_off, gated, self.n_heads, self.norm_eps, "silu", weight=self.norm_all)
        return gated
