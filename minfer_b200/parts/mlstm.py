"""mLSTM as a mixer: a matrix-valued state per head that exponential gates fill and empty, kept in range
by a running maximum, with a normalizer.

    q = Wq u * head_dim^(-1/2),  k = Wk u  (heads of ``head_dim``),  v = Wv u  (heads of ``value_dim``)
    per head  i = cap tanh((Wi u + bi) / cap),  f = log sigmoid(cap tanh((Wf u + bf) / cap))
    m_t = max(f + m_(t-1), i)                       m starts at 0, S and n at zero
    S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k_t v_t^T;   n_t likewise with k_t alone
    o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
    o <- o / sqrt(mean(o^2) + eps) per head, times a weight over all heads, times sigmoid(Wg u);  Wo

State per sequence (float32, zeroed when a slot is handed out): S with n as one more column, and the
maximum.  A step may bring any number of tokens per sequence; the recurrence walks them in order.
One packed product gives q | k | v | g | i | f in float32; everything between it and the output
product is float32 in both engines.  Tensor names behind ``prefix + tensor_prefix``: ``q``, ``k``, ``v``,
``g``, ``i``, ``i.b``, ``f``, ``f.b``, ``norm``, ``o``.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from ..kernels import api as K
from ..weights.spec import MATRIX, VECTOR, Init, TensorSpec
from .base import CallBinding, Mixer, StateRequest, StepContext
from .linear import Linear
from .sink_attention import project_out

MLSTM_STATE = "mlstm.state"
MLSTM_MAXIMUM = "mlstm.maximum"


class MLstm(Mixer):
    capturable = True      # launches kernels only; safe inside a CUDA graph capture
    stores_fresh_output = True     # its last product goes through ``project_out``

    def libraries(self, dtype: torch.dtype) -> List[str]:
        return ["ops", "outer_scan", "retention", "gemm_tc" if dtype == torch.bfloat16 else "gemm_simt"]

    def __init__(self, hidden_size: int, n_heads: int, head_dim: int, value_dim: int, gate_cap: float,
                 norm_eps: float, tensor_prefix: str = "mix.", init_std: float = 0.02):
        if min(n_heads, head_dim, value_dim) < 1:
            raise ValueError("mlstm: every size must be at least 1")
        if head_dim > 256:
            raise ValueError("mlstm: the kernel takes keys up to 256 wide")
        if not gate_cap > 0.0:
            raise ValueError("mlstm: the cap of the gates must be positive")
        self.hidden_size = int(hidden_size)
        self.n_heads, self.head_dim, self.value_dim = int(n_heads), int(head_dim), int(value_dim)
        self.gate_cap, self.norm_eps = float(gate_cap), float(norm_eps)
        self.tensor_prefix = tensor_prefix
        self.init_std = float(init_std)
        self.proj: Optional[Linear] = None
        self.out: Optional[Linear] = None
        self.w: Dict[str, torch.Tensor] = {}

    def _segments(self):
        """(name of the tensor, rows) in the order of the packed projection."""
        nq, nv = self.n_heads * self.head_dim, self.n_heads * self.value_dim
        return [("q", nq), ("k", nq), ("v", nv), ("g", nv), ("i", self.n_heads), ("f", self.n_heads)]

    # ---- weights ----------------------------------------------------------------------
    def tensor_specs(self, prefix: str) -> List[TensorSpec]:
        p = f"{prefix}{self.tensor_prefix}"
        init = Init(0.0, self.init_std)
        nv = self.n_heads * self.value_dim
        specs = [TensorSpec(f"{p}{n}", (rows, self.hidden_size), MATRIX, init) for n, rows in self._segments()]
        specs += [TensorSpec(f"{p}i.b", (self.n_heads,), VECTOR, Init(0.0, 0.5)),
                  TensorSpec(f"{p}f.b", (self.n_heads,), VECTOR, Init(3.0, 1.0)),
                  TensorSpec(f"{p}norm", (nv,), VECTOR, Init(1.0, 0.0)),
                  TensorSpec(f"{p}o", (self.hidden_size, nv), MATRIX, init)]
        return specs

    def load(self, prefix: str, weights: Dict[str, torch.Tensor]) -> None:
        p = f"{prefix}{self.tensor_prefix}"
        parts = [weights[f"{p}{n}"] for n, _ in self._segments()]
        if len({t.dtype for t in parts}) != 1:
            parts = [t.to(torch.float32) for t in parts]
        self.proj = Linear(torch.cat(parts, dim=0).contiguous())
        self.w = {n: weights[f"{p}{n}"] for n in ("i.b", "f.b", "norm")}
        self.out = Linear(weights[f"{p}o"])
        self.accepts_row_scale = self.proj.takes_row_scale()

    def export(self, prefix: str) -> Dict[str, torch.Tensor]:
        p = f"{prefix}{self.tensor_prefix}"
        out, at = {}, 0
        for n, rows in self._segments():
            out[f"{p}{n}"] = self.proj.weight[at:at + rows]
            at += rows
        out.update({f"{p}{n}": t for n, t in self.w.items()})
        out[f"{p}o"] = self.out.weight
        return out

    # ---- what it keeps per sequence -----------------------------------------------------
    def state_request(self) -> Sequence[StateRequest]:
        return (StateRequest(MLSTM_STATE, (self.n_heads, self.value_dim + 1, self.head_dim), torch.float32),
                StateRequest(MLSTM_MAXIMUM, (self.n_heads, self.value_dim + 1), torch.float32))

    # ---- the step -----------------------------------------------------------------------
    def forward_add(self, x: torch.Tensor, ctx: StepContext, binding: CallBinding,
                    residual: torch.Tensor) -> None:
        n, dev = x.shape[0], x.device
        nh = self.n_heads
        nq, nv = nh * self.head_dim, nh * self.value_dim
        proj = self.proj.forward(x, torch.float32, row_scale=ctx.input_scale)
        o = torch.empty((n, nv), dtype=torch.float32, device=dev)
        den = torch.empty((n, nh), dtype=torch.float32, device=dev)
        i_off = 2 * nq + 2 * nv
        K.mlstm_scan(proj, 0, nq, 2 * nq, i_off, i_off + nh, self.w["i.b"], self.w["f.b"], self.gate_cap,
                     self.head_dim ** -0.5, binding.state[MLSTM_STATE], binding.state[MLSTM_MAXIMUM],
                     ctx.cu_seqlens, ctx.slots, o, den, ctx.n_rows, ctx.max_row_tokens)
        gated = torch.empty((n, nv), dtype=ctx.act_dtype, device=dev)
        K.unit_norm_gate(o, proj, 2 * nq + nv, gated, nh, self.norm_eps, "sigmoid", den=den,
                         weight=self.w["norm"])
        project_out(self.out, gated, ctx, residual)
