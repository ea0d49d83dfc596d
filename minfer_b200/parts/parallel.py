"""Two mixers side by side on the same input, in one of two forms:

    out = left_scale * left(x) + right_scale * right(x)
    out = mult * (norm(left(x), w_left) + norm(right(x), w_right))        (``norms``: an RMS norm each)

First form: each side is any registered mixer that takes an ``out_scale`` (the constant it multiplies
the operand of its last product with), so both sides add their scaled outputs into the same stream
and no kernel of this part's own runs.  Second form: the outputs are kept apart as two terms, K splits
of their last products included, and one kernel norms and adds them (``kernels.api.norm_terms``); a block
that norms the mixer's output again takes the terms themselves (``ctx.extras["takes_terms"]``) and runs
that kernel with its own norms in it.  Sides that can start from a packed projection (``in_proj``,
``run``) share one product in this form.  At most one side may keep cached keys; the per-sequence
state of the two sides is kept side by side under the names ``left.<name>`` / ``right.<name>``.
Tensor names: the sides' own, behind ``prefix + tensor_prefix + "left." / "right."``.
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Dict, List, Mapping, Any, Optional, Sequence, Tuple

import torch

from ..config.base import PartSpec
from ..kernels import api as K
from ..weights.spec import VECTOR, Init, TensorSpec
from .base import CacheRequest, CallBinding, Mixer, StateRequest, StepContext, settle_pending
from .linear import Linear
from .sink_attention import project_out


# MINFER_B200_OVERLAP_SIDES=0: both sides of a step with one token a row on one stream (for comparison)
OVERLAP = os.environ.get("MINFER_B200_OVERLAP_SIDES", "1") != "0"
_other_streams: Dict[Any, torch.cuda.Stream] = {}


def other_stream(device: torch.device) -> torch.cuda.Stream:
    """The stream beside the step's own on which a second side runs, one per device."""
    if device not in _other_streams:
        _other_streams[device] = torch.cuda.Stream(device)
    return _other_streams[device]


@dataclass
class Terms:
    """An output that is still mult * sum_k rms-normed terms: (y, partial, weight) each, as
    ``kernels.api.norm_terms`` takes them."""

    terms: List[Tuple[Optional[torch.Tensor], Optional[torch.Tensor], torch.Tensor]]
    eps: float
    mult: float


def output_term(out: Linear, o: torch.Tensor, ctx: StepContext):
    """out(o) as (y, None) or, where the product leaves K splits, (None, partial)."""
    y = torch.empty((o.shape[0], out.out_features), dtype=torch.float32, device=o.device)
    ctx.extras["fresh_output"] = True
    project_out(out, o, ctx, y)
    pending = ctx.extras.pop("pending", None)
    if pending is None:
        return y, None
    ctx.extras.pop("pending_only", None)
    if pending.bias is not None:
        K.splitk_reduce(pending.partial, pending.bias, y, accumulate=False)
        return y, None
    return None, pending.partial


class ParallelMixer(Mixer):
    stores_fresh_output = True     # answers ``ctx.extras["fresh_output"]`` (see ``project_out``)

    def __init__(self, left: PartSpec, right: PartSpec, left_scale: float = 1.0,
                 right_scale: float = 1.0, tensor_prefix: str = "mix.",
                 norms: Optional[Mapping[str, Any]] = None):
        """``norms``: {width, eps, mult, left, right} (the last two the names of the weights behind
        ``prefix + tensor_prefix``) for the second form, whose sides take no scale."""
        from ..registry import build_part
        self.tensor_prefix = tensor_prefix
        self.sides = []
        self.norms = dict(norms) if norms is not None else None
        self.offers_terms = self.norms is not None
        self.norm_w: List[torch.Tensor] = []
        self.packed: Optional[Linear] = None
        for name, spec, scale in (("left", left, left_scale), ("right", right, right_scale)):
            if self.norms is not None:
                part = build_part("mixer", spec.with_params(tensor_prefix=f"{tensor_prefix}{name}."))
                if not (hasattr(part, "run") and hasattr(part, "in_proj")):
                    raise ValueError(f"the {name} mixer ({spec.kind}) cannot hand its output on as a term")
                self.sides.append((name, part))
                continue
            part = build_part("mixer", spec.with_params(out_scale=float(scale),
                                                        tensor_prefix=f"{tensor_prefix}{name}."))
            if not hasattr(part, "out_scale"):
                raise ValueError(f"the {name} mixer ({spec.kind}) takes no output scale")
            self.sides.append((name, part))
        if sum(1 for _, p in self.sides if p.cache_request() is not None) > 1:
            raise ValueError("only one side of a parallel mixer may keep cached keys")
        if self.norms is not None:
            self.stores_fresh_output = False       # adds into what the buffer holds
        self.capturable = all(getattr(p, "capturable", False) for _, p in self.sides)

    def libraries(self, dtype: torch.dtype) -> List[str]:
        libs: List[str] = ["ops"] if self.norms is not None else []
        for _, part in self.sides:
            libs += [n for n in part.libraries(dtype) if n not in libs]
        return libs

    def tensor_specs(self, prefix: str):
        own = [] if self.norms is None else [
            TensorSpec(f"{prefix}{self.tensor_prefix}{self.norms[name]}", (int(self.norms["width"]),), VECTOR,
                       Init(1.0, 0.0)) for name, _ in self.sides]
        return [s for _, part in self.sides for s in part.tensor_specs(prefix)] + own

    def load(self, prefix: str, weights: Dict[str, torch.Tensor]) -> None:
        for _, part in self.sides:
            part.load(prefix, weights)
        if self.norms is None:
            return
        self.norm_w = [weights[f"{prefix}{self.tensor_prefix}{self.norms[name]}"] for name, _ in self.sides]
        # both sides' first products in one: each side's own becomes a view of its rows
        first = [part.in_proj for _, part in self.sides]
        self.packed = None
        if all(p.bias is None for p in first) and len({p.weight.dtype for p in first}) == 1:
            self.packed = Linear(torch.cat([p.weight for p in first], dim=0).contiguous())
            at = 0
            for p in first:
                p.weight = self.packed.weight[at:at + p.out_features]
                at += p.out_features

    def export(self, prefix: str) -> Dict[str, torch.Tensor]:
        out: Dict[str, torch.Tensor] = {}
        for _, part in self.sides:
            out.update(part.export(prefix))
        for (name, _), w in zip(self.sides, self.norm_w):
            out[f"{prefix}{self.tensor_prefix}{self.norms[name]}"] = w
        return out

    def cache_request(self) -> Optional[CacheRequest]:
        for _, part in self.sides:
            req = part.cache_request()
            if req is not None:
                return req
        return None

    def state_request(self) -> Sequence[StateRequest]:
        return tuple(StateRequest(f"{name}.{r.name}", r.shape, r.dtype)
                     for name, part in self.sides for r in part.state_request())

    def _side_binding(self, name: str, part, binding: CallBinding) -> CallBinding:
        own = {k[len(name) + 1:]: t for k, t in binding.state.items() if k.startswith(name + ".")}
        return CallBinding(cache=binding.cache if part.cache_request() is not None else None,
                           writes_cache=binding.writes_cache, entry=binding.entry,
                           has_readers=binding.has_readers, state=own)

    def _add_terms(self, x: torch.Tensor, ctx: StepContext, binding: CallBinding,
                   residual: Optional[torch.Tensor]) -> None:
        takes = ctx.extras.pop("takes_terms", False)
        proj = self.packed.forward(x, torch.float32) if self.packed is not None else None
        at = [0, self.sides[0][1].in_proj.out_features if proj is not None else 0]

        def term(i: int):
            name, part = self.sides[i]
            rows = proj if proj is not None else part.in_proj.forward(x, torch.float32)
            o = part.run(rows, at[i], ctx, self._side_binding(name, part, binding))
            return output_term(part.out, o, ctx) + (self.norm_w[i],)

        if ctx.single_token and OVERLAP:
            # one token a row: neither side fills the GPU, and both wait on memory.  Every stretch on the
            # other stream begins after all of this one's work and is waited for before this returns, so
            # no memory is handed from one to the other early.
            here, other = torch.cuda.current_stream(x.device), other_stream(x.device)
            other.wait_stream(here)
            with torch.cuda.stream(other):
                second = term(1)
            terms = [term(0), second]
            here.wait_stream(other)
        else:
            terms = [term(0), term(1)]
        out = Terms(terms, float(self.norms["eps"]), float(self.norms["mult"]))
        if takes:
            ctx.extras["terms"] = out
        else:
            settle_pending(ctx, residual)
            K.norm_terms(residual, out.terms, out.eps, out.mult)

    def forward_add(self, x: torch.Tensor, ctx: StepContext, binding: CallBinding,
                    residual: torch.Tensor) -> None:
        ctx.extras.pop("prepare_for", None)        # neither side's product completes the stream alone
        if self.norms is not None:
            self._add_terms(x, ctx, binding, residual)
            return
        fresh = ctx.extras.pop("fresh_output", False)
        for i, (name, part) in enumerate(self.sides):
            if fresh and i == 0:
                ctx.extras["fresh_output"] = True  # the first side stores, the second adds
            part.forward_add(x, ctx, self._side_binding(name, part, binding), residual)
            if i == 0:
                # never two pending products at once; K splits of a first side that stored nothing
                # become the buffer's content
                pending = ctx.extras.pop("pending", None)
                if pending is not None:
                    K.splitk_reduce(pending.partial, pending.bias, residual,
                                    accumulate=not ctx.extras.pop("pending_only", False))
