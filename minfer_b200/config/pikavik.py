"""Typed configuration of the Pikavik decoder, read from its own config.json keys.

The design: token embedding; layers with one norm that both sublayers read, x += a1 * mixer(y) +
a2 * ff(y) with learned vectors a1 and a2 (the feed-forward optional); the
norms of the stream multiply by 1 + w.  The mixer is WKV, mLSTM, or latent
attention whose queries go through a latent too (rotated part shared by all heads, a learned
sink per head); the feed-forward is routed (sigmoid scores, experts chosen within the best groups, a
clamped activation, a gated shared expert).  Final norm, head.  config.json keys:

    architecture        "Pikavik"
    vocab, width        sizes; norm.eps: eps of every norm
    layers[i].type      "wkv" | "mlstm" | "latent_attention"
    layers[i].mixer     wkv: heads, dim (decay_rank: only for random weights; a checkpoint's tensors
                        give it); mlstm: heads, dim, vdim, gate_cap; latent_attention: heads, dim,
                        rot_dim, vdim, kv_rank, q_rank, scale, rot {base, dims}
    layers[i].mlp       null or {kind: "moe", expert {ff, limit}, router {experts, top, scale,
                        groups {count, keep}}, shared {ff, limit} or null}
    max_positions       optional bound on a sequence's length (default 2^20)

Tensor names: ``embed``, ``final.norm``, ``head``, and per layer ``l<i>.norm1``, ``l<i>.ls1``,
``l<i>.ls2``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field, replace
from typing import Any, Mapping, Optional, Sequence, Tuple

from .base import ConfigError, ConfigReader, LayerSpec, ModelPlan, PartSpec, default_schedule

ARCHITECTURE = "Pikavik"
MIXERS = ("wkv", "mlstm", "latent_attention")
DEFAULT_MAX_POSITIONS = 1 << 20
DEFAULT_DECAY_RANK = 64


@dataclass(frozen=True)
class PikavikLayer:
    type: str
    mixer: Mapping[str, Any]        # the mixer's object as config.json gives it (checked)
    mlp: Optional[Mapping[str, Any]]
    decay_rank: Optional[int] = None     # wkv: rows of the decay's first matrix, if known


def _object(data: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    if not isinstance(data.get(key), Mapping):
        raise ConfigError(f"{where}: key '{key}' must be an object")
    return data[key]


@dataclass(frozen=True)
class PikavikConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[PikavikLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str = "config.json") -> "PikavikConfig":
        r = ConfigReader(data, where)
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, (list, tuple)) or not raw_layers:
            raise ConfigError(f"{where}: key 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw_layers):
            w = f"{where}.layers[{i}]"
            kind = ConfigReader(entry, w).string("type")
            if kind not in MIXERS:
                raise ConfigError(f"{w}: unknown mixer type {kind!r} (known: {', '.join(MIXERS)})")
            mixer = _object(entry, "mixer", w)
            mlp = entry.get("mlp")
            if mlp is not None:
                mlp_kind = ConfigReader(mlp, f"{w}.mlp").string("kind", default="moe")
                if mlp_kind != "moe":
                    raise ConfigError(f"{w}.mlp: unknown kind {mlp_kind!r} (known: moe)")
            layers.append(PikavikLayer(
                kind, dict(mixer), None if mlp is None else dict(mlp),
                ConfigReader(mixer, f"{w}.mixer").optional_integer("decay_rank", minimum=1)))
        cfg = cls(
            vocab=r.integer("vocab", minimum=1),
            width=r.integer("width", minimum=1),
            norm_eps=ConfigReader(data.get("norm") or {}, f"{where}.norm").number("eps", positive=True),
            layers=tuple(layers),
            max_positions=r.integer("max_positions", default=DEFAULT_MAX_POSITIONS, minimum=1),
            extra={k: v for k, v in data.items()},
        )
        cfg.plan()          # every key of every layer is read (and refused) here, not at the first step
        return cfg

    @classmethod
    def from_folder(cls, folder: str) -> "PikavikConfig":
        path = os.path.join(folder, "config.json")
        with open(path, "r", encoding="utf-8") as f:
            return cls.from_dict(json.load(f), where=path)

    def with_tensor_shapes(self, shapes: Mapping[str, Sequence[int]]) -> "PikavikConfig":
        """The sizes that only a checkpoint's tensors give: the ranks of the decays."""
        layers = []
        for i, layer in enumerate(self.layers):
            w1 = shapes.get(f"l{i}.mix.w1")
            if layer.type == "wkv" and w1 is not None and len(w1) == 2:
                layer = replace(layer, decay_rank=int(w1[0]))
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        layers = []
        for layer in self.layers:
            mixer = dict(layer.mixer)
            if layer.type == "wkv":
                mixer["decay_rank"] = layer.decay_rank or DEFAULT_DECAY_RANK
            layers.append({"type": layer.type, "mixer": mixer,
                           "mlp": None if layer.mlp is None else dict(layer.mlp)})
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": layers}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    # ---- lowering to parts ----------------------------------------------------------
    def _mixer(self, i: int, layer: PikavikLayer) -> PartSpec:
        w = f"config.layers[{i}].mixer"
        m = layer.mixer
        r = ConfigReader(m, w)
        heads = r.integer("heads", minimum=1)
        dim = r.integer("dim", minimum=1)
        common = dict(hidden_size=self.width, norm_eps=self.norm_eps, n_heads=heads, head_dim=dim,
                      tensor_prefix="mix.")
        if layer.type == "wkv":
            return PartSpec("wkv", dict(common, rank=layer.decay_rank or DEFAULT_DECAY_RANK))
        if layer.type == "mlstm":
            return PartSpec("mlstm", dict(common, value_dim=r.integer("vdim", default=dim, minimum=1),
                                          gate_cap=r.number("gate_cap", positive=True)))
        rot_dim = r.integer("rot_dim", default=0, minimum=0)
        position = None
        if rot_dim > 0 and m.get("rot") is not None:
            rr = ConfigReader(_object(m, "rot", w), f"{w}.rot")
            dims = rr.integer("dims", default=rot_dim, minimum=0)
            if dims % 2 != 0 or dims > rot_dim:
                raise ConfigError(f"{w}.rot: dims {dims} must be even and at most rot_dim {rot_dim}")
            if dims > 0:
                position = PartSpec("rotary", {"head_dim": rot_dim, "rotary_dim": dims,
                                               "theta": rr.number("base", positive=True), "style": "neox"})
        return PartSpec("latent_attention", dict(
            common, rot_dim=rot_dim, value_dim=r.integer("vdim", default=dim, minimum=1),
            kv_rank=r.integer("kv_rank", minimum=1), q_rank=r.integer("q_rank", minimum=1),
            scale=r.number("scale"), window=0, sink=True, gate=False, position=position))

    def _feed_forward(self, i: int, layer: PikavikLayer) -> Optional[PartSpec]:
        if layer.mlp is None:
            return None
        w = f"config.layers[{i}].mlp"
        er = ConfigReader(_object(layer.mlp, "expert", w), f"{w}.expert")
        router = _object(layer.mlp, "router", w)
        rr = ConfigReader(router, f"{w}.router")
        experts = rr.integer("experts", minimum=1)
        top = rr.integer("top", minimum=1)
        count = keep = 1
        if router.get("groups") is not None:
            gr = ConfigReader(_object(router, "groups", f"{w}.router"), f"{w}.router.groups")
            count = gr.integer("count", minimum=1)
            keep = gr.integer("keep", default=count, minimum=1)
            if experts % count != 0 or keep > count:
                raise ConfigError(f"{w}.router: {experts} experts do not form {count} groups of which "
                                  f"{keep} are kept")
        if top > keep * (experts // count):
            raise ConfigError(f"{w}.router: top {top} exceeds the {keep * (experts // count)} experts that "
                              f"{keep} of {count} groups hold")
        shared = None
        if layer.mlp.get("shared") is not None:
            sr = ConfigReader(_object(layer.mlp, "shared", w), f"{w}.shared")
            shared = {"ff": sr.integer("ff", minimum=1), "limit": sr.number("limit", positive=True),
                      "name": "mlp.shared", "gate_name": "mlp.shared.sg"}
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": er.integer("ff", minimum=1),
            "n_experts": experts, "top": top, "activation": "clamped_swish",
            "limit": er.number("limit", positive=True), "scoring": "sigmoid_groups", "groups": count,
            "keep_groups": keep, "weight_scale": rr.number("scale", default=1.0),
            "router_name": "mlp.router", "router_bias_name": None, "expert_name": "mlp.e{e}",
            "shared": shared})

    def plan(self) -> ModelPlan:
        norm = PartSpec("rms_norm", {"size": self.width, "eps": self.norm_eps, "offset": 1.0})
        layers = []
        unused = []
        for i, layer in enumerate(self.layers):
            ffn = self._feed_forward(i, layer)
            if ffn is None:
                unused.append(f"l{i}.ls2")
            layers.append(LayerSpec(
                prefix=f"l{i}.",
                block=PartSpec("parallel", {"layer_scale": ("ls1", "ls2")}),
                mixer=self._mixer(i, layer),
                mixer_norm=norm.with_params(name="norm1", tensor_name="norm1"),
                feed_forward=ffn,
                feed_forward_norm=None,
            ))
        plan = ModelPlan(
            architecture=ARCHITECTURE,
            vocab_size=self.vocab,
            hidden_size=self.width,
            embedding_name="embed",
            head_name="head",
            final_norm=norm.with_params(name="final.norm", tensor_name="final.norm"),
            final_norm_prefix="",
            layers=layers,
            schedule=default_schedule(len(layers)),
            max_positions=self.max_positions,
            model_part_prefix="",
            ignorable_tensors=tuple(unused),
        )
        plan.validate()
        return plan
