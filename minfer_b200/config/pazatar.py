"""Typed configuration of the Pazatar decoder, read from its own config.json keys.

The design: token embedding; layers that norm before and after each sublayer, x += norm1b(mixer(norm1(x))),
x += norm2b(ff(norm2(x))) (the second half optional); the mixer is grouped attention whose values are its
keys before norm and rotation (q and k normed over all heads, an interleaved YaRN-scaled rotation, a chunk
mask), or two mixers side by side, each output normed, half their sum: grouped attention behind short
convolutions (q and k normed per head, a partial rotation scaled by bands of wavelength, soft-capped scores,
a chunk mask, one added to the softmax's sum) and gated linear attention (a decay per key channel,
per-sequence state).  A stretch of the layers may run several times in a row with the same weights (each pass
with keys and states of its own), a learned vector added before each pass.  Dense feed-forward with the
square of relu; final norm; the head is the embedding table.  config.json keys:

    architecture        "Pazatar"
    vocab, width        sizes; norm.eps: eps of every norm
    loop                null, or {start, stop, times}: layers start .. stop-1 run `times` times
    layers[i].type      "attention" | "parallel"
    layers[i].mixer     attention: heads, kv_heads, dim, vdim (= dim), scale, mask {size},
                        rot {base, dims, scaling {factor, original, fast, slow}}
                        parallel: left {heads, kv_heads, dim, vdim, scale, softcap, conv, mask {size},
                        rot {base, dims, scaling {factor, original, low, high}}}, right {heads, dim, vdim, tau}
    layers[i].mlp       null, or {kind: "dense", ff}
    max_positions       optional bound on a sequence's length (default 2^20)

The rank of the decay's pair of matrices is no key: a checkpoint's shapes give it (``with_tensor_shapes``);
a written configuration may name it as ``right.decay_rank``.  Tensor names: ``embed``, ``loop.step``,
``final.norm``, and per layer ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.*``,
``l<i>.mlp.{up,down}``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field, replace
from typing import Any, Mapping, Optional, Tuple

from .base import (ConfigError, ConfigReader, LayerSpec, ModelPlan, PartSpec, default_schedule,
                   looped_schedule)

ARCHITECTURE = "Pazatar"
MIXERS = ("attention", "parallel")
FEED_FORWARDS = ("dense",)
DEFAULT_MAX_POSITIONS = 1 << 20
DEFAULT_DECAY_RANK = 16


def _object(data: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = data.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"{where}: key '{key}' must be an object")
    return value


def _rotation(m: Mapping[str, Any], where: str, head_width: int, style: str,
              scaling_keys: Tuple[str, ...]) -> Optional[PartSpec]:
    """The ``rot`` object of a mixer as a rotary part (None: no rotation)."""
    if m.get("rot") is None:
        return None
    w = f"{where}.rot"
    data = _object(m, "rot", where)
    r = ConfigReader(data, w)
    dims = r.integer("dims", default=head_width, minimum=0)
    if dims == 0:
        return None
    if dims % 2 != 0 or dims > head_width:
        raise ConfigError(f"{w}: dims {dims} must be even and at most {head_width}")
    params = {"head_dim": head_width, "rotary_dim": dims, "theta": r.number("base", positive=True), "style": style}
    if data.get("scaling") is not None:
        sr = ConfigReader(_object(data, "scaling", w), f"{w}.scaling")
        params["scaling"] = {k: sr.number(k, positive=True) for k in scaling_keys}
    return PartSpec("rotary", params)


def _chunk(m: Mapping[str, Any], where: str) -> int:
    if m.get("mask") is None:
        return 0
    return ConfigReader(_object(m, "mask", where), f"{where}.mask").integer("size", minimum=1)


@dataclass(frozen=True)
class PazatarLayer:
    type: str
    mixer: Mapping[str, Any]        # the mixer's object as config.json gives it (checked)
    mlp_kind: Optional[str]         # None: no feed-forward
    ff: int = 0
    decay_rank: int = 0             # parallel: rank of the decay's matrices (0: not known, the default)


@dataclass(frozen=True)
class PazatarConfig:
    vocab: int
    width: int
    norm_eps: float
    loop: Optional[Tuple[int, int, int]]      # (start, stop, times)
    layers: Tuple[PazatarLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, data: Mapping[str, Any], where: str = "config.json") -> "PazatarConfig":
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
            rank = 0
            if kind == "parallel":
                right = _object(mixer, "right", f"{w}.mixer")
                rank = ConfigReader(right, f"{w}.mixer.right").integer("decay_rank", default=0, minimum=0)
            mlp_kind, ff = None, 0
            if entry.get("mlp") is not None:
                mr = ConfigReader(_object(entry, "mlp", w), f"{w}.mlp")
                mlp_kind = mr.string("kind")
                if mlp_kind not in FEED_FORWARDS:
                    raise ConfigError(f"{w}.mlp: unknown kind {mlp_kind!r} (known: {', '.join(FEED_FORWARDS)})")
                ff = mr.integer("ff", minimum=1)
            layers.append(PazatarLayer(kind, dict(mixer), mlp_kind, ff, rank))
        loop = None
        if data.get("loop") is not None:
            lo = ConfigReader(_object(data, "loop", where), f"{where}.loop")
            loop = (lo.integer("start", minimum=0), lo.integer("stop", minimum=1),
                    lo.integer("times", minimum=1))
            if not loop[0] < loop[1] <= len(layers):
                raise ConfigError(f"{where}.loop: layers [{loop[0]}, {loop[1]}) do not lie within the "
                                  f"{len(layers)} layers")
        cfg = cls(
            vocab=r.integer("vocab", minimum=1),
            width=r.integer("width", minimum=1),
            norm_eps=ConfigReader(data.get("norm") or {}, f"{where}.norm").number("eps", positive=True),
            loop=loop,
            layers=tuple(layers),
            max_positions=r.integer("max_positions", default=DEFAULT_MAX_POSITIONS, minimum=1),
            extra={k: v for k, v in data.items()},
        )
        cfg.plan()          # every mixer's keys are read (and refused) here, not at the first step
        return cfg

    @classmethod
    def from_folder(cls, folder: str) -> "PazatarConfig":
        path = os.path.join(folder, "config.json")
        with open(path, "r", encoding="utf-8") as f:
            return cls.from_dict(json.load(f), where=path)

    def with_tensor_shapes(self, shapes: Mapping[str, Tuple[int, ...]]) -> "PazatarConfig":
        """The sizes that only a checkpoint's tensors give: the ranks of the decays."""
        layers = []
        for i, layer in enumerate(self.layers):
            a1 = shapes.get(f"l{i}.mix.right.a1")
            if layer.type == "parallel" and a1 is not None and len(a1) == 2:
                layer = replace(layer, decay_rank=int(a1[0]))
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    def to_dict(self) -> dict:
        layers = []
        for layer in self.layers:
            mixer = dict(layer.mixer)
            if layer.type == "parallel":
                mixer["right"] = dict(mixer["right"], decay_rank=layer.decay_rank or DEFAULT_DECAY_RANK)
            layers.append({"type": layer.type, "mixer": mixer,
                           "mlp": None if layer.mlp_kind is None else {"kind": layer.mlp_kind, "ff": layer.ff}})
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "layers": layers,
               "loop": None if self.loop is None else
               {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    # ---- lowering to parts ----------------------------------------------------------
    def _heads(self, m: Mapping[str, Any], w: str) -> dict:
        """What both kinds of attention read alike."""
        r = ConfigReader(m, w)
        heads = r.integer("heads", minimum=1)
        kv = r.integer("kv_heads", default=heads, minimum=1)
        if heads % kv != 0:
            raise ConfigError(f"{w}: heads {heads} is not a multiple of kv_heads {kv}")
        dim = r.integer("dim", minimum=1)
        softcap = r.number("softcap", default=0.0)
        if softcap < 0.0:
            raise ConfigError(f"{w}: key 'softcap' must not be negative, got {softcap}")
        return dict(hidden_size=self.width, norm_eps=self.norm_eps, n_heads=heads, n_kv_heads=kv, head_dim=dim,
                    value_dim=r.integer("vdim", default=dim, minimum=1), scale=r.number("scale"), softcap=softcap,
                    chunk=_chunk(m, w), conv=r.integer("conv", default=0, minimum=0), bias=False, qk_norm=True)

    def _mixer(self, i: int, layer: PazatarLayer) -> PartSpec:
        w = f"config.layers[{i}].mixer"
        m = layer.mixer
        if layer.type == "attention":
            params = self._heads(m, w)
            if params["value_dim"] != params["head_dim"]:
                raise ConfigError(f"{w}: the values are the keys, but vdim {params['value_dim']} is not dim "
                                  f"{params['head_dim']}")
            return PartSpec("qk_norm_attention", dict(
                params, norm_scope="all", values="keys", tensor_prefix="mix.",
                position=_rotation(m, w, params["head_dim"], "interleaved", ("factor", "original", "fast", "slow"))))
        left, right = _object(m, "left", w), _object(m, "right", w)
        params = self._heads(left, f"{w}.left")
        rr = ConfigReader(right, f"{w}.right")
        dim = rr.integer("dim", minimum=1)
        return PartSpec("parallel", dict(
            tensor_prefix="mix.",
            norms={"width": self.width, "eps": self.norm_eps, "mult": 0.5, "left": "left.out", "right": "right.out"},
            left=PartSpec("qk_norm_attention", dict(
                params, norm_scope="head", sink=True,
                position=_rotation(left, f"{w}.left", params["head_dim"], "neox",
                                   ("factor", "original", "low", "high")))),
            right=PartSpec("gated_linear_attention", dict(
                hidden_size=self.width, norm_eps=self.norm_eps, n_heads=rr.integer("heads", minimum=1), head_dim=dim,
                value_dim=rr.integer("vdim", default=dim, minimum=1), tau=rr.number("tau", positive=True),
                rank=layer.decay_rank or DEFAULT_DECAY_RANK))))

    def plan(self) -> ModelPlan:
        norm = PartSpec("rms_norm", {"size": self.width, "eps": self.norm_eps})

        def named(name: str) -> PartSpec:
            return norm.with_params(name=name, tensor_name=name)

        layers = []
        for i, layer in enumerate(self.layers):
            ffn = None
            if layer.mlp_kind == "dense":
                ffn = PartSpec("dense_mlp", {
                    "hidden_size": self.width, "intermediate_size": layer.ff, "activation": "relu2",
                    "up_name": "mlp.up", "down_name": "mlp.down"})
            layers.append(LayerSpec(
                prefix=f"l{i}.",
                block=PartSpec("sandwich_norm", {"output_norms": (named("norm1b"), named("norm2b"))}),
                mixer=self._mixer(i, layer),
                mixer_norm=named("norm1"),
                feed_forward=ffn,
                feed_forward_norm=None if ffn is None else named("norm2"),
            ))
        injection = None
        schedule = default_schedule(len(layers))
        if self.loop is not None:
            schedule = looped_schedule(len(layers), *self.loop)
            injection = PartSpec("pass_injection", {"width": self.width, "passes": self.loop[2],
                                                    "tensor_name": "loop.step", "add_embedding": False})
        plan = ModelPlan(
            architecture=ARCHITECTURE,
            vocab_size=self.vocab,
            hidden_size=self.width,
            embedding_name="embed",
            head_name=None,
            final_norm=named("final.norm"),
            final_norm_prefix="",
            layers=layers,
            schedule=schedule,
            max_positions=self.max_positions,
            pass_injection=injection,
            model_part_prefix="",
            # (a layer without a feed-forward reads no norms for it)
            ignorable_tensors=tuple(f"l{i}.{n}" for i, layer in enumerate(self.layers) if layer.mlp_kind is None
                                    for n in ("norm2", "norm2b")),
        )
        plan.validate()
        return plan
