"""Small Pazatar configurations of the tests, each with sizes of its own, and their folders."""
from __future__ import annotations

import os
import tempfile

import torch


def _att(heads, kv, dim, scale, chunk, base=1e4, dims=None, yarn=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale}
    if chunk:
        m["mask"] = {"size": chunk}
    if dims != 0:
        m["rot"] = {"base": base, "dims": dim if dims is None else dims}
        if yarn:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "attention", "mixer": m}


def _par(left, right):
    heads, kv, dim, vdim, scale, cap, taps, chunk, base, dims, bands = left
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap}
    if taps:
        m["conv"] = taps
    if chunk:
        m["mask"] = {"size": chunk}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
        if bands:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "low", "high"), bands))
    return {"type": "parallel", "mixer": {"left": m, "right": dict(zip(("heads", "dim", "vdim", "tau", "decay_rank"),
                                                                       right))}}


def _ff(layer, ff):
    return dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


# both mixers, sizes that differ everywhere; chunks of 20 and 33 positions; a loop over the middle with
# two layers of different kinds; a layer without a feed-forward
PAZ_A = {
    "architecture": "Pazatar", "vocab": 97, "width": 64, "norm": {"eps": 1e-6},
    "layers": [_ff(_par((4, 2, 16, 24, 0.4, 5.0, 4, 20, 1e3, 8, (3.0, 40, 1.0, 6.0)), (3, 12, 20, 4.0, 5)), 80),
               _ff(_att(3, 1, 24, 0.3, 33, 5e3, 16, (1.5, 30, 4.0, 0.5)), 56),
               _ff(_par((2, 2, 40, 16, 0.2, 9.0, 2, 70, 500.0, 40, (8.0, 128, 0.5, 2.0)), (2, 16, 8, 9.0, 9)), None),
               _ff(_att(4, 4, 16, 0.45, 50, 1e4, 10), 96)],
    "loop": {"start": 1, "stop": 3, "times": 3},
}
# a width the tensor-core product does not take, heads that are multiples of nothing (the generic attention
# kernel), one tap and no convolution, layers without a chunk mask, rotation or its scaling; no loop
PAZ_B = {
    "architecture": "Pazatar", "vocab": 131, "width": 100, "norm": {"eps": 1e-5},
    "layers": [_ff(_att(5, 5, 10, 0.35, 45, 300.0, 4, (2.5, 60, 3.0, 0.3)), 36),
               _ff(_par((6, 3, 10, 14, 0.5, 3.0, 1, 0, 2e3, 6, (2.0, 100, 1.0, 3.0)), (5, 10, 7, 2.0, 3)), 44),
               _ff(_att(4, 1, 18, 0.3, 0, dims=0), 52),
               _ff(_par((3, 1, 12, 9, 0.6, 12.0, 0, 128, 1e4, 0, None), (1, 40, 33, 25.0, 1)), 28)],
    "loop": None,
}
# keys and values of 128 and 64 (the tensor-memory kernel), keys wider than 128 in the recurrence, chunks of
# a page, two pages and a little more than two; a loop over one layer
PAZ_C = {
    "architecture": "Pazatar", "vocab": 211, "width": 192, "norm": {"eps": 1e-5},
    "layers": [_ff(_att(4, 2, 128, 0.09, 130, 8e4, 128, (4.0, 64, 8.0, 1.0)), 320),
               _ff(_par((8, 2, 64, 64, 0.15, 7.0, 3, 128, 3e4, 32, (6.0, 90, 1.0, 5.0)), (2, 160, 48, 12.0, 24)), 256),
               _ff(_att(2, 1, 64, 0.2, 64, 1e3, 64), 128)],
    "loop": {"start": 1, "stop": 2, "times": 2},
}
# many query heads on one key head, eight taps, a loop over all layers, keys of 128 with values of 96
PAZ_D = {
    "architecture": "Pazatar", "vocab": 173, "width": 128, "norm": {"eps": 1e-6},
    "layers": [_ff(_par((20, 1, 24, 32, 0.3, 4.0, 8, 90, 2e3, 12, (5.0, 200, 2.0, 4.0)), (4, 24, 16, 11.0, 2)), 200),
               _ff(_par((2, 1, 128, 96, 0.1, 15.0, 5, 200, 6e4, 64, None), (1, 64, 128, 6.0, 40)), 72),
               _ff(_att(18, 1, 32, 0.25, 96, 700.0, 20), 152)],
    "loop": {"start": 0, "stop": 3, "times": 2},
}
CASES = {"A": (PAZ_A, 71), "B": (PAZ_B, 72), "C": (PAZ_C, 73), "D": (PAZ_D, 74)}


def loud_weights(folder: str, seed: int) -> None:
    """Rewrites the small learned tensors of a folder so that every one of them matters: decays from fast
    to slow, taps of every sign, steps of the loop as large as the stream, norm weights away from 1."""
    from minfer_b200.weights.safetensors_io import load_all, save_file
    w = load_all(folder)
    gen = torch.Generator().manual_seed(seed)

    def rnd(shape, mean, std):
        return torch.randn(shape, generator=gen) * std + mean

    for name in sorted(w):
        t = w[name]
        if name.endswith(".conv"):
            new = rnd(t.shape, 0.2, 0.6)
        elif name.endswith("a2"):
            new = rnd(t.shape, 0.0, 1.0 * t.shape[-1] ** -0.5)
        elif name.endswith("a1"):
            new = rnd(t.shape, 0.0, 1.5 * t.shape[-1] ** -0.5)
        elif name.endswith("a2.b"):
            new = rnd(t.shape, 1.0, 2.0)
        elif name == "loop.step":
            new = rnd(t.shape, 0.0, 0.5)
        elif "norm" in name or name.endswith(".out"):
            new = rnd(t.shape, 1.0, 0.25)
        else:
            continue
        w[name] = new.to(t.dtype)
    save_file(w, os.path.join(folder, "model.safetensors"), metadata={"format": "pt"})


def make_folder(name: str, store: str = "bfloat16", cfg=None, seed=None) -> str:
    """A folder with seeded weights: matrices N(0, 0.08), the small learned tensors loud
    (``loud_weights``)."""
    from minfer_b200.model import write_random_model
    if cfg is None:
        cfg, seed = CASES[name]
    folder = tempfile.mkdtemp(prefix=f"minfer_b200_paz{name}_")
    write_random_model(folder, cfg, seed, store, weight_std=0.08)
    loud_weights(folder, seed)
    return folder
