"""Small Pikavik configurations of the tests, each with sizes of its own, and their folders."""
from __future__ import annotations

import os
import tempfile

import torch


def _wkv(heads, dim, rank):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}}


def _mlstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, dims=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "q_rank": q_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim if dims is None else dims}}}


def _moe(layer, experts, top, groups, keep, scale, ff, limit, shared):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups, "keep": keep}
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": router,
           "shared": None if shared is None else {"ff": shared[0], "limit": shared[1]}}
    return dict(layer, mlp=mlp)


def _bare(layer):
    return dict(layer, mlp=None)


# every mixer once, sizes that differ everywhere; latent vectors the mma.sync kernels take (48 wide),
# expanded keys of 32 with values of 24; a layer without a feed-forward
PIK_A = {
    "architecture": "Pikavik", "vocab": 97, "width": 64, "norm": {"eps": 1e-6},
    "layers": [_moe(_wkv(3, 12, 5), 6, 2, 3, 2, 1.5, 24, 0.9, (40, 1.2)),
               _moe(_latent(3, 16, 16, 24, 32, 24, 0.3, 10000.0), 8, 3, 2, 1, 0.8, 16, 1.4, (8, 0.7)),
               _bare(_mlstm(2, 16, 20, 9.0)),
               _moe(_wkv(2, 32, 16), 5, 2, None, None, 1.0, 20, 2.0, None)],
}
# a width the tensor-core product does not take; latent vectors that are no multiple of 8 (the generic
# attention kernel), a rotation of part of the rotated dimensions; groups of one expert; no shared expert
PIK_B = {
    "architecture": "Pikavik", "vocab": 131, "width": 100, "norm": {"eps": 1e-5},
    "layers": [_moe(_latent(5, 10, 6, 14, 21, 17, 0.35, 500.0, 4), 4, 2, 4, 3, 2.2, 28, 1.1, (12, 1.6)),
               _moe(_mlstm(5, 10, 7, 4.0), 3, 1, 1, 1, 1.7, 36, 0.8, None),
               _bare(_wkv(5, 10, 3)),
               _moe(_mlstm(1, 40, 33, 20.0), 9, 4, 3, 2, 1.0, 20, 1.0, (36, 0.5))],
}
# latent vectors of 224 numbers (the kernel for wide vectors), expanded keys and values of 128 (the
# tensor-memory kernel); keys of 128 and 64 in the recurrences
PIK_C = {
    "architecture": "Pikavik", "vocab": 211, "width": 256, "norm": {"eps": 1e-5},
    "layers": [_moe(_mlstm(2, 128, 96, 15.0), 16, 4, 8, 3, 2.5, 64, 1.5, (128, 1.0)),
               _moe(_latent(4, 64, 64, 128, 160, 72, 0.09, 300000.0), 12, 3, 4, 2, 1.25, 40, 0.7, (56, 1.9)),
               _bare(_wkv(4, 64, 24)),
               _moe(_latent(2, 96, 48, 64, 304, 40, 0.08, 20000.0), 8, 2, 2, 2, 1.0, 96, 1.0, (64, 1.0))],
}
# keys wider than 128 in the recurrences; 20 heads on one latent vector of 136; two layers of a kind in a row
PIK_D = {
    "architecture": "Pikavik", "vocab": 173, "width": 128, "norm": {"eps": 1e-6},
    "layers": [_bare(_latent(20, 8, 24, 16, 112, 64, 0.2, 1000.0)),
               _moe(_wkv(1, 160, 32), 10, 5, 5, 4, 3.0, 48, 3.0, (24, 0.4)),
               _moe(_mlstm(1, 200, 16, 12.0), 4, 1, 2, 1, 0.5, 56, 1.0, (72, 2.5)),
               _bare(_mlstm(3, 24, 48, 6.0))],
}
CASES = {"A": (PIK_A, 61), "B": (PIK_B, 62), "C": (PIK_C, 63), "D": (PIK_D, 64)}


def loud_weights(folder: str, seed: int) -> None:
    """Rewrites the small learned tensors of a folder so that every one of them matters: routers that
    decide, decays from fast to slow, bonuses, mixes with the token before, gates that open and close,
    sinks, norm weights and layer scales away from their neutral values."""
    from minfer_b200.weights.safetensors_io import load_all, save_file
    w = load_all(folder)
    gen = torch.Generator().manual_seed(seed)

    def rnd(shape, mean, std):
        return torch.randn(shape, generator=gen) * std + mean

    for name in sorted(w):
        t = w[name]
        width = t.shape[-1]
        if name.endswith("mlp.router"):
            new = rnd(t.shape, 0.0, 1.5 * width ** -0.5)
        elif name.endswith("shared.sg"):
            new = rnd(t.shape, 0.0, 1.0 * width ** -0.5)
        elif ".mu." in name:
            new = torch.rand(t.shape, generator=gen)
        elif name.endswith("mix.w1"):
            new = rnd(t.shape, 0.0, 1.0 * width ** -0.5)
        elif name.endswith("mix.w2"):
            new = rnd(t.shape, 0.0, 0.7 * width ** -0.5)
        elif name.endswith("mix.w0"):
            new = rnd(t.shape, -2.5, 1.5)
        elif name.endswith("mix.u"):
            new = rnd(t.shape, 0.3, 0.6)
        elif name.endswith((".mix.i", ".mix.f")):
            new = rnd(t.shape, 0.0, 1.5 * width ** -0.5)
        elif name.endswith("mix.i.b"):
            new = rnd(t.shape, 0.0, 1.0)
        elif name.endswith("mix.f.b"):
            new = rnd(t.shape, 3.0, 2.0)
        elif name.endswith("sink"):
            new = rnd(t.shape, 0.5, 1.0)
        elif name.endswith(("mix.norm", "dq.norm", "dkv.norm")):
            new = rnd(t.shape, 1.0, 0.2)
        elif name.endswith(("norm1", "final.norm")):
            new = rnd(t.shape, 0.0, 0.2)
        elif name.endswith((".ls1", ".ls2")):
            new = rnd(t.shape, 0.9, 0.3)
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
    folder = tempfile.mkdtemp(prefix=f"minfer_b200_pik{name}_")
    write_random_model(folder, cfg, seed, store, weight_std=0.08)
    loud_weights(folder, seed)
    return folder
