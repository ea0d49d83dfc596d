"""Random Pazatar configurations (sizes, order of layers, loops, masks, constants drawn from a seed): the
engine against the plain implementation, whole prompts, a batch of two, the last tokens one by one and
portions of a random size, in both precisions."""
import random

import pytest
import torch

import plain_pazatar as P
from helpers import ROW_RMS_TOL, random_ids
from pazatar_cases import make_folder
from test_pazatar_engine_gpu import _close as _close_rows

pytestmark = pytest.mark.gpu


def _close(got, want, dtype):
    """The bounds of the engine tests, wider where the drawn sizes leave a norm a handful of numbers."""
    _close_rows(got, want, dtype, float32_bound=5e-5, bf16_bound=3 * ROW_RMS_TOL, few=0.1)


def make(rng):
    """A configuration drawn from ``rng``: 1 to 5 layers of either kind in any order, sizes that are
    multiples of nothing, with or without every optional key."""
    width = rng.choice([40, 48, 64, 96, 100, 128, 160, 192, 256, 320])

    def attention(dims_of):
        kv = rng.choice([1, 1, 2, 3])
        dim = rng.choice([8, 10, 16, 24, 32, 48, 64, 80, 96, 128, 136])
        m = {"heads": kv * rng.choice([1, 2, 3, 4, 17]), "kv_heads": kv, "dim": dim,
             "scale": rng.choice([dim ** -0.5, 0.125, 0.25])}
        if rng.random() < 0.85:
            m["mask"] = {"size": rng.choice([1, 3, 16, 20, 33, 63, 64, 65, 100, 128, 150])}
        if rng.random() < 0.85:
            m["rot"] = {"base": rng.choice([1e2, 1e3, 1e4, 5e5]), "dims": rng.choice([dim, dim, 2 * rng.randint(1, dim // 2)])}
            if rng.random() < 0.8:
                m["rot"]["scaling"] = dims_of()
        return m

    def yarn():
        return {"factor": rng.choice([1.5, 4.0, 32.0]), "original": rng.choice([32, 100, 4096]),
                "fast": rng.choice([32.0, 4.0]), "slow": rng.choice([1.0, 0.5])}

    def bands():
        low = rng.choice([1.0, 0.5, 2.0])
        return {"factor": rng.choice([2.0, 8.0]), "original": rng.choice([32, 100, 8192]), "low": low,
                "high": low * rng.choice([1.5, 4.0])}

    layers = []
    for _ in range(rng.randint(1, 5)):
        if rng.random() < 0.5:
            m = attention(yarn)
            m["vdim"] = m["dim"]
            layer = {"type": "attention", "mixer": m}
        else:
            left = attention(bands)
            left["vdim"] = rng.choice([left["dim"], left["dim"], 8, 12, 40, 64, 128])
            left["softcap"] = rng.choice([1.0, 5.0, 30.0])
            taps = rng.choice([0, 1, 2, 3, 4, 7, 8])
            if taps:
                left["conv"] = taps
            right = {"heads": rng.choice([1, 2, 3, 5, 8]), "dim": rng.choice([8, 10, 16, 32, 48, 64, 96, 128, 132]),
                     "vdim": rng.choice([8, 9, 16, 40, 64, 128]), "tau": rng.choice([1.0, 4.0, 16.0, 30.0]),
                     "decay_rank": rng.choice([1, 3, 8, 16, 40])}
            layer = {"type": "parallel", "mixer": {"left": left, "right": right}}
        layer["mlp"] = {"kind": "dense", "ff": rng.choice([8, 36, 64, 100, 256])} if rng.random() < 0.85 else None
        layers.append(layer)
    loop = None
    if rng.random() < 0.6:
        start = rng.randrange(len(layers))
        loop = {"start": start, "stop": rng.randint(start + 1, len(layers)), "times": rng.randint(1, 3)}
    return {"architecture": "Pazatar", "vocab": rng.randint(50, 700), "width": width,
            "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers, "loop": loop}


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11, 12])
def test_random_configuration(seed):
    check(seed)


def check(seed):
    from minfer_b200.engine.step import Engine
    from minfer_b200.model import Model
    rng = random.Random(seed)
    cfg = make(rng)
    folder = make_folder("r", "bfloat16", cfg, seed)
    c, w = P.load_folder(folder)
    n = rng.choice([5, 37, 70, 130, 210])
    ids = random_ids(n, cfg["vocab"], seed)
    ids2 = random_ids(rng.randint(1, 60), cfg["vocab"], seed + 1000)
    cut = max(1, n - rng.randint(1, 24))
    portion = rng.choice([2, 3, 50, 64, 170])
    want, want2 = P.forward(c, w, ids), P.forward(c, w, ids2)
    for dtype in ("float32", "bfloat16"):
        eng = Engine(Model.from_folder(folder, dtype, "cuda:0"), max_tokens=2048)
        s = eng.acquire()
        got = eng.step([s], [ids], [list(range(n))])
        eng.release(s)
        _close(got, want, dtype)
        a, b = eng.acquire(), eng.acquire()
        out = eng.step([a, b], [ids[:cut], ids2], [list(range(cut)), list(range(len(ids2)))])
        _close(out[cut:], want2, dtype)
        eng.release(b)
        rows = [out[:cut]] + [eng.step([a], [[ids[t]]], [[0]]) for t in range(cut, n)]
        eng.release(a)
        _close(torch.cat(rows), want, dtype)
        s = eng.acquire()
        rows = []
        for lo in range(0, n, portion):
            part = ids[lo:lo + portion]
            rows.append(eng.step([s], [part], [list(range(len(part)))]))
        eng.release(s)
        _close(torch.cat(rows), want, dtype)
        eng.check_status()
        eng.cache.check_canaries()
