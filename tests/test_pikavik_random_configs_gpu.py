"""Random Pikavik configurations (sizes, order of layers, groups, routers, constants drawn from a
seed): the engine against the plain implementation, whole prompts, a batch of two, the last tokens
one by one and portions of a random size, in both precisions."""
import random

import pytest
import torch

import plain_pikavik as P
from helpers import random_ids
from test_pikavik_engine_gpu import LEAST_MARGIN, Plain
from test_pikavik_engine_gpu import _close as _close_rows
from pikavik_cases import make_folder

pytestmark = pytest.mark.gpu


def _close(got, want, dtype):
    """The bounds of the engine tests, wider where the drawn sizes leave a norm or a normalizer a
    handful of numbers that may nearly cancel."""
    _close_rows(got, want, dtype, float32_bound=1e-4, few=0.2)


def make(rng):
    """A configuration drawn from ``rng``: 1 to 6 layers of any kind in any order, sizes that are
    multiples of nothing, with or without every optional key."""
    width = rng.choice([40, 48, 64, 96, 100, 128, 160, 192, 256, 320])
    layers = []
    for _ in range(rng.randint(1, 6)):
        kind = rng.choice(["wkv", "mlstm", "latent_attention"])
        heads = rng.choice([1, 2, 3, 4, 5, 8])
        if kind == "wkv":
            m = {"heads": heads, "dim": rng.choice([8, 10, 16, 32, 48, 64, 96, 128, 132]),
                 "decay_rank": rng.choice([1, 3, 8, 16, 40])}
        elif kind == "mlstm":
            dim = rng.choice([8, 10, 16, 32, 64, 96, 128, 132])
            m = {"heads": heads, "dim": dim, "vdim": rng.choice([dim, 8, 9, 16, 40, 64, 128]),
                 "gate_cap": rng.choice([3.0, 8.0, 15.0, 30.0])}
        else:
            rot = rng.choice([2, 8, 8, 16, 32, 64])
            dim = rng.choice([8, 10, 16, 24, 32, 64, 96])
            m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": rng.choice([dim, 8, 12, 32, 64, 128]),
                 "kv_rank": rng.choice([16, 30, 48, 64, 96, 112, 128, 200, 320]), "q_rank": rng.choice([8, 20, 48, 96, 130]),
                 "scale": rng.choice([(dim + rot) ** -0.5, 0.125, 0.25]),
                 "rot": {"base": rng.choice([1e3, 1e4, 5e5]), "dims": rng.choice([rot, rot, 2 * rng.randint(1, rot // 2)])}}
        layer = {"type": kind, "mixer": m, "mlp": None}
        if rng.random() < 0.85:
            count = rng.choice([1, 1, 2, 3, 4])
            size = rng.randint(1, 5)
            keep = rng.randint(1, count)
            router = {"experts": count * size, "top": rng.randint(1, min(8, keep * size)),
                      "scale": rng.choice([0.5, 1.0, 1.5, 2.5])}
            if count > 1 or rng.random() < 0.5:
                router["groups"] = {"count": count, "keep": keep}
            layer["mlp"] = {"kind": "moe", "expert": {"ff": rng.choice([8, 16, 24, 36, 64, 96]), "limit": rng.choice([0.7, 1.5, 4.0])},
                            "router": router,
                            "shared": rng.choice([None, {"ff": rng.choice([8, 40, 128]), "limit": rng.choice([0.9, 2.0])}])}
        layers.append(layer)
    return {"architecture": "Pikavik", "vocab": rng.randint(50, 700), "width": width,
            "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10])
def test_random_configuration(seed):
    from minfer_b200.engine.step import Engine
    from minfer_b200.model import Model
    rng = random.Random(seed)
    cfg = make(rng)
    folder = make_folder("r", "bfloat16", cfg, seed)
    c, w = P.load_folder(folder)
    n = rng.choice([1, 5, 37, 70, 130, 210])
    ids = random_ids(n, cfg["vocab"], seed)
    ids2 = random_ids(rng.randint(1, 60), cfg["vocab"], seed + 1000)
    cut = max(1, n - rng.randint(1, 24))
    portion = rng.choice([2, 3, 50, 64, 170])
    for dtype in ("float32", "bfloat16"):
        want = Plain(*P.forward_marked(c, w, ids, LEAST_MARGIN[dtype]))
        want2 = Plain(*P.forward_marked(c, w, ids2, LEAST_MARGIN[dtype]))
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
