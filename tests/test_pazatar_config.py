"""The Pazatar configuration reader, its lowering to a plan, the rotations' tables and the plain
implementation's own mechanisms (no GPU)."""
import copy
import math

import pytest
import torch

import plain_pazatar as P
from pazatar_cases import CASES, PAZ_A, PAZ_B, PAZ_C
from minfer_b200.config.base import ConfigError
from minfer_b200.model import Model
from minfer_b200.parts.rotary import Rotary
from minfer_b200.registry import read_config


def test_reads_every_size_and_constant():
    cfg = read_config(PAZ_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.loop) == (97, 64, 1e-6, (1, 3, 3))
    plan = cfg.plan()
    assert plan.head_name is None and plan.after_embedding is None and plan.on_logits is None
    assert [l.mixer.kind for l in plan.layers] == ["parallel", "qk_norm_attention", "parallel", "qk_norm_attention"]
    assert all(l.block.kind == "sandwich_norm" for l in plan.layers)
    par = plan.layers[0].mixer.params
    assert (par["norms"]["mult"], par["norms"]["eps"], par["norms"]["width"]) == (0.5, 1e-6, 64)
    left, right = par["left"].params, par["right"].params
    assert (left["n_heads"], left["n_kv_heads"], left["head_dim"], left["value_dim"]) == (4, 2, 16, 24)
    assert (left["scale"], left["softcap"], left["conv"], left["chunk"]) == (0.4, 5.0, 4, 20)
    assert left["sink"] and left["norm_scope"] == "head" and not left["bias"]
    rot = left["position"].params
    assert (rot["rotary_dim"], rot["theta"], rot["style"]) == (8, 1000.0, "neox")
    assert rot["scaling"] == {"factor": 3.0, "original": 40.0, "low": 1.0, "high": 6.0}
    assert (right["n_heads"], right["head_dim"], right["value_dim"], right["tau"], right["rank"]) == (3, 12, 20, 4.0, 5)
    att = plan.layers[1].mixer.params
    assert (att["n_heads"], att["n_kv_heads"], att["head_dim"], att["chunk"], att["scale"]) == (3, 1, 24, 33, 0.3)
    assert att["values"] == "keys" and att["norm_scope"] == "all" and att["softcap"] == 0.0 and not att.get("sink")
    rot = att["position"].params
    assert (rot["rotary_dim"], rot["style"]) == (16, "interleaved")
    assert rot["scaling"] == {"factor": 1.5, "original": 30.0, "fast": 4.0, "slow": 0.5}
    assert "scaling" not in plan.layers[3].mixer.params["position"].params
    ff = plan.layers[0].feed_forward.params
    assert (ff["intermediate_size"], ff["activation"]) == (80, "relu2") and plan.layers[2].feed_forward is None
    assert read_config(cfg.to_dict()) == cfg


def test_run_order_of_the_loop():
    plan = read_config(PAZ_A).plan()
    assert [(c.layer, c.cache, c.pass_start) for c in plan.schedule] == [
        (0, 0, None), (1, 1, 0), (2, 2, None), (1, 3, 1), (2, 4, None), (1, 5, 2), (2, 6, None), (3, 7, None)]
    assert plan.pass_injection.params["add_embedding"] is False and plan.pass_injection.params["passes"] == 3
    assert [(c.layer, c.pass_start) for c in plan.schedule] == P.run_order(PAZ_A)
    plan = read_config(PAZ_B).plan()
    assert plan.pass_injection is None and [c.layer for c in plan.schedule] == [0, 1, 2, 3]


def test_defaults_and_absent_keys():
    plan = read_config(PAZ_B).plan()
    assert plan.layers[1].mixer.params["left"].params["conv"] == 1
    last = plan.layers[3].mixer.params["left"].params
    assert last["conv"] == 0 and last["position"] is None
    assert plan.layers[2].mixer.params["chunk"] == 0 and plan.layers[2].mixer.params["position"] is None
    c = copy.deepcopy(PAZ_A)
    for m in (c["layers"][1]["mixer"], c["layers"][2]["mixer"]["left"], c["layers"][2]["mixer"]["right"]):
        del m["vdim"]
    del c["layers"][2]["mixer"]["left"]["softcap"]
    del c["loop"]
    plan = read_config(c).plan()
    left = plan.layers[2].mixer.params["left"].params
    assert (left["value_dim"], left["softcap"]) == (40, 0.0)
    assert plan.layers[2].mixer.params["right"].params["value_dim"] == 16 and plan.pass_injection is None


def test_the_decay_rank_comes_from_the_checkpoint():
    c = copy.deepcopy(PAZ_A)
    for layer in c["layers"]:
        if layer["type"] == "parallel":
            del layer["mixer"]["right"]["decay_rank"]
    cfg = read_config(c).with_tensor_shapes({"l0.mix.right.a1": (7, 64), "l2.mix.right.a1": (11, 64)})
    assert [cfg.plan().layers[i].mixer.params["right"].params["rank"] for i in (0, 2)] == [7, 11]


def test_tensor_names_and_shapes():
    cfg = read_config(PAZ_A)
    model = Model(cfg.plan(), "float32", cfg)
    specs = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    for n, shape in {"embed": (97, 64), "loop.step": (3, 64), "final.norm": (64,), "l0.norm1": (64,), "l0.norm1b": (64,),
                     "l0.norm2": (64,), "l0.norm2b": (64,), "l0.mix.left.q": (64, 64), "l0.mix.left.k": (32, 64),
                     "l0.mix.left.v": (48, 64), "l0.mix.left.q.conv": (64, 4), "l0.mix.left.v.conv": (48, 4),
                     "l0.mix.left.q.norm": (16,), "l0.mix.left.k.norm": (16,), "l0.mix.left.o": (64, 96),
                     "l0.mix.right.q": (36, 64), "l0.mix.right.v": (60, 64), "l0.mix.right.g": (60, 64),
                     "l0.mix.right.a1": (5, 64), "l0.mix.right.a2": (36, 5), "l0.mix.right.a2.b": (36,),
                     "l0.mix.right.norm": (20,), "l0.mix.right.o": (64, 60), "l0.mix.left.out": (64,),
                     "l0.mix.right.out": (64,), "l0.mlp.up": (80, 64), "l0.mlp.down": (64, 80),
                     "l1.mix.q": (72, 64), "l1.mix.k": (24, 64), "l1.mix.q.norm": (72,), "l1.mix.k.norm": (24,),
                     "l1.mix.o": (64, 72)}.items():
        assert specs[n] == shape, n
    for absent in ("head", "l1.mix.v", "l1.mix.q.b", "l1.mix.q.conv", "l2.norm2", "l2.norm2b", "l2.mlp.up", "embed.norm"):
        assert absent not in specs, absent
    assert "l2.norm2b" in model.ignorable_tensors()


@pytest.mark.parametrize("change,where", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("low"), "low"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=20), "vdim"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_refusals(change, where):
    cfg = copy.deepcopy(PAZ_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        read_config(cfg)
    assert where in str(e.value)


def test_every_case_reads_and_builds():
    for c, _ in CASES.values():
        cfg = read_config(c)
        assert len(Model(cfg.plan(), "bfloat16", cfg).blocks) == len(c["layers"])


# ---- the rotations' tables, and the plain implementation's own mechanisms ----------------------
@pytest.mark.parametrize("dims,base,bands", [(8, 1e3, (3.0, 40, 1.0, 6.0)), (64, 5e5, (8.0, 8192, 1.0, 4.0)),
                                             (10, 100.0, (2.0, 30, 2.0, 2.5)), (2, 1e4, (4.0, 3, 1.0, 4.0))])
def test_banded_frequencies(dims, base, bands):
    sc = dict(zip(("factor", "original", "low", "high"), bands))
    part = Rotary(dims, dims, base, scaling=sc)
    assert part.magnitude() == 1.0
    want = torch.tensor(P.banded_frequencies(dims, base, sc), dtype=torch.float64)
    assert torch.allclose(part.inverse_frequencies(), want, rtol=1e-14, atol=0)
    plain = torch.tensor(P.plain_frequencies(dims, base), dtype=torch.float64)
    assert torch.all(want <= plain * (1 + 1e-12)) and torch.all(want >= plain / bands[0] * (1 - 1e-12))


def test_bands_keep_short_waves_and_slow_long_ones():
    sc = {"factor": 4.0, "original": 64, "low": 1.0, "high": 4.0}
    f = P.plain_frequencies(16, 1e4)
    got = P.banded_frequencies(16, 1e4, sc)
    waves = [2 * math.pi / x for x in f]
    kinds = {"short": 0, "long": 0, "between": 0}
    for x, y, w in zip(f, got, waves):
        if w < 16:
            assert y == x
            kinds["short"] += 1
        elif w > 64:
            assert y == x / 4
            kinds["long"] += 1
        else:
            assert x / 4 < y < x
            kinds["between"] += 1
    assert min(kinds.values()) > 0
    assert sum(kinds.values()) == 8


def test_plain_recurrence_is_a_decayed_sum():
    """o_t = sum_{s <= t} (q_t . prod_{s < i <= t} d_i k_s) v_s."""
    torch.manual_seed(0)
    T, D, Dv = 7, 4, 3
    q, k, v = (torch.randn(T, 1, n).double() for n in (D, D, Dv))
    d = torch.rand(T, 1, D).double()
    want = torch.zeros(T, Dv).double()
    for t in range(T):
        for s in range(t + 1):
            keep = torch.ones(D).double()
            for i in range(s + 1, t + 1):
                keep = keep * d[i, 0]
            want[t] += (q[t, 0] * keep * k[s, 0]).sum() * v[s, 0]
    got, S = P.gla_recurrence(q, k, v, d)
    assert torch.allclose(got[:, 0], want, atol=1e-12)
    head, S1 = P.gla_recurrence(q[:3], k[:3], v[:3], d[:3])
    tail, S2 = P.gla_recurrence(q[3:], k[3:], v[3:], d[3:], S1)
    assert torch.allclose(torch.cat([head, tail]), got, atol=1e-12) and torch.allclose(S2, S, atol=1e-12)


def test_plain_decay_is_a_root_of_the_sigmoid():
    w = {"a1": torch.eye(2).double(), "a2": torch.tensor([[1.0, 0.0], [0.0, -3.0]]).double(), "a2.b": torch.tensor([0.5, 0.0]).double()}
    y = torch.tensor([[1.5, 2.0]]).double()
    got = P.gla_decay(y, w, "", 4.0)
    want = [(1 / (1 + math.exp(-2.0))) ** 0.25, (1 / (1 + math.exp(6.0))) ** 0.25]
    assert torch.allclose(got, torch.tensor([want]).double(), atol=1e-14)


def test_plain_sink_chunk_and_convolution():
    q, k = torch.zeros(5, 1, 2).double(), torch.randn(5, 1, 2).double()
    v = torch.ones(5, 1, 1).double()
    o = P.grouped_attention(q, k, v, 1.0, 3, 2.0, True)[:, 0, 0]
    assert torch.allclose(o, torch.tensor([1 / 2, 2 / 3, 3 / 4, 1 / 2, 2 / 3]).double())
    assert torch.allclose(P.grouped_attention(q, k, v, 1.0, 3, 0.0, False), torch.ones(5, 1, 1).double())
    big = P.grouped_attention(q + 100.0, k * 0 + 100.0, v, 1.0, 0, 2.0, True)[0, 0, 0]      # the score is capped at 2
    assert float(big) == pytest.approx(math.exp(2.0) / (1 + math.exp(2.0)))
    u = torch.tensor([[1.0], [2.0], [4.0]]).double()
    assert P.causal_conv(u, torch.tensor([[10.0, 1.0]]).double()).flatten().tolist() == [1.0, 12.0, 24.0]


def test_plain_side_by_side_is_half_the_sum_of_normed_outputs():
    left, right = torch.tensor([[3.0, 4.0]]).double(), torch.tensor([[30.0, -40.0]]).double()
    one = torch.ones(2).double()
    s = math.sqrt(12.5)
    got = P.side_by_side(left, right, one, 2 * one, 0.0)
    assert torch.allclose(got, torch.tensor([[(3 + 2 * 3) / s / 2, (4 - 2 * 4) / s / 2]]).double())


def test_plain_values_are_the_raw_keys():
    """Scaling k's norm weight changes scores only: with one visible key the output stays."""
    torch.manual_seed(2)
    m = PAZ_C["layers"][2]["mixer"]
    y = torch.randn(1, 8).double()
    w = {"q": torch.randn(128, 8).double(), "k": torch.randn(64, 8).double(), "q.norm": torch.ones(128).double(),
         "k.norm": torch.rand(64).double(), "o": torch.eye(128).double()}
    out = P.attention_mixer(y, w, "", m, 1e-6)
    k = (y @ w["k"].T)
    assert torch.allclose(out, torch.cat([k, k], dim=1), atol=1e-12)
