"""The Pikavik configuration reader, its lowering to a plan and the plain implementation's own
mechanisms (no GPU)."""
import copy
import math

import pytest
import torch

import plain_pikavik as P
from pikavik_cases import CASES, PIK_A, PIK_B
from minfer_b200.config.base import ConfigError
from minfer_b200.model import Model
from minfer_b200.registry import read_config


def test_reads_every_size_and_constant():
    cfg = read_config(PIK_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (97, 64, 1e-6)
    plan = cfg.plan()
    assert [l.mixer.kind for l in plan.layers] == ["wkv", "latent_attention", "mlstm", "wkv"]
    assert all(l.block.kind == "parallel" and l.feed_forward_norm is None for l in plan.layers)
    assert all(l.mixer_norm.params["offset"] == 1.0 for l in plan.layers) and plan.final_norm.params["offset"] == 1.0
    wkv = plan.layers[0].mixer.params
    assert (wkv["n_heads"], wkv["head_dim"], wkv["rank"], wkv["norm_eps"]) == (3, 12, 5, 1e-6)
    att = plan.layers[1].mixer.params
    assert (att["n_heads"], att["head_dim"], att["rot_dim"], att["value_dim"]) == (3, 16, 16, 24)
    assert (att["kv_rank"], att["q_rank"], att["scale"], att["window"]) == (32, 24, 0.3, 0)
    assert att["sink"] and not att["gate"]
    rot = att["position"].params
    assert (rot["head_dim"], rot["rotary_dim"], rot["theta"], rot["style"]) == (16, 16, 10000.0, "neox")
    lstm = plan.layers[2].mixer.params
    assert (lstm["n_heads"], lstm["head_dim"], lstm["value_dim"], lstm["gate_cap"]) == (2, 16, 20, 9.0)
    assert plan.layers[2].feed_forward is None
    moe = plan.layers[1].feed_forward.params
    assert (moe["n_experts"], moe["top"], moe["groups"], moe["keep_groups"]) == (8, 3, 2, 1)
    assert (moe["weight_scale"], moe["intermediate_size"], moe["limit"]) == (0.8, 16, 1.4)
    assert (moe["shared"]["ff"], moe["shared"]["limit"]) == (8, 0.7)
    assert moe["scoring"] == "sigmoid_groups" and moe["activation"] == "clamped_swish"
    assert read_config(cfg.to_dict()) == cfg


def test_defaults_and_absent_keys():
    cfg = read_config(PIK_A)
    moe = cfg.plan().layers[3].feed_forward.params
    assert (moe["groups"], moe["keep_groups"], moe["weight_scale"], moe["shared"]) == (1, 1, 1.0, None)
    assert read_config(PIK_B).plan().layers[0].mixer.params["position"].params["rotary_dim"] == 4
    c = copy.deepcopy(PIK_A)
    del c["layers"][2]["mixer"]["vdim"]
    del c["layers"][1]["mixer"]["rot"]
    plan = read_config(c).plan()
    assert plan.layers[2].mixer.params["value_dim"] == 16 and plan.layers[1].mixer.params["position"] is None


def test_the_decay_rank_comes_from_the_checkpoint():
    c = copy.deepcopy(PIK_A)
    for layer in c["layers"]:
        layer["mixer"].pop("decay_rank", None)
    cfg = read_config(c).with_tensor_shapes({"l0.mix.w1": (7, 64), "l3.mix.w1": (11, 64)})
    assert [l.mixer.params.get("rank") for l in cfg.plan().layers] == [7, None, None, 11]


def test_tensor_names_and_shapes():
    cfg = read_config(PIK_A)
    model = Model(cfg.plan(), "float32", cfg)
    specs = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    for n, shape in {"embed": (97, 64), "head": (97, 64), "final.norm": (64,), "l0.norm1": (64,), "l0.ls1": (64,),
                     "l0.ls2": (64,), "l0.mix.mu.r": (64,), "l0.mix.mu.w": (64,), "l0.mix.r": (36, 64),
                     "l0.mix.g": (36, 64), "l0.mix.w1": (5, 64), "l0.mix.w2": (36, 5), "l0.mix.w0": (36,),
                     "l0.mix.u": (3, 12), "l0.mix.norm": (36,), "l0.mix.o": (64, 36),
                     "l1.mix.dq": (24, 64), "l1.mix.dq.norm": (24,), "l1.mix.uq": (96, 24), "l1.mix.dkv": (48, 64),
                     "l1.mix.dkv.norm": (32,), "l1.mix.uk": (48, 32), "l1.mix.uv": (72, 32), "l1.mix.sink": (3,),
                     "l1.mix.o": (64, 72), "l1.mlp.router": (8, 64), "l1.mlp.e7.gate": (16, 64),
                     "l1.mlp.e0.down": (64, 16), "l1.mlp.shared.up": (8, 64), "l1.mlp.shared.sg": (1, 64),
                     "l2.mix.q": (32, 64), "l2.mix.k": (32, 64), "l2.mix.v": (40, 64), "l2.mix.g": (40, 64),
                     "l2.mix.i": (2, 64), "l2.mix.i.b": (2,), "l2.mix.f": (2, 64), "l2.mix.f.b": (2,),
                     "l2.mix.norm": (40,), "l2.mix.o": (64, 40), "l2.ls1": (64,)}.items():
        assert specs[n] == shape, n
    for absent in ("l1.mix.q", "l1.mix.g", "l1.mlp.e8.gate", "l2.ls2", "l2.mlp.router", "l3.mlp.shared.sg",
                   "l0.norm2", "l0.mlp.correction"):
        assert absent not in specs, absent
    assert "l2.ls2" in model.ignorable_tensors()


@pytest.mark.parametrize("change,where", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][0].pop("mixer"), "mixer"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), "heads"),
    (lambda c: c["layers"][2]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][2]["mixer"].update(gate_cap=-1.0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=3), "groups"),
    (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_refusals(change, where):
    cfg = copy.deepcopy(PIK_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        read_config(cfg)
    assert where in str(e.value)


def test_every_case_reads_and_builds():
    for c, _ in CASES.values():
        cfg = read_config(c)
        assert len(Model(cfg.plan(), "bfloat16", cfg).blocks) == len(c["layers"])


# ---- the plain implementation's own mechanisms, against closed forms ---------------------------
def test_plain_wkv_is_a_decayed_sum_with_a_bonus():
    """o_t = sum_{s < t} (r_t . prod_{s < i < t} d_i k_s) v_s + (r_t . u k_t) v_t."""
    torch.manual_seed(0)
    T, D, Dv = 7, 4, 3
    r, k, v = torch.randn(T, 1, D).double(), torch.randn(T, 1, D).double(), torch.randn(T, 1, Dv).double()
    d, u = torch.rand(T, 1, D).double(), torch.randn(1, D).double()
    want = torch.zeros(T, Dv).double()
    for t in range(T):
        want[t] = (r[t, 0] * u[0] * k[t, 0]).sum() * v[t, 0]
        for s in range(t):
            keep = torch.ones(D).double()
            for i in range(s + 1, t):
                keep = keep * d[i, 0]
            want[t] += (r[t, 0] * keep * k[s, 0]).sum() * v[s, 0]
    got, S = P.wkv_recurrence(r, k, v, d, u)
    assert torch.allclose(got[:, 0], want, atol=1e-12)
    head, S1 = P.wkv_recurrence(r[:3], k[:3], v[:3], d[:3], u)
    tail, S2 = P.wkv_recurrence(r[3:], k[3:], v[3:], d[3:], u, S1)
    assert torch.allclose(torch.cat([head, tail]), got, atol=1e-12) and torch.allclose(S2, S, atol=1e-12)


def test_plain_mlstm_without_the_maximum():
    """The running maximum only keeps numbers in range: with plain exponentials,
    o = sum_s w_ts (q . k_s) v_s / (max(|sum_s w_ts q . k_s|, 1) + 1e-6 e^m), w_ts = exp(i_s + sum_{r > s} f_r)."""
    torch.manual_seed(1)
    T, D, Dv = 8, 3, 4
    q, k, v = (torch.randn(T, 1, n).double() for n in (D, D, Dv))
    i, f = torch.randn(T, 1).double() * 2, -torch.rand(T, 1).double()
    got, (_, _, m) = P.mlstm_recurrence(q, k, v, i, f)
    run = 0.0
    for t in range(T):
        run = max(run + float(f[t]), float(i[t]))
        num, den = torch.zeros(Dv).double(), 0.0
        for s in range(t + 1):
            w = math.exp(float(i[s]) + float(f[s + 1:t + 1].sum())) * float(q[t, 0] @ k[s, 0])
            num, den = num + w * v[s, 0], den + w
        assert torch.allclose(got[t, 0], num / (max(abs(den), 1.0) + 1e-6 * math.exp(run)), atol=1e-12)
    assert float(m[0]) == pytest.approx(run)


def test_plain_mlstm_maximum_starts_at_zero():
    """With closed input gates and open forget gates the maximum stays near 0, and the small normalizer
    is bounded from below by e^(-m) = 1: from minus infinity it would not be."""
    q = k = torch.full((1, 1, 1), 0.1).double()
    v = torch.ones(1, 1, 1).double()
    got, (_, _, m) = P.mlstm_recurrence(q, k, v, torch.full((1, 1), -8.0).double(), torch.full((1, 1), -1e-9).double())
    assert float(m) == pytest.approx(-1e-9)
    assert float(got) == pytest.approx(0.01 * math.exp(-8.0), rel=1e-5)


def test_plain_sink_takes_its_share():
    q = torch.zeros(3, 1, 2).double()
    k, v = torch.randn(3, 1, 2).double(), torch.ones(3, 1, 1).double()
    o = P.sink_attention(q, k, v, 5.0, torch.tensor([math.log(2.0)]).double())
    assert torch.allclose(o[:, 0, 0], torch.tensor([1 / 3, 2 / 4, 3 / 5]).double())


def test_plain_router_chooses_within_the_best_groups():
    logit = lambda p: math.log(p / (1 - p))
    # groups (0.9, 0.1), (0.6, 0.55), (0.8, 0.3): sums 1.0, 1.15, 1.1
    z = torch.tensor([[logit(p) for p in (0.9, 0.1, 0.6, 0.55, 0.8, 0.3)]]).double()
    chosen, weight, _ = P.choose(z, 2, 3, 2, 2.0)
    assert chosen.tolist() == [[4, 2]]                                  # expert 0's group is left out
    assert torch.allclose(weight, torch.tensor([[0.8, 0.6]]).double() / 1.4 * 2.0)
    chosen, weight, _ = P.choose(z, 2, 1, 1, 1.0)
    assert chosen.tolist() == [[0, 4]]
    # groups of three count their two largest only: (0.5, 0.4, 0.39) against (0.6, 0.35, 0.1)
    z = torch.tensor([[logit(p) for p in (0.5, 0.4, 0.39, 0.6, 0.35, 0.1)]]).double()
    assert P.choose(z, 1, 2, 1, 1.0)[0].tolist() == [[3]]


def test_plain_rotation_is_relative():
    torch.manual_seed(1)
    q, k = torch.randn(1, 1, 8).double(), torch.randn(1, 1, 8).double()
    rq, rk = P.rotate_half(q.repeat(20, 1, 1), 6, 100.0), P.rotate_half(k.repeat(20, 1, 1), 6, 100.0)
    assert abs(float(rq[7, 0] @ rk[3, 0]) - float(rq[19, 0] @ rk[15, 0])) < 1e-12
    assert torch.equal(rq[..., 6:], q.repeat(20, 1, 1)[..., 6:])
    ang = 5 * 100.0 ** (-2.0 / 6)                                       # pair (1, 4) at position 5
    assert abs(float(rq[5, 0, 1]) - (float(q[0, 0, 1]) * math.cos(ang) - float(q[0, 0, 4]) * math.sin(ang))) < 1e-12
