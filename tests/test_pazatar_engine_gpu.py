"""Pazatar through the engine against the plain implementation, in float32 and bfloat16: whole prompts
and the stream after every layer run; the last tokens one by one; every token a step from the first;
prompts in portions down to two tokens; batches of unequal requests against each alone, one batch after
another so that slots, pages and states are used again; a mixed step; long decoding; models of one kind
of layer, of sizes that are 1, with loops of every form; greedy generation through the generator, the
command line and the trace replay."""
import copy
import json
import os
import subprocess
import sys
import tempfile

import numpy as np
import pytest
import torch

import plain_pazatar as P
from helpers import ROW_RMS_TOL, TOL, random_ids
from pazatar_cases import PAZ_A, PAZ_B, PAZ_C, PAZ_D, make_folder

pytestmark = pytest.mark.gpu

LENGTHS = [37, 5, 131, 64, 1, 65, 11]
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module", params=["A", "B", "C", "D"])
def case(request):
    folder = make_folder(request.param)
    cfg, w = P.load_folder(folder)
    prompts = [random_ids(n, cfg["vocab"], 900 + i) for i, n in enumerate(LENGTHS)]
    return {"name": request.param, "folder": folder, "cfg": cfg, "w": w, "prompts": prompts,
            "plain": [P.forward(cfg, w, ids) for ids in prompts]}


def _engine(folder, dtype, max_tokens=4096, **kw):
    from minfer_b200.engine.step import Engine
    from minfer_b200.model import Model
    return Engine(Model.from_folder(folder, dtype, "cuda:0"), max_tokens=max_tokens, **kw)


def _close(got, want, dtype, float32_bound=3e-5, bf16_bound=2 * ROW_RMS_TOL, few=0.03):
    """Row by row: within the bound (bfloat16: of its root mean square), but for a few rows up to 8 times that:
    a recurrent head's output is divided by its root mean square, so where q . k nearly cancels (at a
    sequence's first token o = (q . k) v, of which the norm leaves a sign) a token has its rounding errors
    scaled up.  A fault of the cache, a state or the batch moves every later row by tens of per cent."""
    g = got.detach().to(torch.float64).cpu()
    assert g.shape == want.shape
    top = max(1e-30, float(want.abs().max()))
    if dtype == "float32":
        err, bound = (g - want).abs().max(dim=-1).values / top, float32_bound
    else:
        err, bound = (g - want).pow(2).mean(dim=-1).sqrt() / top, bf16_bound
    if 0 < int((err >= bound).sum()) <= max(3, int(few * len(err))):
        bound *= 8
    assert float(err.max()) < bound, (int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_and_every_layer(case, dtype):
    eng = _engine(case["folder"], dtype)
    for ids, want in zip(case["prompts"], case["plain"]):
        s = eng.acquire()
        got = eng.step([s], [ids], [list(range(len(ids)))])
        eng.release(s)
        _close(got, want, dtype)
    ids = case["prompts"][2]
    taps, seen = [], []
    P.forward(case["cfg"], case["w"], ids, taps)
    eng.layer_tap = lambda i, h: seen.append(h.detach().cpu().to(torch.float64))
    s = eng.acquire()
    eng.step([s], [ids], [list(range(len(ids)))])
    eng.release(s)
    eng.layer_tap = None
    assert len(seen) == len(taps)
    for got, want in zip(seen, taps):
        rows = (got - want).abs().max(dim=-1).values / float(want.abs().max())
        assert float(rows.median()) < (1e-5 if dtype == "float32" else 2e-2)
        assert float(rows.max()) < (2e-4 if dtype == "float32" else 0.4)
    eng.check_status()
    eng.cache.check_canaries()


@pytest.mark.parametrize("dtype", DTYPES)
def test_last_tokens_one_by_one(case, dtype):
    eng = _engine(case["folder"], dtype)
    for ids, want in zip(case["prompts"], case["plain"]):
        n = len(ids)
        head = max(1, n - 40)
        s = eng.acquire()
        rows = [eng.step([s], [ids[:head]], [list(range(head))])]
        for t in range(head, n):
            rows.append(eng.step([s], [[ids[t]]], [[0]]))
        eng.release(s)
        _close(torch.cat(rows), want, dtype)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_token_by_token_from_the_first(case, dtype):
    """Every token a step of its own, from position 0: the first tokens see the zeros before the sequence
    in the convolutions, empty states, and nothing but themselves (and the sink) in attention."""
    eng = _engine(case["folder"], dtype)
    ids, want = case["prompts"][0], case["plain"][0]
    s = eng.acquire()
    rows = [eng.step([s], [[t]], [[0]]) for t in ids]
    eng.release(s)
    _close(torch.cat(rows), want, dtype)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [2, 3, 7, 16, 17, 20, 33, 63, 64, 65])
def test_prompts_in_portions(case, dtype, portion):
    """Portions around the recurrence's chunks of 16 tokens, the attention's chunks and a page of 64."""
    eng = _engine(case["folder"], dtype)
    for ids, want in zip(case["prompts"][:4], case["plain"][:4]):
        s = eng.acquire()
        rows = []
        for lo in range(0, len(ids), portion):
            part = ids[lo:lo + portion]
            rows.append(eng.step([s], [part], [list(range(len(part)))]))
        eng.release(s)
        _close(torch.cat(rows), want, dtype)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batches_slots_reused(case, dtype):
    """The prompts' first parts in one step, then one token each; a request that runs out of tokens leaves
    the batch; the next batch starts in the slots, pages and states the first one gave back.  Every
    request's logits equal those it has alone."""
    eng = _engine(case["folder"], dtype, max_tokens=1024, max_seqs=4)
    prompts, plain = case["prompts"], case["plain"]
    for batch in ([0, 1, 2], [3, 4, 5, 6], [2, 0], [6, 2, 4]):
        slots = {r: eng.acquire() for r in batch}
        heads = {r: max(1, len(prompts[r]) - 9) for r in batch}
        got = {r: [] for r in batch}
        out = eng.step([slots[r] for r in batch], [prompts[r][:heads[r]] for r in batch],
                       [list(range(heads[r])) for r in batch])
        at = 0
        for r in batch:
            got[r].append(out[at:at + heads[r]])
            at += heads[r]
        pos = dict(heads)
        live = [r for r in batch if pos[r] < len(prompts[r])]
        while live:
            out = eng.step([slots[r] for r in live], [[prompts[r][pos[r]]] for r in live], [[0]] * len(live))
            for i, r in enumerate(live):
                got[r].append(out[i:i + 1])
                pos[r] += 1
            live = [r for r in live if pos[r] < len(prompts[r])]
        for r in batch:
            _close(torch.cat(got[r]), plain[r], dtype)
            eng.release(slots[r])
    eng.check_status()
    eng.cache.check_canaries()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_stale_slot_does_not_leak_into_the_next_request(case, dtype):
    """A long request fills a slot's recurrent states, last projections and pages; the slot is given back
    and the next, short request in it must start from nothing."""
    eng = _engine(case["folder"], dtype, max_tokens=512, max_seqs=1)
    prompts, plain = case["prompts"], case["plain"]
    for r in (2, 1, 4, 0, 4):
        s = eng.acquire()
        got = eng.step([s], [prompts[r]], [list(range(len(prompts[r])))])
        eng.release(s)
        _close(got, plain[r], dtype)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_step_and_wanted_rows_out_of_order(case, dtype):
    """One request goes on by 20 tokens while two others go on by one, in the same step; only some rows are
    wanted, so the last layer's feed-forward runs on kept rows."""
    eng = _engine(case["folder"], dtype)
    prompts, plain = case["prompts"], case["plain"]
    a, b, c = 2, 0, 6
    sa, sb, sc = eng.acquire(), eng.acquire(), eng.acquire()
    eng.step([sa, sb, sc], [prompts[a][:100], prompts[b][:30], prompts[c][:10]], [[], [], []])
    out = eng.step([sb, sa, sc], [[prompts[b][30]], prompts[a][100:120], [prompts[c][10]]], [[0], [19, 3, 7], [0]])
    _close(out[0:1], plain[b][30:31], dtype)
    _close(out[1:4], plain[a][[119, 103, 107]], dtype)      # (rows in the order they were asked for)
    _close(out[4:5], plain[c][10:11], dtype)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_long_decoding(name, dtype):
    """330 tokens: a prompt of 70, then one by one over several pages and chunks, through graphs of growing
    bounds, with the states carried all the way; the same in portions of 50."""
    folder = make_folder(name)
    cfg, w = P.load_folder(folder)
    ids = random_ids(330, cfg["vocab"], 91)
    want = P.forward(cfg, w, ids)
    eng = _engine(folder, dtype, max_tokens=1024)
    s = eng.acquire()
    rows = [eng.step([s], [ids[:70]], [list(range(70))])]
    for t in range(70, 330):
        rows.append(eng.step([s], [[ids[t]]], [[0]]))
    eng.release(s)
    _close(torch.cat(rows), want, dtype)
    assert eng._graphs
    s = eng.acquire()
    rows = []
    for lo in range(0, 330, 50):
        part = ids[lo:lo + 50]
        rows.append(eng.step([s], [part], [list(range(len(part)))]))
    _close(torch.cat(rows), want, dtype)
    eng.check_status()
    eng.cache.check_canaries()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["C", "D"])
def test_a_long_prompt_in_large_portions(name, dtype):
    """430 tokens in portions of 200, 220 and 10: the later portions attend over the cache's pages; then
    the same prompt whole beside a short one."""
    folder = make_folder(name)
    cfg, w = P.load_folder(folder)
    ids = random_ids(430, cfg["vocab"], 17)
    want = P.forward(cfg, w, ids)
    eng = _engine(folder, dtype, max_tokens=2048)
    s = eng.acquire()
    rows, at = [], 0
    for n in (200, 220, 10):
        rows.append(eng.step([s], [ids[at:at + n]], [list(range(n))]))
        at += n
    eng.release(s)
    _close(torch.cat(rows), want, dtype)
    short = random_ids(33, cfg["vocab"], 18)
    a, b = eng.acquire(), eng.acquire()
    out = eng.step([b, a], [short, ids], [[32], [429, 0, 215]])
    _close(out[0:1], P.forward(cfg, w, short)[32:33], dtype)
    _close(out[1:4], want[[429, 0, 215]], dtype)
    eng.check_status()
    eng.cache.check_canaries()


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_key_of_a_chunk_seen_and_not_seen_through_the_engine(dtype):
    """One attention layer whose queries and keys point the same way for one token id: that token's value
    fills the output of every later query of its chunk.  Its place is moved over a chunk's edge, in prompts
    and in decoding: the plain run says which logits follow it and how far the next chunk's are."""
    chunk = 70
    cfg = {"architecture": "Pazatar", "vocab": 60, "width": 64, "norm": {"eps": 1e-6}, "loop": None,
           "layers": [{"type": "attention", "mlp": None,
                       "mixer": {"heads": 2, "kv_heads": 1, "dim": 32, "vdim": 32, "scale": 8.0, "mask": {"size": chunk}}}]}
    folder = make_folder("m", "float32", cfg, 5)
    cfg, w = P.load_folder(folder)
    from minfer_b200.weights.safetensors_io import load_all, save_file
    t = load_all(folder)
    for name in ("embed", "l0.mix.q", "l0.mix.k"):
        t[name] = torch.randn(t[name].shape, generator=torch.Generator().manual_seed(len(name)))
    t["embed"] *= 0.3
    t["embed"][:, 0] = 0.0
    t["embed"][7] = 0.0
    t["embed"][7, 0] = 6.0                                   # token 7 alone lives on dimension 0
    t["embed"][:7, 1], t["embed"][8:, 1] = 4.0, 4.0          # every other token asks along dimension 1
    t["l0.mix.q"][:, 1] = 0.0
    t["l0.mix.q"][0:64:32, 1] = 20.0
    t["l0.mix.k"][:, 0] = 0.0
    t["l0.mix.k"][0, 0] = 20.0
    save_file(t, os.path.join(folder, "model.safetensors"), metadata={"format": "pt"})
    cfg, w = P.load_folder(folder)
    base = [int(x) for x in random_ids(160, 60, 3)]
    base = [x if x != 7 else 8 for x in base]
    eng = _engine(folder, dtype, max_tokens=1024)
    bound = 2 * ROW_RMS_TOL
    for mark in (69, 70, 71, 139, 140):
        ids = list(base)
        ids[mark] = 7
        want, without = P.forward(cfg, w, ids), P.forward(cfg, w, base)
        edge = (mark // chunk + 1) * chunk
        moved = (want - without).pow(2).mean(-1).sqrt() / float(want.abs().max())
        if mark + 1 < min(edge, 160):
            assert float(moved[mark + 1:edge].min()) > 2 * bound          # seen: it shows
        assert float(moved[edge:].max() if edge < 160 else 0.0) < 1e-12    # not seen: it does not
        for cut in (160, mark, mark + 1):
            s = eng.acquire()
            rows = [eng.step([s], [ids[:cut]], [list(range(cut))])]
            rows += [eng.step([s], [[x]], [[0]]) for x in ids[cut:]]
            eng.release(s)
            _close(torch.cat(rows), want, dtype, bf16_bound=bound)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_generator(case, dtype):
    from minfer_b200.engine.generate import Generator
    from minfer_b200.model import Model
    from minfer_b200.sampling.params import SamplingParams
    cfg, w = case["cfg"], case["w"]
    prompts = [case["prompts"][0], case["prompts"][1], case["prompts"][6]]
    gen = Generator(Model.from_folder(case["folder"], dtype, "cuda:0"), max_tokens=2048, max_batch=4)
    got = gen.generate(prompts, 8, SamplingParams.greedy(), stop_token_ids=[])
    for prompt, res in zip(prompts, got):
        assert len(res.tokens) == 8
        ids = list(prompt)
        for tok in res.tokens:             # each token on the prefix the engine itself produced
            logits = P.forward(cfg, w, ids)[-1]
            if dtype == "float32":
                assert tok == int(torch.argmax(logits))
            else:
                slack = 2 * TOL["bfloat16"] * float(logits.abs().max())
                assert float(logits[tok]) >= float(logits.max()) - slack
            ids.append(tok)


def test_command_line_generates(capsys):
    from minfer_b200 import cli
    folder = make_folder("B")
    cfg, w = P.load_folder(folder)
    rc = cli.main([folder, "5,17,3", "--greedy", "--repeat-penalty", "1.0", "-n", "6", "--dtype", "float32",
                   "--stop", "100000"])
    out = capsys.readouterr().out
    assert rc == 0
    want = P.generate_greedy(cfg, w, [5, 17, 3], 6)
    assert " ".join(str(t) for t in want) in out
    assert "Prefill: 3 tokens" in out and "Generated: 6 tokens" in out


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_as_a_process(dtype):
    """``bin/trace_run`` on a folder: two prompts of unequal length in one step, then one request's last
    tokens one by one beside another that ends earlier; logits files against the plain implementation."""
    folder = make_folder("A")
    cfg, w = P.load_folder(folder)
    a, b = random_ids(70, cfg["vocab"], 1), random_ids(9, cfg["vocab"], 2)
    plain = {"a": P.forward(cfg, w, a), "b": P.forward(cfg, w, b)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:60], "want": [0, 59]},
                                     {"id": "b", "tokens": b[:7], "want": [6]}], "end": []}]
    expect = {0: [("a", [0, 59]), ("b", [6])]}
    for i in range(10):
        entries = [{"id": "a", "tokens": [a[60 + i]], "want": [0] if i % 2 == 0 else []}]
        rows = [("a", [60 + i])] if i % 2 == 0 else []
        if i < 2:
            entries.append({"id": "b", "tokens": [b[7 + i]], "want": [0]})
            rows.append(("b", [7 + i]))
        end = (["b"] if i == 1 else []) + (["a"] if i == 9 else [])
        steps.append({"step": i + 1, "entries": entries, "end": end})
        expect[i + 1] = rows
    out = tempfile.mkdtemp()
    root = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..")
    proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder,
                           "--dtype", dtype, "--out", out, "--max-tokens", "128"],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                          text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(11)]
    for step, rows in expect.items():
        path = os.path.join(out, f"{step}.f32")
        if not rows:
            assert not os.path.exists(path)
            continue
        got = torch.from_numpy(np.fromfile(path, dtype="<f4").reshape(-1, cfg["vocab"]))
        _close(got, torch.cat([plain[r][places] for r, places in rows]), dtype)


def _run_cuts(cfg, seed, dtype, n=90):
    folder = make_folder("x", "bfloat16", cfg, seed)
    cfg, w = P.load_folder(folder)
    ids = random_ids(n, cfg["vocab"], 4)
    want = P.forward(cfg, w, ids)
    eng = _engine(folder, dtype, max_tokens=512)
    s = eng.acquire()
    rows = [eng.step([s], [ids[:50]], [list(range(50))])]
    rows.append(eng.step([s], [ids[50:53]], [[0, 1, 2]]))
    for t in range(53, n):
        rows.append(eng.step([s], [[ids[t]]], [[0]]))
    eng.release(s)
    _close(torch.cat(rows), want, dtype, bf16_bound=3 * ROW_RMS_TOL)
    s = eng.acquire()
    _close(eng.step([s], [ids], [[n - 1, 3]]), want[[n - 1, 3]], dtype, bf16_bound=3 * ROW_RMS_TOL)
    eng.release(s)
    eng.check_status()
    return eng


@pytest.mark.parametrize("dtype", DTYPES)
def test_models_of_one_kind_of_layer_and_loops_of_every_form(dtype):
    """One layer alone of each kind, the last (and only) layer's rows dropped or not; a loop of one layer,
    of all layers, run once and several times; layers without a feed-forward before a pass starts."""
    for i in range(4):
        cfg = dict(copy.deepcopy(PAZ_A), loop=None)
        cfg["layers"] = [cfg["layers"][i]]
        _run_cuts(cfg, 50 + i, dtype)
    for start, stop, times in ((0, 1, 3), (1, 2, 2), (0, 4, 2), (3, 4, 1), (2, 4, 2)):
        _run_cuts(dict(copy.deepcopy(PAZ_A), loop={"start": start, "stop": stop, "times": times}), 60 + start, dtype)
    cfg = copy.deepcopy(PAZ_B)
    cfg["layers"] = [dict(layer, mlp=None) for layer in cfg["layers"]]
    cfg["loop"] = {"start": 1, "stop": 4, "times": 2}
    _run_cuts(cfg, 70, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_of_one(dtype):
    """One head, one channel, one tap, a chunk of one position (every token sees itself alone), rank one."""
    cfg = copy.deepcopy(PAZ_D)
    cfg["loop"] = {"start": 0, "stop": 2, "times": 2}
    left = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 1.5, "softcap": 1.0, "conv": 1,
            "mask": {"size": 1}, "rot": {"base": 10.0, "dims": 2}}
    right = {"heads": 1, "dim": 1, "vdim": 1, "tau": 1.0, "decay_rank": 1}
    cfg["layers"][0]["mixer"] = {"left": left, "right": right}
    cfg["layers"][1]["mixer"]["left"]["mask"]["size"] = 2
    cfg["layers"][2]["mixer"].update(heads=1, kv_heads=1, dim=8, vdim=8, rot={"base": 50.0, "dims": 2})
    cfg["layers"][2]["mixer"]["mask"]["size"] = 1
    # (one number normed by itself keeps its sign only: a product near 0 that rounds to the other side
    # would turn it, so this is checked in 32-bit)
    if dtype == "float32":
        _run_cuts(cfg, 81, dtype)
    cfg["layers"][0]["mixer"]["left"].update(dim=8, vdim=8)
    cfg["layers"][0]["mixer"]["right"].update(dim=8, vdim=8)
    _run_cuts(cfg, 82, dtype)


@pytest.mark.parametrize("store", ["float32", "bfloat16"])
def test_weights_stored_in_32_bit_and_exported(store):
    """A checkpoint in 32-bit stays 32-bit; what the model exports is what it read."""
    from minfer_b200.model import Model
    from minfer_b200.weights.safetensors_io import load_all
    folder = make_folder("f", store, PAZ_A, 33)
    cfg, w = P.load_folder(folder)
    ids = random_ids(40, cfg["vocab"], 9)
    for dtype in DTYPES:
        eng = _engine(folder, dtype, max_tokens=256)
        s = eng.acquire()
        _close(eng.step([s], [ids], [list(range(40))]), P.forward(cfg, w, ids), dtype)
        out = eng.model.export_state_dict()
        stored = load_all(folder)
        assert set(out) == set(stored)
        for n, t in stored.items():
            assert torch.equal(out[n].cpu().float(), t.float()), n
