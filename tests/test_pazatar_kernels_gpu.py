"""The kernels of the Pazatar mechanisms, each alone against its plain function
(``tests/plain_pazatar.py``): gated linear attention over cuts of every size with the state carried in
scattered slots and its decays, the convolution without an activation, values taken from the keys, the
normed terms joining the stream, relu squared with and without the product, and attention with a chunk
mask, soft-capped scores and a sink at once, on every kernel, with marked keys at the chunks' edges."""
import pytest
import torch

import plain_pazatar as P

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def _status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def _close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max()) / max(float(want.abs().max()), 1e-30)
    assert err < tol, err


def _steps(lens, cuts):
    """For every step: (rows that bring tokens, their first token, how many)."""
    at = [0] * len(lens)
    for cut in cuts:
        rows = [b for b in range(len(lens)) if at[b] < lens[b]]
        if not rows:
            return
        take = [min(cut, lens[b] - at[b]) for b in rows]
        yield rows, [at[b] for b in rows], take
        for b, t in zip(rows, take):
            at[b] += t


def _cu(take):
    cu = [0]
    for t in take:
        cu.append(cu[-1] + t)
    return cu


LENS, SLOTS = [75, 1, 34], [4, 0, 2]
CUTS = [1, 2, 33, 3, 1, 32, 40]          # around the recurrence's chunks of 16 tokens


# ---- gated linear attention ------------------------------------------------------------------------
@pytest.mark.parametrize("H,D,Dv", [(3, 12, 20), (2, 64, 64), (1, 128, 33), (5, 7, 5), (2, 160, 40), (1, 1, 1),
                                    (4, 32, 48), (1, 256, 16), (4, 1, 6)])
@pytest.mark.parametrize("known", [True, False])
@pytest.mark.parametrize("off", [0, 3])
def test_gla_scan_over_cuts_and_slots(H, D, Dv, known, off):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(D + Dv)
    state = torch.randn(6, H, Dv, D, generator=g).to(DEV)               # stale values in every slot
    state[SLOTS] = 0.0
    stale = state[[1, 3, 5]].clone()
    scale = D ** -0.5
    seqs = []
    for n in LENS:
        d = torch.sigmoid(torch.randn(n, H, D, generator=g) * 3 + 2) ** 0.25
        seqs.append((torch.randn(n, H, D, generator=g), torch.randn(n, H, D, generator=g),
                     torch.randn(n, H, Dv, generator=g), d))
    got = [[] for _ in LENS]
    q_off, k_off, v_off = off, off + H * D, off + 2 * H * D + 1
    for rows, first, take in _steps(LENS, CUTS):
        q, k, v, d = (torch.cat([seqs[b][i][f:f + t] for b, f, t in zip(rows, first, take)]).flatten(1)
                      for i in range(4))
        n = q.shape[0]
        proj = torch.randn(n, v_off + H * Dv + 2, generator=g)
        proj[:, q_off:q_off + H * D], proj[:, k_off:k_off + H * D], proj[:, v_off:v_off + H * Dv] = q, k, v
        out = torch.empty(n, H * Dv, device=DEV)
        K.gla_scan(proj.to(DEV), q_off, k_off, v_off, d.contiguous().to(DEV), scale, state, _i32(_cu(take)),
                   _i32([SLOTS[b] for b in rows]), out, len(rows), max(take) if known else 0)
        for i, b in enumerate(rows):
            lo = _cu(take)[i]
            got[b].append(out[lo:lo + take[i]].cpu())
    for b, (q, k, v, d) in enumerate(seqs):
        want, S = P.gla_recurrence(q.double() * scale, k.double(), v.double(), d.double())
        _close(torch.cat(got[b]).view(want.shape), want, 3e-6)
        _close(state[SLOTS[b]], S.transpose(1, 2), 3e-6)
    assert torch.equal(state[[1, 3, 5]], stale)


@pytest.mark.parametrize("n,rank,channels", [(1, 5, 36), (7, 64, 300), (65, 16, 128), (130, 1, 33), (200, 160, 256)])
@pytest.mark.parametrize("tau", [1.0, 16.5])
def test_sigmoid_decay(n, rank, channels, tau):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(n + rank)
    wide = torch.randn(n, rank + 9, generator=g) * 2                     # rows of a wider tensor
    a2, b = torch.randn(channels, rank, generator=g), torch.randn(channels, generator=g) * 5
    out = torch.empty(n, channels, device=DEV)
    K.sigmoid_decay(wide.to(DEV)[:, 4:4 + rank], a2.t().contiguous().to(DEV), b.to(DEV), tau, out)
    w = {"a1": torch.eye(rank).double(), "a2": a2.double(), "a2.b": b.double()}
    want = P.gla_decay(wide[:, 4:4 + rank].double(), w, "", tau)
    _close(out, want, 4e-6)
    small = (want < 0.1) & (want > 1e-30)                                                   # fast decays: relative, too
    if bool(small.any()):
        assert float((out.double().cpu() / want - 1)[small].abs().max()) < 1e-3


# ---- convolution without an activation ---------------------------------------------------------------
@pytest.mark.parametrize("channels,taps", [(40, 4), (33, 2), (300, 8), (17, 1), (256, 3)])
def test_plain_convolution_over_cuts_and_slots(channels, taps):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(channels)
    w = torch.randn(channels, taps, generator=g)
    state = torch.randn(6, channels, taps - 1, generator=g).to(DEV)
    state[SLOTS] = 0.0
    stale = state[[1, 3, 5]].clone()
    seqs = [torch.randn(n, channels, generator=g) for n in LENS]
    got = [[] for _ in LENS]
    for rows, first, take in _steps(LENS, CUTS):
        x = torch.cat([seqs[b][f:f + t] for b, f, t in zip(rows, first, take)])
        proj = torch.cat([torch.randn(x.shape[0], 5, generator=g), x, torch.randn(x.shape[0], 2, generator=g)], 1)
        out = torch.empty(x.shape, device=DEV)
        K.conv_silu(proj.to(DEV), 5, channels, w.to(DEV), None, state, _i32([i for i, t in enumerate(take) for _ in range(t)]),
                    _i32(_cu(take)), _i32([SLOTS[b] for b in rows]), out, len(rows), single=max(take) == 1,
                    activation="none")
        for i, b in enumerate(rows):
            lo = _cu(take)[i]
            got[b].append(out[lo:lo + take[i]].cpu())
    for b, x in enumerate(seqs):
        _close(torch.cat(got[b]), P.causal_conv(x.double(), w.double()), 1e-6)
        if taps > 1:
            tail = torch.cat([torch.zeros(taps - 1, channels), x])[-(taps - 1):]
            assert torch.equal(state[SLOTS[b]].cpu(), tail.t())
    assert torch.equal(state[[1, 3, 5]], stale)


# ---- q and k normed as a whole, the values the raw keys ------------------------------------------------
@pytest.mark.parametrize("nh,nk,hd,rot", [(3, 1, 24, 16), (4, 2, 64, 64), (5, 5, 10, 4), (2, 2, 18, 0)])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_values_are_the_keys_before_norm_and_rotation(nh, nk, hd, rot, dt):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(nh + hd)
    n, off, base, eps = 90, 4, 700.0, 1e-3
    sc = {"factor": 2.5, "original": 50, "fast": 4.0, "slow": 0.5}
    proj = torch.randn(n, off + (nh + nk) * hd + 3, generator=g)
    qw, kw = torch.rand(nh * hd, generator=g) + 0.5, torch.rand(nk * hd, generator=g) + 0.5
    freqs, mag = P.yarn_frequencies(rot, base, sc) if rot else ([], 1.0)
    q, k, v = (torch.empty(n, h, hd, dtype=dt, device=DEV) for h in (nh, nk, nk))
    pages = torch.zeros(4, nk, 64, hd, dtype=dt, device=DEV)
    vpages = torch.zeros_like(pages)
    k_off = off + nh * hd
    status = _status()
    K.qk_prepare(proj.to(DEV), _i32(list(range(n))), _i32([0] * n), _i32([n]), q, k, v, pages, vpages, _i32([[2, 1]]), 2, 0,
                 q_off=off, n_heads=nh, q_width=hd, k_off=k_off, n_kv=nk, k_width=hd, v_off=k_off, v_width=hd,
                 v_from_k=False, q_norm=qw.to(DEV), k_norm=kw.to(DEV), eps=eps,
                 inv_freq=torch.tensor(freqs, dtype=torch.float64, device=DEV) if rot else None, rot_dims=rot,
                 rot_style=1, rot_magnitude=mag, q_rot_off=0, k_rot_off=0, status=status)
    p64 = proj.double()
    wq = P.rotate_interleaved(P.norm(p64[:, off:k_off], qw.double(), eps).view(n, nh, hd), freqs, mag)
    raw = p64[:, k_off:k_off + nk * hd]
    wk = P.rotate_interleaved(P.norm(raw, kw.double(), eps).view(n, nk, hd), freqs, mag)
    tol = 2e-6 if dt == torch.float32 else 6e-3
    _close(q, wq, tol)
    _close(k, wk, tol)
    _close(v, raw.view(n, nk, hd), tol)
    for p in (0, 63, 64, 89):
        page = [2, 1][p // 64]
        assert torch.equal(pages[page, :, p % 64], k[p]) and torch.equal(vpages[page, :, p % 64], v[p])
    assert int(status) == 0


# ---- normed terms into the stream ------------------------------------------------------------------------
@pytest.mark.parametrize("width", [64, 100, 33, 2048, 4096, 5000])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("form", ["one", "one, splits", "pair", "pair, splits", "pair, no outer", "no next"])
def test_norm_terms(width, dt, form):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(width)
    n = 9
    r = lambda *s: torch.randn(*s, generator=g)
    h, y1, y2, p1, p2 = r(n, width), r(n, width) * 3, r(n, width) * 0.01, r(5, n, width), r(9, n, width)
    w1, w2, wo, wn = (r(width) for _ in range(4))
    e1, eo, en, mult = 1e-3, 1e-4, 1e-2, 0.5
    dev = lambda t: t.to(DEV)
    hd, x = dev(h), torch.empty(n, width, dtype=dt, device=DEV)
    pair = form.startswith("pair") or form == "no next"
    splits = "splits" in form
    terms = [(None if splits else dev(y1), dev(p1) if splits else None, dev(w1))]
    sums = [p1.sum(0) if splits else y1]
    if pair:
        terms.append((dev(y2), dev(p2) if splits else None, dev(w2)))
        sums.append(y2 + p2.sum(0) if splits else y2)
    outer = (dev(wo), eo) if form in ("pair", "pair, splits", "no next") else None
    if form == "no next":
        K.norm_terms(hd, terms, e1, mult, outer)
    else:
        K.norm_terms(hd, terms, e1, mult, outer, (dev(wn), en), x)
    v = mult * sum(P.norm(s.double(), w.double(), e1) for s, w in zip(sums, (w1, w2)))
    if outer is not None:
        v = P.norm(v, wo.double(), eo)
    want = h.double() + v
    _close(hd, want, 2e-6)
    if form != "no next":
        _close(x, P.norm(want, wn.double(), en), 2e-6 if dt == torch.float32 else 6e-3)


def test_norm_terms_rows_do_not_depend_on_the_batch():
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(3)
    h, y, w = (torch.randn(700, 160, generator=g).to(DEV) for _ in range(3))
    a, b = h.clone(), h[5:6].clone()
    K.norm_terms(a, [(y, None, w[0])], 1e-5)
    K.norm_terms(b, [(y[5:6].contiguous(), None, w[0])], 1e-5)
    assert torch.equal(a[5:6], b)


# ---- relu squared ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_relu_squared(dt):
    from minfer_b200.kernels import api as K
    z = torch.randn(13, 77, generator=torch.Generator().manual_seed(0)) * 4
    out = torch.empty(13, 77, dtype=dt, device=DEV)
    K.unary_act(z.to(DEV), out, "relu2")
    _close(out, torch.clamp(z.double(), min=0) ** 2, 1e-6 if dt == torch.float32 else 5e-3)
    assert bool((out[z.to(DEV) <= 0] == 0).all())


@pytest.mark.parametrize("m,n,k", [(1, 64, 64), (7, 130, 200), (40, 257, 72), (300, 256, 136), (513, 100, 64)])
def test_relu_squared_in_the_products_epilogue(m, n, k):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(m)
    x, w = torch.randn(m, k, generator=g).bfloat16(), torch.randn(n, k, generator=g).bfloat16()
    status = _status()
    want = torch.clamp(x.double() @ w.double().T, min=0) ** 2
    out = torch.empty(m, n, dtype=torch.bfloat16, device=DEV)
    K.gemm_tc_xielu(x.to(DEV), w.to(DEV), out, 1.0, 0.0, status, act_l=0.0)
    _close(out, want, 6e-3)
    assert bool((out[(want == 0).to(DEV)] == 0).all()) and int(status) == 0


# ---- attention with a chunk mask, a cap and a sink at once -----------------------------------------------
DIM, CAP = 3, 9.0


@pytest.mark.parametrize("hd,vd,nh,nk,chunk", [(16, 24, 4, 2, 20), (64, 64, 8, 2, 100), (12, 12, 3, 3, 65),
                                               (10, 14, 6, 3, 64), (128, 128, 2, 1, 130), (64, 64, 2, 2, 128),
                                               (96, 96, 20, 1, 63), (128, 96, 2, 2, 33), (200, 136, 2, 1, 50)])
@pytest.mark.parametrize("dt,kernel", [(torch.float32, "any"), (torch.bfloat16, "any"),
                                       (torch.bfloat16, "mma"), (torch.bfloat16, "generic")])
@pytest.mark.parametrize("sink,cap", [(True, CAP), (False, 0.0)])
def test_chunks_caps_and_sinks(hd, vd, nh, nk, chunk, dt, kernel, sink, cap, monkeypatch):
    """In head 0 one key a chunk stands out: the first of chunk 1, the last of chunk 2, one in the middle of
    chunk 3.  A query's output is that key's value from its position to the chunk's last query and not one
    query longer.  Whole prompts over packed keys, the last queries as one step over scattered pages (a
    cache that keeps every position, and a ring), then single queries at the edges."""
    from minfer_b200.parts.sink_attention import ScoreSpec, scored_attention
    from minfer_b200.parts import sink_attention
    from minfer_b200.parts.base import CacheView, StepContext
    if kernel == "mma":
        monkeypatch.setattr(sink_attention, "PROMPT_KERNEL", "mma")
    if kernel == "generic":
        monkeypatch.setattr(sink_attention, "FORCE_GENERIC", True)
    g = torch.Generator().manual_seed(hd + chunk)
    n = max(5 * chunk - 7, 250)
    marks = [chunk, 3 * chunk - 1, 3 * chunk + chunk // 2]
    q, k = torch.randn(n, nh, hd, generator=g), torch.randn(n, nk, hd, generator=g)
    v = torch.randn(n, nk, vd, generator=g)
    q[:, 0], k[:, 0, DIM] = 0.0, 0.0
    q[:, 0, DIM] = 30.0
    for j in marks:
        k[j, 0] = 0.0
        k[j, 0, DIM] = 30.0
    q, k, v = q.to(dt), k.to(dt), v.to(dt)
    scale = 0.1
    want = P.grouped_attention(q.double(), k.double(), v.double(), scale, chunk, cap, sink)
    spec = ScoreSpec(n_heads=nh, n_kv_heads=nk, head_dim=hd, value_dim=vd, scale=scale, chunk=chunk, softcap=cap,
                     sink=sink)
    tol = 1e-5 if dt == torch.float32 else 2e-2

    def ctx(from_start, rows_tokens, positions, seq_end):
        cu = _cu(rows_tokens)
        return StepContext(device=torch.device(DEV), act_dtype=dt, n_tokens=cu[-1], n_rows=len(rows_tokens),
                           token_ids=_i32([0] * cu[-1]), positions=_i32(positions),
                           token_row=_i32([b for b, t in enumerate(rows_tokens) for _ in range(t)]),
                           cu_seqlens=_i32(cu), seq_end=_i32(seq_end), slots=_i32(list(range(len(rows_tokens)))),
                           from_start=from_start, single_token=all(t == 1 for t in rows_tokens),
                           max_row_tokens=max(rows_tokens), max_end=max(seq_end), status=_status())

    def check(got, end):
        got = got.reshape(-1, nh, vd)
        first = end - got.shape[0]
        _close(got, want[first:end], tol)
        share = 1.0 if not cap else float(torch.exp(torch.tensor(cap)) / (torch.exp(torch.tensor(cap)) + chunk + 1))
        for j in marks:
            last = (j // chunk + 1) * chunk - 1              # the last query of the key's chunk
            if first <= last < end:
                assert torch.allclose(got[last - first, 0].float().cpu(), v[j, 0].float(), atol=4e-2 + 4 * (1 - share)), j
            if first <= last + 1 < end:
                assert not torch.allclose(got[last + 1 - first, 0].float().cpu(), v[j, 0].float(), atol=0.3), j

    # the whole prompt over packed keys, beside a short one
    q2, k2, v2 = (torch.cat([x[:5], x]).to(DEV) for x in (q, k, v))
    c = ctx(True, [5, n], list(range(5)) + list(range(n)), [5, n])
    o = torch.empty(n + 5, nh * vd, dtype=dt, device=DEV)
    scored_attention(spec, q2, k2, v2, None, c, o)
    check(o[5:], n)
    _close(o[:5].view(5, nh, vd), want[:5], tol)
    tail = 200
    for ring in (0, (chunk + tail + 63) // 64 * 64):
        held = ring // 64 if ring else (n + 63) // 64
        kc = (torch.randn(held + 5, nk, 64, hd, generator=g) * 20).to(dt).to(DEV)
        vc = (torch.randn(held + 5, nk, 64, vd, generator=g) * 20).to(dt).to(DEV)
        order = torch.randperm(held + 5, generator=g)[:held].tolist()

        def put(lo, hi):
            for p in range(lo, hi):
                e = p % ring if ring else p
                kc[order[e // 64], :, e % 64] = k[p].to(DEV)
                vc[order[e // 64], :, e % 64] = v[p].to(DEV)

        cache = CacheView(k=kc, v=vc, page_table=_i32([order]), table_stride=held, ring=ring)
        put(0, n)
        for m in (tail, 60):                                   # the kernels for large and for small portions
            c = ctx(False, [m], list(range(n - m, n)), [n])
            o = torch.empty(m, nh * vd, dtype=dt, device=DEV)
            scored_attention(spec, q[n - m:].contiguous().to(DEV), None, None, cache, c, o)
            check(o, n)
        if ring:
            continue
        edges = sorted({p for j in marks for p in (j - 1, j, (j // chunk + 1) * chunk - 1, (j // chunk + 1) * chunk)
                        if p < n} | {0, 1, n - 1})
        for p in edges:
            c = ctx(False, [1], [p], [p + 1])
            o1 = torch.empty(1, nh * vd, dtype=dt, device=DEV)
            scored_attention(spec, q[p:p + 1].contiguous().to(DEV), None, None, cache, c, o1)
            _close(o1.reshape(nh, vd), want[p], tol)


def test_a_sink_takes_its_share_of_few_keys():
    """All scores 0: t visible keys with value 1 give t / (t + 1)."""
    from minfer_b200.parts.sink_attention import ScoreSpec, scored_attention
    from minfer_b200.parts.base import StepContext
    n, hd, chunk = 30, 64, 7
    for dt in (torch.float32, torch.bfloat16):
        q, k, v = (torch.zeros(n, 2, hd, dtype=dt, device=DEV) for _ in range(3))
        v += 1.0
        c = StepContext(device=torch.device(DEV), act_dtype=dt, n_tokens=n, n_rows=1, token_ids=_i32([0] * n),
                        positions=_i32(list(range(n))), token_row=_i32([0] * n), cu_seqlens=_i32([0, n]),
                        seq_end=_i32([n]), slots=_i32([0]), from_start=True, single_token=False, max_row_tokens=n,
                        max_end=n, status=_status())
        o = torch.empty(n, 2 * hd, dtype=dt, device=DEV)
        scored_attention(ScoreSpec(2, 2, hd, hd, 0.125, chunk=chunk, sink=True, softcap=3.0), q, k, v, None, c, o)
        want = torch.tensor([(p % chunk + 1) / (p % chunk + 2) for p in range(n)])
        _close(o[:, 0], want, 1e-6 if dt == torch.float32 else 5e-3)


# ---- heads prepared one by one, with and without the convolution in the same kernel --------------------------
@pytest.mark.parametrize("nh,nk,qw,vw,rot,style,taps", [(4, 2, 16, 24, 8, 0, 4), (3, 1, 128, 128, 64, 0, 2),
                                                        (6, 3, 64, 64, 64, 1, 8), (2, 2, 8, 4, 0, 0, 5),
                                                        (1, 1, 10, 14, 6, 0, 3), (5, 1, 36, 12, 24, 0, 1),
                                                        (2, 1, 136, 128, 16, 0, 4), (9, 3, 32, 40, 16, 0, 0)])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("lens", [LENS, [600, 3, 521]])
def test_heads_behind_a_convolution(nh, nk, qw, vw, rot, style, taps, dt, lens):
    """Rows in scattered slots over cuts of every size (runs of tokens that cross rows and chunks, single
    tokens), positions that go on from the cut before, keys and values into scattered pages."""
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(nh * qw + taps)
    nq, nkw, nv = nh * qw, nk * qw, nk * vw
    channels, off, eps, base = nq + nkw + nv, 4, 1e-3, 400.0
    cw = torch.randn(channels, max(taps, 1), generator=g)
    qn, kn = torch.rand(qw, generator=g) + 0.5, torch.rand(qw, generator=g) + 0.5
    freqs = P.plain_frequencies(rot, base) if rot else []
    inv = torch.tensor(freqs, dtype=torch.float64, device=DEV) if rot else None
    seqs = [torch.randn(n, channels, generator=g) for n in lens]
    state = torch.randn(6, channels, max(taps - 1, 0), generator=g).to(DEV)
    state[SLOTS] = 0.0
    stale = state[[1, 3, 5]].clone()
    pages = (max(lens) + 63) // 64
    order = torch.randperm(3 * pages, generator=g).view(3, pages)
    kc = torch.zeros(3 * pages, nk, 64, qw, dtype=dt, device=DEV)
    vc = torch.zeros(3 * pages, nk, 64, vw, dtype=dt, device=DEV)
    status = _status()
    got = [[[], [], []] for _ in lens]
    cuts = CUTS if max(lens) < 100 else [1, 3, 517, 200]
    for rows, first, take in _steps(lens, cuts):
        x = torch.cat([seqs[b][f:f + t] for b, f, t in zip(rows, first, take)])
        n = x.shape[0]
        proj = torch.cat([torch.randn(n, off, generator=g), x, torch.randn(n, 4, generator=g)], 1).to(DEV)
        outs = [torch.empty(n, h, w, dtype=dt, device=DEV) for h, w in ((nh, qw), (nk, qw), (nk, vw))]
        conv = (cw.to(DEV), cw.t().contiguous().to(DEV), state, _i32(_cu(take)), _i32([SLOTS[b] for b in rows]), len(rows), max(take) == 1) if taps else None
        K.head_prepare(proj, _i32([f + i for f, t in zip(first, take) for i in range(t)]),
                       _i32([i for i, t in enumerate(take) for _ in range(t)]), _i32([f + t for f, t in zip(first, take)]),
                       *outs, kc, vc, order[rows].int().to(DEV).contiguous(), pages, 0, q_off=off, n_heads=nh, q_width=qw,
                       k_off=off + nq, n_kv=nk, k_width=qw, v_off=off + nq + nkw, v_width=vw, q_norm=qn.to(DEV),
                       k_norm=kn.to(DEV), eps=eps, inv_freq=inv, rot_dims=rot, rot_style=style, rot_magnitude=1.25,
                       q_mul=1.0, k_mul=0.5, status=status, conv=conv)
        for i, b in enumerate(rows):
            lo = _cu(take)[i]
            for j in range(3):
                got[b][j].append(outs[j][lo:lo + take[i]].cpu())
    tol = 3e-6 if dt == torch.float32 else 6e-3
    done = sum(cuts)
    for b, x in enumerate(seqs):
        n = min(lens[b], done)
        u = P.causal_conv(x.double(), cw.double()) if taps else x.double()
        q, k, v = u[:, :nq].view(-1, nh, qw), u[:, nq:nq + nkw].view(-1, nk, qw), u[:, nq + nkw:].view(-1, nk, vw)
        q, k = P.norm(q, qn.double(), eps), P.norm(k, kn.double(), eps)
        turn = (lambda z: P.rotate_interleaved(z, freqs, 1.25)) if style else (
            lambda z: torch.cat([P.rotate_half(z, freqs)[..., :rot] * 1.25, z[..., rot:]], -1))
        q, k = turn(q), turn(k) * 0.5
        for j, want in enumerate((q, k, v)):
            _close(torch.cat(got[b][j]), want[:n], tol)
        for p in {p for p in (0, 1, n // 2, n - 1, 63, 64) if p < n}:
            at = int(order[b, p // 64])
            _close(kc[at, :, p % 64], k[p], tol)
            _close(vc[at, :, p % 64], v[p], tol)
        if taps > 1:
            assert torch.equal(state[SLOTS[b]].cpu(), torch.cat([torch.zeros(taps - 1, channels), x[:n]])[-(taps - 1):].t())
    assert torch.equal(state[[1, 3, 5]], stale) and int(status) == 0
