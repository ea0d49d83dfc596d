"""The kernels of the Pikavik mechanisms, each alone against its plain function
(``tests/plain_pikavik.py``): the mixes with the token before, the decays, both recurrences over cuts
of every size with the state carried in scattered slots, the head norm with divisor and weight, the
group-limited router with ties, the scaled add with and without the next norm, grouped products over
ragged groups, the attention over wide latent vectors with marked keys far back, at page borders and
at a window's edge over scrambled pages and a ring."""
import pytest
import torch

import plain_pikavik as P

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


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
CUTS = [1, 2, 33, 3, 1, 32, 40]          # around the recurrences' chunks of 16 and 32 tokens


# ---- mixes with the token before ---------------------------------------------------------------------
@pytest.mark.parametrize("width", [64, 100, 33, 2056])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_shift_mix(width, dt):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(width)
    mu = torch.rand(5, width, generator=g)
    seqs = [torch.randn(n, width, generator=g).to(dt) for n in LENS]
    state = torch.randn(6, width, generator=g).to(DEV)                 # stale values in every slot
    state[SLOTS] = 0.0
    stale = state[[1, 3, 5]].clone()
    got = [[] for _ in LENS]
    for rows, first, take in _steps(LENS, CUTS):
        x = torch.cat([seqs[b][f:f + t] for b, f, t in zip(rows, first, take)]).to(DEV)
        n = x.shape[0]
        token_row = [i for i, t in enumerate(take) for _ in range(t)]
        out = torch.empty(5, n, width, dtype=dt, device=DEV)
        K.shift_mix(x, mu.to(DEV), _i32(token_row), _i32(_cu(take)), _i32([SLOTS[b] for b in rows]), state, out,
                    len(rows), max(take) == 1)
        for i, b in enumerate(rows):
            lo = _cu(take)[i]
            got[b].append(out[:, lo:lo + take[i]].cpu())
    for b, x in enumerate(seqs):
        x = x.double()
        want = torch.stack([x + (P.shifted(x) - x) * mu[s].double() for s in range(5)])
        _close(torch.cat(got[b], dim=1), want, 1e-6 if dt == torch.float32 else 5e-3)
        assert torch.equal(state[SLOTS[b]].cpu().double(), x[-1])
    assert torch.equal(state[[1, 3, 5]], stale)


@pytest.mark.parametrize("n,rank,channels", [(1, 5, 36), (7, 64, 300), (65, 16, 128), (130, 3, 33), (200, 160, 256)])
def test_wkv_decay(n, rank, channels):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(n + rank)
    wide = torch.randn(n, rank + 9, generator=g) * 2                   # rows of a wider tensor
    w2, w0 = torch.randn(channels, rank, generator=g) * 0.2, torch.randn(channels, generator=g) * 2 - 2
    out = torch.empty(n, channels, device=DEV)
    K.wkv_decay(wide.to(DEV)[:, 4:4 + rank], w2.t().contiguous().to(DEV), w0.to(DEV), out)
    t1 = wide[:, 4:4 + rank].double()
    _close(out, torch.exp(-torch.exp(torch.tanh(t1) @ w2.double().T + w0.double())), 2e-6)


# ---- the recurrences -----------------------------------------------------------------------------------
@pytest.mark.parametrize("H,D,Dv", [(3, 12, 20), (2, 64, 64), (1, 128, 33), (5, 7, 5), (2, 160, 40), (1, 1, 1),
                                    (4, 32, 48), (1, 256, 16)])
@pytest.mark.parametrize("known", [True, False])
def test_wkv_scan_over_cuts_and_slots(H, D, Dv, known):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(D + Dv)
    state = torch.randn(6, H, Dv, D, generator=g).to(DEV)
    state[SLOTS] = 0.0
    stale = state[[1, 3, 5]].clone()
    u = torch.randn(H, D, generator=g)
    seqs = []
    for n in LENS:
        r, k = torch.randn(n, H, D, generator=g), torch.randn(n, H, D, generator=g) * D ** -0.5
        v, d = torch.randn(n, H, Dv, generator=g), torch.exp(-torch.exp(torch.randn(n, H, D, generator=g) * 2 - 3))
        seqs.append((r, k, v, d))
    got = [[] for _ in LENS]
    for rows, first, take in _steps(LENS, CUTS):
        r, k, v, d = (torch.cat([seqs[b][i][f:f + t] for b, f, t in zip(rows, first, take)]).flatten(1)
                      .contiguous().to(DEV) for i in range(4))
        out = torch.empty(r.shape[0], H * Dv, device=DEV)
        K.wkv_scan(r, k, v, d, u.to(DEV), state, _i32(_cu(take)), _i32([SLOTS[b] for b in rows]), out, len(rows),
                   max(take) if known else 0)
        for i, b in enumerate(rows):
            lo = _cu(take)[i]
            got[b].append(out[lo:lo + take[i]].cpu())
    for b, (r, k, v, d) in enumerate(seqs):
        want, S = P.wkv_recurrence(r.double(), k.double(), v.double(), d.double(), u.double())
        _close(torch.cat(got[b]).view(want.shape), want, 3e-6)
        _close(state[SLOTS[b]], S.transpose(1, 2), 3e-6)
    assert torch.equal(state[[1, 3, 5]], stale)


@pytest.mark.parametrize("H,D,Dv,cap,forget", [(3, 12, 20, 9.0, 3.0), (2, 64, 128, 15.0, 5.0), (1, 128, 31, 4.0, 0.0),
                                               (5, 7, 5, 30.0, 2.0), (2, 160, 40, 12.0, 8.0), (1, 1, 1, 1.0, 0.0),
                                               (4, 32, 15, 15.0, -6.0)])
@pytest.mark.parametrize("known", [True, False])
def test_mlstm_scan_over_cuts_and_slots(H, D, Dv, cap, forget, known):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(D * 3 + Dv)
    state = torch.randn(6, H, Dv + 1, D, generator=g).to(DEV)
    top = torch.randn(6, H, Dv + 1, generator=g).to(DEV)
    state[SLOTS] = 0.0
    top[SLOTS] = 0.0
    ib, fb = torch.randn(H, generator=g), torch.randn(H, generator=g) + forget
    scale = D ** -0.5
    seqs = []
    for n in LENS:
        seqs.append((torch.randn(n, H, D, generator=g), torch.randn(n, H, D, generator=g),
                     torch.randn(n, H, Dv, generator=g), torch.randn(n, H, generator=g) * 6,
                     torch.randn(n, H, generator=g) * 3))
    got = [[] for _ in LENS]
    q_off, k_off = 4, 4 + H * D
    v_off = k_off + H * D
    i_off = v_off + H * Dv + 3
    f_off = i_off + H
    for rows, first, take in _steps(LENS, CUTS):
        q, k, v, i, f = (torch.cat([seqs[b][x][a:a + t] for b, a, t in zip(rows, first, take)]).flatten(1)
                         for x in range(5))
        n = q.shape[0]
        proj = torch.randn(n, f_off + H + 1, generator=g)
        proj[:, q_off:k_off], proj[:, k_off:v_off], proj[:, v_off:v_off + H * Dv] = q, k, v
        proj[:, i_off:f_off], proj[:, f_off:f_off + H] = i, f
        out, den = torch.empty(n, H * Dv, device=DEV), torch.empty(n, H, device=DEV)
        K.mlstm_scan(proj.to(DEV), q_off, k_off, v_off, i_off, f_off, ib.to(DEV), fb.to(DEV), cap, scale, state, top,
                     _i32(_cu(take)), _i32([SLOTS[b] for b in rows]), out, den, len(rows), max(take) if known else 0)
        y = out.view(n, H, Dv) / den[:, :, None]
        for j, b in enumerate(rows):
            lo = _cu(take)[j]
            got[b].append(y[lo:lo + take[j]].cpu())
    for b, (q, k, v, i, f) in enumerate(seqs):
        li = cap * torch.tanh((i.double() + ib.double()) / cap)
        lf = P.log_sigmoid(cap * torch.tanh((f.double() + fb.double()) / cap))
        want, (S, nrm, m) = P.mlstm_recurrence(q.double() * scale, k.double(), v.double(), li, lf)
        # (a normalizer that nearly cancels scales rounding up; the state itself is held tighter below)
        _close(torch.cat(got[b]), want, 1e-4)
        back = torch.exp(m)[:, None, None]         # (the kernel's own maximum is the stabilizer of its state)
        mine = state[SLOTS[b]].double().cpu() * torch.exp(top[SLOTS[b]].double().cpu())[:, :, None]
        _close(mine[:, :Dv], S.transpose(1, 2) * back, 1e-5)
        _close(mine[:, Dv], nrm * back[:, :, 0], 1e-5)
        _close(top[SLOTS[b]], m[:, None].expand(H, Dv + 1), 1e-5)


@pytest.mark.parametrize("heads,dv", [(3, 20), (2, 128), (1, 1), (5, 33)])
@pytest.mark.parametrize("act", ["silu", "sigmoid"])
def test_head_norm_with_divisor_and_weight(heads, dv, act):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(dv)
    n, off = 13, 6
    o, gate = torch.randn(n, heads * dv, generator=g), torch.randn(n, off + heads * dv + 2, generator=g)
    den, w = torch.rand(n, heads, generator=g) * 3 + 0.01, torch.randn(heads * dv, generator=g)
    out = torch.empty(n, heads * dv, device=DEV)
    K.unit_norm_gate(o.to(DEV), gate.to(DEV), off, out, heads, 1e-3, act, den=den.to(DEV), weight=w.to(DEV))
    x = P.rms_unit(o.double().view(n, heads, dv) / den.double()[:, :, None], 1e-3).reshape(n, -1)
    z = gate.double()[:, off:off + heads * dv]
    _close(out, x * w.double() * (P.silu(z) if act == "silu" else torch.sigmoid(z)), 2e-6)


# ---- the router --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("experts,groups,keep,top", [(16, 4, 3, 4), (6, 3, 2, 2), (12, 1, 1, 5), (64, 64, 9, 7),
                                                     (40, 5, 5, 8), (96, 8, 1, 3), (1, 1, 1, 1), (8, 4, 2, 4)])
def test_route_groups(experts, groups, keep, top):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(experts + top)
    n = 100
    z = torch.randn(n, experts + 3, generator=g) * 1.5                 # rows carry more columns than the router's
    idx, wts = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
    K.moe_route_groups(z.to(DEV), idx, wts, top, experts, groups, keep, 1.75)
    chosen, weight, margin = P.choose(z[:, :experts].double(), top, groups, keep, 1.75)
    sure = margin > 1e-5
    assert sure.float().mean() > 0.9
    assert torch.equal(idx.cpu().long()[sure], chosen[sure])
    _close(wts[sure.to(DEV)], weight[sure], 2e-6)


def test_route_groups_ties_go_to_the_lower_index():
    from minfer_b200.kernels import api as K
    z = torch.zeros(2, 12, device=DEV)
    z[1, 7], z[1, 10] = 1.0, 1.0
    idx, wts = torch.empty(2, 3, dtype=torch.int32, device=DEV), torch.empty(2, 3, device=DEV)
    K.moe_route_groups(z, idx, wts, 3, 12, 4, 2, 1.0)
    assert idx.tolist() == [[0, 1, 2], [7, 10, 6]]
    s, h = float(torch.sigmoid(torch.tensor(1.0))), 0.5
    _close(wts, torch.tensor([[1 / 3] * 3, [s / (2 * s + h), s / (2 * s + h), h / (2 * s + h)]]), 1e-6)


# ---- the end of a layer --------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [64, 100, 33, 2048, 5000])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("form", ["both", "one", "splits", "no norm"])
def test_scaled_add(width, dt, form):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(width)
    n = 9
    r = lambda *s: torch.randn(*s, generator=g)
    h, y1, y2, p1, p2 = r(n, width), r(n, width), r(n, width), r(5, n, width), r(3, n, width)
    a1, a2, w = r(width), r(width), r(width)
    hd = h.to(DEV)
    x = torch.empty(n, width, dtype=dt, device=DEV)
    dev = lambda t: t.to(DEV)
    first, second = {"both": ((dev(y1), None, dev(a1)), (dev(y2), None, dev(a2))),
                     "one": ((dev(y1), None, dev(a1)), None),
                     "splits": ((None, dev(p1), dev(a1)), (dev(y2), dev(p2), dev(a2))),
                     "no norm": ((dev(y1), dev(p1), dev(a1)), (None, dev(p2), dev(a2)))}[form]
    if form == "no norm":
        K.scaled_add(hd, first, second)
    else:
        K.scaled_add(hd, first, second, dev(w), 1e-4, x)
    t1 = {"both": y1, "one": y1, "splits": p1.sum(0), "no norm": y1 + p1.sum(0)}[form].double()
    t2 = {"both": y2, "one": 0 * y2, "splits": y2 + p2.sum(0), "no norm": p2.sum(0)}[form].double()
    want = h.double() + a1.double() * t1 + a2.double() * t2
    _close(hd, want, 2e-6)
    if form != "no norm":
        _close(x, P.rms_unit(want, 1e-4) * w.double(), 2e-6 if dt == torch.float32 else 6e-3)


# ---- grouped products --------------------------------------------------------------------------------------
@pytest.mark.parametrize("counts", [[5, 0, 17, 1], [130, 0, 0, 300, 128, 7], [64] * 40, [0, 0, 3], [200, 33]])
@pytest.mark.parametrize("N,Kd", [(96, 64), (256, 200), (130, 520)])
def test_grouped_product_over_ragged_groups(counts, N, Kd):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(N + len(counts))
    rows, G = sum(counts), len(counts)
    x, w = torch.randn(rows, Kd, generator=g).bfloat16(), torch.randn(G, N, Kd, generator=g).bfloat16()
    first = _cu(counts)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((rows + 2, N), 7.0, device=DEV)
    K.gemm_tc_grouped(x.to(DEV), w.to(DEV), out[:rows], _i32(first), status)
    want = torch.cat([x[a:b].double() @ w[i].double().T for i, (a, b) in enumerate(zip(first, first[1:]))])
    _close(out[:rows], want, 1e-5)
    assert bool((out[rows:] == 7.0).all())
    act = torch.empty(rows, N // 2, dtype=torch.bfloat16, device=DEV)
    K.gemm_tc_grouped(x.to(DEV), w.to(DEV), act, _i32(first), status, "clamped_swish", 1.1, 1.702)
    gate, up = want[:, 0::2].clamp(max=1.1), want[:, 1::2].clamp(-1.1, 1.1)
    _close(act, gate * torch.sigmoid(1.702 * gate) * (up + 1), 8e-3)
    assert int(status) == 0


@pytest.mark.parametrize("n", [1, 8, 50, 255, 300])
def test_grouped_projection(n):
    from minfer_b200.parts.linear import GroupedLinear
    g = torch.Generator().manual_seed(n)
    w = [torch.randn(72, 136, generator=g) for _ in range(4)]
    x = torch.randn(4, n, 136, generator=g)
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 1e-5)):
        ws, xs = [t.to(dt) for t in w], x.to(dt)
        out = GroupedLinear([t.to(DEV) for t in ws]).forward(xs.to(DEV))
        _close(out, torch.stack([xs[i].double() @ ws[i].double().T for i in range(4)]), tol)


# ---- attention over wide latent vectors ----------------------------------------------------------------
def _latent_case(H, kw, vd, window, ring, lens, seed, queries=1):
    """Sequences of ``lens`` positions in scrambled pages; the last ``queries`` positions of each ask."""
    g = torch.Generator().manual_seed(seed)
    pages_of = [((ring if ring else n) + 63) // 64 for n in lens]
    total = sum(pages_of) + 3
    order = torch.randperm(total, generator=g).tolist()
    cache = torch.randn(total, 1, 64, kw, generator=g).bfloat16() * 50          # what nobody may see
    width = max(pages_of)
    table = torch.full((len(lens), width), -1, dtype=torch.int32)
    keys = [torch.randn(n, kw, generator=g).bfloat16() for n in lens]
    for b, n in enumerate(lens):
        for j in range(pages_of[b]):
            table[b, j] = order.pop()
        for p in range(n):
            e = p % ring if ring else p
            cache[int(table[b, e >> 6]), 0, e & 63] = keys[b][p]
    q = [torch.randn(queries, H, kw, generator=g).bfloat16() for _ in lens]
    return g, cache, table, keys, q


def _latent_run(K, q, cache, table, lens, H, kw, vd, window, ring, scale, sink, queries=1):
    rows = [(b, n - queries + i) for b, n in enumerate(lens) for i in range(queries)]
    out = torch.empty(len(rows), H * vd, dtype=torch.bfloat16, device=DEV)
    K.latent_decode(torch.cat(q).contiguous().to(DEV), cache.to(DEV), _i32([b for b, _ in rows]),
                    _i32([p for _, p in rows]), table.to(DEV), table.shape[1], ring, out, H, kw, vd, window,
                    sink is not None, scale, min(window, max(lens)) if window else max(lens),
                    sink_logit=None if sink is None else sink.to(DEV))
    return rows, out.view(len(rows), H, vd)


@pytest.mark.parametrize("H,kw,vd,window,ring", [(4, 160, 128, 0, 0), (16, 576, 512, 0, 0), (20, 136, 112, 0, 0),
                                                 (1, 640, 640, 0, 0), (33, 144, 80, 0, 0), (3, 200, 200, 0, 0),
                                                 (4, 352, 304, 70, 128), (2, 136, 136, 1, 64)])
@pytest.mark.parametrize("lens", [[1, 64, 65], [700, 3, 129, 128, 640]])
def test_latent_decode(H, kw, vd, window, ring, lens):
    from minfer_b200.kernels import api as K
    scale = 1.2 * kw ** -0.5
    g, cache, table, keys, q = _latent_case(H, kw, vd, window, ring, lens, H + kw)
    sink = torch.randn(H, generator=g)
    rows, out = _latent_run(K, q, cache, table, lens, H, kw, vd, window, ring, scale, sink)
    for i, (b, p) in enumerate(rows):
        lo = max(0, p - window + 1) if window else 0
        k = keys[b][lo:p + 1].double()
        s = torch.einsum("hd,jd->hj", q[b][0].double(), k) * scale
        s = torch.cat([s, sink.double()[:, None]], dim=1)
        want = torch.softmax(s, dim=-1)[:, :-1] @ k[:, :vd]
        _close(out[i], want, 1.5e-2)


@pytest.mark.parametrize("kw,vd", [(160, 128), (576, 512)])
@pytest.mark.parametrize("window,ring", [(0, 0), (70, 192)])
def test_latent_decode_sees_the_marked_key_and_no_later_one(kw, vd, window, ring):
    """Every query's weight lies on one marked key: far back, at a page's first and last position, at
    the query itself, at the window's last position and one beyond it (not seen: the key before
    the query then stands out instead)."""
    from minfer_b200.kernels import api as K
    H, n = 4, 150
    g, cache, table, keys, q = _latent_case(H, kw, vd, window, ring, [n], 5)
    pos = n - 1
    marks = [pos, pos - 1, 128, 127] + ([pos - window + 1, pos - window] if window else [0, 1, 63, 64])
    for mark in marks:
        seen = mark <= pos and (not window or pos - mark < window)
        k = keys[0].clone() * 0.01
        d = torch.randn(kw, generator=g)
        d[vd:] = d[vd:] + 1.0
        other = torch.randn(kw, generator=g)
        k[mark] = (d / d.norm() * 30).bfloat16()
        if not seen:
            k[pos - 1] = (d / d.norm() * 10 + other / other.norm()).bfloat16()
        c = cache.clone()
        for p in range(max(0, n - (ring or n)), n):
            e = p % ring if ring else p
            c[int(table[0, e >> 6]), 0, e & 63] = k[p]
        qq = [(d / d.norm() * 30).bfloat16().expand(1, H, kw).contiguous()]
        _, out = _latent_run(K, qq, c, table, [n], H, kw, vd, window, ring, 1.0, None)
        _close(out[0], k[mark if seen else pos - 1][:vd].double().expand(H, vd), 1e-2)


def test_latent_decode_sink_takes_its_share():
    from minfer_b200.kernels import api as K
    H, kw, vd = 3, 160, 128
    cache = torch.zeros(2, 1, 64, kw).bfloat16()
    cache[..., 0] = 1.0
    sink = torch.tensor([0.0, 1.5, -2.0])
    for n in (1, 5, 64, 100):
        q = [torch.zeros(1, H, kw).bfloat16()]
        _, out = _latent_run(K, q, cache, torch.tensor([[1, 0]], dtype=torch.int32), [n], H, kw, vd, 0, 0, 0.3, sink)
        _close(out[0, :, 0], n / (n + torch.exp(sink.double())), 5e-3)


def test_latent_decode_every_token_of_a_portion_is_a_query():
    from minfer_b200.kernels import api as K
    H, kw, vd, n, m = 6, 184, 152, 140, 37
    g, cache, table, keys, q = _latent_case(H, kw, vd, 0, 0, [n], 9, queries=m)
    rows, out = _latent_run(K, q, cache, table, [n], H, kw, vd, 0, 0, 0.1, None, queries=m)
    for i, (_, p) in enumerate(rows):
        k = keys[0][:p + 1].double()
        want = torch.softmax(torch.einsum("hd,jd->hj", q[0][i].double(), k) * 0.1, dim=-1) @ k[:, :vd]
        _close(out[i], want, 1.5e-2)


# ---- few tokens ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("n,top,experts,width", [(1, 1, 1, 8), (5, 3, 7, 64), (48, 4, 16, 100), (200, 5, 40, 24)])
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_group_few(n, top, experts, width, dt):
    """Pairs grouped by expert in their order, the experts' first rows (also of experts nobody chose)
    and the gathered inputs."""
    from minfer_b200.kernels import api as K
    if width * (4 if dt == torch.float32 else 2) % 16:
        width += 4
    g = torch.Generator().manual_seed(n)
    idx = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(n)]).int()
    x = torch.randn(n, width, generator=g).to(dt)
    out = torch.empty(n * top, width, dtype=dt, device=DEV)
    first, where = torch.empty(experts + 1, dtype=torch.int32, device=DEV), torch.empty(n, top, dtype=torch.int32, device=DEV)
    K.moe_group_few(idx.to(DEV), x.to(DEV), experts, out, first, where)
    order = torch.argsort(idx.flatten().long(), stable=True)
    rows = torch.empty_like(order)
    rows[order] = torch.arange(n * top)
    assert torch.equal(where.cpu().flatten().long(), rows)
    assert first.tolist() == [int((idx < e).sum()) for e in range(experts + 1)]
    assert torch.equal(out.cpu(), x[order // top])


@pytest.mark.parametrize("n", [1, 7, 8, 16, 17])
@pytest.mark.parametrize("heads,J,D,tail,gated", [(3, 40, 24, 16, False), (16, 24, 264, 0, True), (1, 5, 8, 8, False)])
def test_per_head_products_of_few_tokens(n, heads, J, D, tail, gated):
    from minfer_b200.kernels import api as K
    g = torch.Generator().manual_seed(n + J)
    x = torch.randn(n, heads * (D + tail), generator=g).bfloat16()
    w = (torch.randn(heads, J, D, generator=g) * D ** -0.5).bfloat16()
    gate = torch.randn(n, 3 + heads * J, generator=g)
    y = torch.empty(n, heads * (J + tail), dtype=torch.bfloat16, device=DEV)
    K.head_linear(x.to(DEV), w.to(DEV), y, x_head=D + tail, x_off=0, y_head=J + tail, tail=tail, x_tail_off=D,
                  gate=gate.to(DEV) if gated else None, gate_off=3)
    xh = x.double().view(n, heads, D + tail)
    want = torch.einsum("hjd,nhd->nhj", w.double(), xh[..., :D])
    if gated:
        want = want * torch.sigmoid(gate.double()[:, 3:].view(n, heads, J))
    _close(y.view(n, heads, J + tail), torch.cat([want, xh[..., D:]], dim=-1), 6e-3)
