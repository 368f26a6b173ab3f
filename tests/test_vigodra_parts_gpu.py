"""Each new mechanism alone on the GPU against the plain implementation, in both dtypes: the layer norm and the norm of the
sum with its output bias, rounded copy and depth average; the embedding's further outputs; the clamped gate as an
element-wise kernel and in the products' epilogues; short filters with biases, norms over the whole projection and the cache
write (from kept inputs, for unequal requests, the same bits however a sequence is cut); rotation in halves of a latent's
parts; the gate per value behind a product per head; attention with a distance bias, a window that keeps the first
positions and a sink (planted keys inside and just outside the window, the last kept and the first not kept position, at
page borders, far back, at distances where the bucket changes), as portions and as decoded tokens in runs."""
from types import SimpleNamespace

import pytest
import torch

import plain_vigodra as pv

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, ref, dtype, f32=2e-5, what=""):
    tol = f32 * max(1.0, float(ref.abs().max())) if dtype == torch.float32 else 2.0 ** -7 * float(ref.abs().max())
    worst = float((got.double().cpu() - ref.double()).abs().max())
    assert worst <= tol, (what, worst, tol)


# ---------------------------------------------------------------------------------------------- the stream

WIDTHS = [(3, 4), (5, 7), (33, 64), (2, 130), (9, 200), (4, 513), (3, 1028), (130, 2048), (2, 4100), (2, 8192), (1, 9000)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,h", WIDTHS)
def test_layer_norm(dtype, n, h):
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(h)
    x = torch.randn(n + 2, h, generator=g) * 3 + 5          # a mean far from zero
    w, b = torch.randn(h, generator=g), torch.randn(h, generator=g)
    rows = torch.randint(0, n + 2, (n,), generator=g)
    out = torch.empty(n, h, dtype=dtype, device=DEV)
    ops.layer_norm(x.to(DEV), w.to(DEV), b.to(DEV), 1e-4, out, i32(rows.tolist()))
    close(out, pv.layer_norm(x.double()[rows], w.double(), b.double(), 1e-4), dtype, what="rows")
    out = torch.empty(n + 2, h, dtype=dtype, device=DEV)
    ops.layer_norm(x.to(DEV), w.to(DEV), b.to(DEV), 1e-4, out)
    close(out, pv.layer_norm(x.double(), w.double(), b.double(), 1e-4), dtype, what="all")
    one = torch.empty(1, h, dtype=dtype, device=DEV)
    ops.layer_norm(x[1:2].to(DEV), w.to(DEV), b.to(DEV), 1e-4, one)
    assert torch.equal(one[0], out[1])                      # a row's bits do not depend on the batch


@pytest.mark.parametrize("n,h", WIDTHS)
@pytest.mark.parametrize("done", [None, 0, 1, 2, 7])
def test_norm_of_the_sum_and_depth_average(n, h, done):
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(h + 1)
    x, branch = torch.randn(n, h, generator=g) + 2, torch.randn(n, h, generator=g)
    w, b, ob = torch.randn(h, generator=g), torch.randn(h, generator=g), torch.randn(h, generator=g)
    for bias, keep, alpha in ((None, True, 1.0), (ob, False, 2.7)):
        stages = torch.randn(9, n, h, generator=g)
        mix = None if done is None else torch.randn(done + 1, generator=g)
        y = pv.layer_norm(alpha * x.double() + branch.double() + (0 if bias is None else bias.double()), w.double(), b.double(), 1e-5)
        ref = y if done is None else pv.depth_average([s.double() for s in stages[:done]] + [y], mix.double())
        xd, bd, sd = x.to(DEV), branch.to(DEV), stages.to(DEV)
        copy = torch.empty(n, h, dtype=torch.bfloat16, device=DEV)
        kw = {} if done is None else {"stages": sd, "done": done, "mix": mix.to(DEV), "keep": keep}
        ops.post_norm_join(bd, xd, w.to(DEV), b.to(DEV), 1e-5, alpha, out_bias=None if bias is None else bias.to(DEV), copy=copy, **kw)
        close(xd, ref, torch.float32, what="stream")
        assert float(bd.abs().max()) == 0.0 and torch.equal(copy, xd.to(torch.bfloat16))
        if done is not None:
            if keep:
                close(sd[done], y, torch.float32, what="stage")
            others = [j for j in range(9) if j != done or not keep]
            assert torch.equal(sd[others].cpu(), stages[others])
            # the average on its own gives what the norm's last lines give, to rounding
            z, s2 = y.float().to(DEV), stages.to(DEV)
            ops.depth_average(z, s2, done, mix.to(DEV), keep)
            close(z, ref, torch.float32, what="average alone")
            assert not keep or torch.equal(s2[done].cpu(), y.float())
    one, b1 = x[:1].to(DEV), branch[:1].to(DEV)             # a row's bits do not depend on the batch
    xd, bd = x.to(DEV), branch.to(DEV)
    ops.post_norm_join(b1, one, w.to(DEV), b.to(DEV), 1e-5, 1.5)
    ops.post_norm_join(bd, xd, w.to(DEV), b.to(DEV), 1e-5, 1.5)
    assert torch.equal(one[0], xd[0])


def test_row_bias_and_the_embeddings_further_outputs():
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(3)
    x, b = torch.randn(5, 70, generator=g), torch.randn(70, generator=g)
    xd = x.to(DEV)
    ops.row_add(xd, b.to(DEV))
    assert torch.equal(xd.cpu(), x + b)
    for dtype in DTYPES:
        table = torch.randn(50, 72, generator=g).to(dtype)
        tokens = [3, 49, 0, 3, 17]
        out, twin = torch.empty(5, 72, device=DEV), torch.empty(5, 72, device=DEV)
        copy = torch.empty(5, 72, dtype=torch.bfloat16, device=DEV)
        ops.embedding(i32(tokens), table.to(DEV), out, scale=7.25, twin=twin, copy=copy)
        assert torch.equal(out.cpu(), table[tokens].float() * 7.25) and torch.equal(twin, out) and torch.equal(copy, out.to(torch.bfloat16))


@pytest.mark.parametrize("limit", [0.3, 2.0, 50.0])
def test_clamped_gate_alone(limit):
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(4)
    for m, inter, block in [(3, 24, 8), (5, 128, 128), (2, 20, 4), (7, 21, 1), (200, 256, 128)]:
        gate, up = torch.randn(m, inter, generator=g) * 3, torch.randn(m, inter, generator=g) * 3
        gate[0, 0], gate[0, 1], up[0, 0] = 200.0, -200.0, -300.0
        both = torch.stack([gate.view(m, -1, block), up.view(m, -1, block)], dim=2).reshape(m, 2 * inter)
        for src, dst, consume in ((torch.float32, torch.float32, False), (torch.float32, torch.bfloat16, True),
                                  (torch.bfloat16, torch.bfloat16, False), (torch.float32, torch.bfloat16, False)):
            q = both.to(src)
            gq = q.view(m, -1, 2, block).double()
            ref = pv.clamped_glu(gq[:, :, 0].reshape(m, inter), gq[:, :, 1].reshape(m, inter), limit)
            dev, out = q.to(DEV), torch.empty(m, inter, dtype=dst, device=DEV)
            ops.silu_mul(dev, out, block, consume=consume, act="clamped", limit=limit)
            close(out, ref, dst, what=(m, inter, src))
            assert not consume or float(dev.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [1, 8, 100, 129, 300])
def test_clamped_gate_behind_its_product(dtype, m):
    """The sizes of every route: the persistent product's epilogue (whole tiles and strips of the last round), the cluster
    product's, split sums with the element-wise kernel, and sizes no epilogue takes."""
    from tiny_llm_b200 import ops
    from tiny_llm_b200.engine import Workspace
    from tiny_llm_b200.parts import interleave_gate_up
    from tiny_llm_b200.parts.feed_forward import gate_up_block
    g = torch.Generator().manual_seed(m)
    for k, inter in [(64, 128), (128, 384), (72, 40), (44, 28), (256, 2560), (64, 9856)]:
        if m < 300 and inter > 3000:
            continue
        a = torch.randn(m, k, generator=g).to(dtype)
        wg, wu = torch.randn(inter, k, generator=g).to(dtype) * 0.3, torch.randn(inter, k, generator=g).to(dtype) * 0.3
        block = gate_up_block(inter)
        w = interleave_gate_up(wg, wu, block).to(DEV)
        out = torch.empty(m, inter, dtype=dtype, device=DEV)
        ops.linear_swiglu(a.to(DEV), w, out, block, Workspace(torch.device(DEV)), act="clamped", limit=1.2)
        ref = pv.clamped_glu(a.double() @ wg.double().T, a.double() @ wu.double().T, 1.2)
        close(out, ref, dtype, what=(m, k, inter))
        ops.linear_swiglu(a.to(DEV), w, out, block, Workspace(torch.device(DEV)))      # SiLU by the same routes
        gp = a.double() @ wg.double().T
        close(out, gp * torch.sigmoid(gp) * (a.double() @ wu.double().T), dtype, what=("silu", m, k, inter))
    ops.check_status()


# ---------------------------------------------------------------------------------------------- filters, norms, cache write

CONV = [(4, 2, 16, 32, 4, 16), (6, 3, 10, 6, 2, 4), (2, 1, 24, 8, 1, 8), (3, 3, 40, 16, 5, 16), (5, 1, 7, 9, 6, 4), (16, 4, 64, 128, 4, 16),
        (8, 1, 128, 64, 3, 8)]


def conv_plain(x, taps, wq, wk, nqc, nkc, eps, before):
    """One request's projected rows `x` (bias added) behind kept inputs `before` through filter and norms."""
    y = pv.short_conv(torch.cat([before, x]), taps)[before.shape[0]:]
    q, k, v = y[:, :nqc], y[:, nqc:nqc + nkc], y[:, nqc + nkc:]
    return pv.rms_unit(q, eps) * wq, pv.rms_unit(k, eps) * wk, v


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,kd,vd,n,page", CONV)
def test_filters_whole_norms_and_cache_write(dtype, nq, nkv, kd, vd, n, page):
    """Steps of unequal requests one after the other: prompts, portions shorter than the filter, single tokens (alone in
    their step, which then also moves the kept inputs), and one step long enough for the tiles of several tokens."""
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(kd + vd)
    nqc, nkc, nvc = nq * kd, nkv * kd, nkv * vd
    c = nqc + nkc + nvc
    bias, taps = torch.randn(c, generator=g), torch.randn(c, n, generator=g) * 0.6
    wq, wk = torch.rand(nqc, generator=g) + 0.5, torch.rand(nkc, generator=g) + 0.5
    kept = torch.zeros(6, max(n - 1, 0), c, device=DEV)
    slots = [4, 0, 5]
    steps = [[5, 1, 9], [1, 2, 1], [1, 1, 1], [3, 1, 700], [1, 1, 1], [2, 2, 2]]
    total = [sum(s[r] for s in steps) for r in range(3)]
    pages = [-(-t // page) for t in total]
    order = torch.randperm(sum(pages) + 3, generator=g).tolist()
    tables = [[order.pop() for _ in range(p)] for p in pages]
    kc = torch.full((sum(pages) + 3, nkv, page, kd), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((sum(pages) + 3, nkv, page, vd), float("nan"), dtype=dtype, device=DEV)
    rows = [(torch.randn(t, c, generator=g) * 1.5).to(dtype) for t in total]
    refs = [conv_plain(rows[r].double() + bias.double(), taps.double(), wq.double(), wk.double(), nqc, nkc, 1e-4,
                       torch.zeros(n - 1, c, dtype=torch.float64)) for r in range(3)]
    extra = -(-(c + 3) // 8) * 8 - c                                         # columns behind q, k, v
    done = [0, 0, 0]
    untouched = kept[1].clone()
    for lens in steps:
        proj = torch.cat([torch.cat([rows[r][done[r]:done[r] + m], torch.full((m, extra), float("nan"), dtype=dtype)], dim=1)
                          for r, m in enumerate(lens)]).to(DEV)
        cu = [0, lens[0], lens[0] + lens[1], sum(lens)]
        where = [(r, done[r] + i) for r, m in enumerate(lens) for i in range(m)]
        batch = SimpleNamespace(cu_q=i32(cu), slots=i32(slots), num_requests=3, max_q_len=max(lens), token_request=i32([r for r, _ in where]))
        q_out = torch.empty(len(where), nqc, dtype=dtype, device=DEV)
        before = proj.clone()
        ops.conv_norm_kv_write(proj, batch, nq, nkv, kd, vd, kc, vc, i32([tables[r][p // page] * page + p % page for r, p in where]),
                               q_out, bias=bias.to(DEV), taps=taps.T.contiguous().to(DEV), kept=kept if n > 1 else None,
                               norm_q=wq.to(DEV), norm_k=wk.to(DEV), eps=1e-4)
        assert torch.equal(proj[:, :c], before[:, :c])
        for r, m in enumerate(lens):
            close(q_out[cu[r]:cu[r + 1]], refs[r][0][done[r]:done[r] + m], dtype, what=("q", r, lens))
            done[r] += m
            if n > 1:
                tail = torch.cat([torch.zeros(n - 1, c), rows[r][:done[r]].float() + bias])[-(n - 1):]
                assert torch.equal(kept[slots[r]].cpu(), tail), (r, lens)
    assert torch.equal(kept[1], untouched)                                    # no request's slot
    for r in range(3):
        for cache, ref, heads, d in ((kc, refs[r][1], nkv, kd), (vc, refs[r][2], nkv, vd)):
            got = torch.stack([cache[tables[r][p // page], :, p % page] for p in range(total[r])])
            close(got.reshape(total[r], heads * d), ref, dtype, what=("cache", r))


@pytest.mark.parametrize("nq,nkv,kd,vd,n", [(4, 2, 16, 32, 4), (6, 3, 10, 6, 2), (3, 1, 24, 8, 3)])
def test_filters_in_portions_give_the_same_bits(nq, nkv, kd, vd, n):
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(9)
    c, t, page = (nq + nkv) * kd + nkv * vd, 640, 16
    bias, taps = torch.randn(c, generator=g).to(DEV), (torch.randn(n, c, generator=g) * 0.6).to(DEV)
    wq, wk = torch.ones(nq * kd, device=DEV), torch.ones(nkv * kd, device=DEV)
    proj = torch.randn(t, -(-c // 8) * 8, generator=g).to(DEV)

    def run(cuts):
        kept = torch.zeros(2, n - 1, c, device=DEV)
        kc, vc = torch.zeros(t // page, nkv, page, kd, device=DEV), torch.zeros(t // page, nkv, page, vd, device=DEV)
        out = []
        for a, b in zip(cuts[:-1], cuts[1:]):
            batch = SimpleNamespace(cu_q=i32([0, b - a]), slots=i32([1]), num_requests=1, max_q_len=b - a, token_request=i32([0] * (b - a)))
            q = torch.empty(b - a, nq * kd, device=DEV)
            ops.conv_norm_kv_write(proj[a:b], batch, nq, nkv, kd, vd, kc, vc, i32(list(range(a, b))), q, bias=bias, taps=taps,
                                   kept=kept, norm_q=wq, norm_k=wk, eps=1e-6)
            out.append(q)
        return torch.cat(out), kc, vc, kept

    whole = run([0, t])
    for cuts in ([0, 2, 3, 30, t], [0, 1, 2, 4, 5, 8, 9, 17, 600, t], list(range(0, t + 1, 1))[:20] + [t]):
        assert all(torch.equal(x, y) for x, y in zip(whole, run(cuts))), cuts


# ---------------------------------------------------------------------------------------------- latent attention's pieces

@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_norm_rotation_in_halves_and_cache_write(dtype):
    from tiny_llm_b200 import ops
    from tiny_llm_b200.parts import pair_frequencies
    g = torch.Generator().manual_seed(6)
    for nq, nd, rd, rank, dims, page in [(3, 16, 16, 32, 16, 16), (5, 6, 10, 18, 6, 4), (1, 9, 2, 5, 2, 8), (4, 48, 64, 192, 64, 16), (2, 8, 12, 24, 0, 4)]:
        positions = [0, 1, 6, 7, 8, 15, 16, 700, 31999]
        t, kd = len(positions), rank + rd
        slots = [8, 9, 10, 20, 21, 1, 2, 3, 15]
        proj = torch.randn(t, nq * (nd + rd) + kd + 5, generator=g).to(dtype)
        wl = torch.rand(rank, generator=g) + 0.5
        freq = pair_frequencies(dims, 300.0).to(DEV) if dims else None
        kc = torch.zeros(24 // page + 8, 1, page, kd, dtype=dtype, device=DEV)
        vc = torch.zeros(24 // page + 8, 1, page, rank, dtype=dtype, device=DEV)
        for owner in (True, False):
            q_out = torch.zeros(t, nq, kd, dtype=dtype, device=DEV)
            args = (wl.to(DEV), 1e-5, q_out, kc, vc, i32(slots)) if owner else (None, 1e-5, q_out, None, None, None)
            ops.latent_kv_write(proj.to(DEV), i32(positions), nq, nd, rd, rank, dims, freq, *args, rot_pairs=False)
            q = proj.double()[:, :nq * (nd + rd)].view(t, nq, nd + rd)[..., nd:]
            pos = torch.tensor(positions)
            want = pv.rotate_halves(q, pos, dims, 300.0) if dims else q
            # (the engine's angle is the 32-bit product of position and frequency)
            close(q_out[..., rank:], want, dtype, f32=3e-3, what="queries")
            assert float(q_out[..., :rank].abs().max()) == 0.0
            small = [i for i, p in enumerate(positions) if p < 100]
            close(q_out[small][..., rank:], want[small], dtype, what="queries near the start")
        lat = proj.double()[:, nq * (nd + rd):]
        c = pv.rms_unit(lat[:, :rank], 1e-5) * wl.double()
        kr = pv.rotate_halves(lat[:, None, rank:kd], pos, dims, 300.0)[:, 0] if dims else lat[:, rank:kd]
        for i, s in enumerate(slots):
            close(vc[s // page, 0, s % page], c[i], dtype, what="value row")
            close(kc[s // page, 0, s % page, :rank], c[i], dtype, what="key row")
            close(kc[s // page, 0, s % page, rank:], kr[i], dtype, f32=2e-5 if positions[i] < 100 else 3e-3, what="rotated part")


@pytest.mark.parametrize("dtype", DTYPES)
def test_product_per_head_with_a_gate_per_value(dtype):
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(7)
    for t, heads, k, n in [(1, 3, 32, 24), (40, 2, 18, 14), (130, 4, 64, 80), (7, 5, 5, 11), (33, 1, 192, 128)]:
        a = torch.randn(t, heads, k, generator=g).to(dtype)
        w = (torch.randn(heads, n, k, generator=g) * 0.3).to(dtype)
        rows = (torch.randn(t, heads * n + 9, generator=g) * 2).to(dtype)        # the gate is a slice of wider rows
        gate = rows.to(DEV)[:, 3:3 + heads * n].view(t, heads, n)
        out = torch.empty(t, heads, n, dtype=dtype, device=DEV)
        ops.head_linear(a.to(DEV), w.to(DEV), out, gate=gate)
        ref = torch.einsum("thk,hnk->thn", a.double(), w.double()) * torch.sigmoid(rows.double()[:, 3:3 + heads * n].view(t, heads, n))
        close(out, ref, dtype, what=(t, heads))


# ---------------------------------------------------------------------------------------------- attention

def rel_tables(g, buckets, heads, far):
    from tiny_llm_b200.parts import distance_buckets
    rel = torch.randn(buckets, heads, generator=g) * 1.5
    tab = rel[torch.tensor(distance_buckets(buckets, far))].T.contiguous()
    return rel, tab.to(DEV), (tab.double() * 1.4426950408889634).float().contiguous().to(DEV)


def attend_plain(q, k, v, positions, scale, rel, far, window, keep, sink):
    """q [n, H, kd] at `positions`, k [T, G, kd], v [T, G, vd]: one row at a time from the definition."""
    heads, per = q.shape[1], q.shape[1] // k.shape[1]
    out = []
    for row, p in zip(q, positions):
        js = [j for j in range(p + 1) if window is None or p - j < window or j < keep]
        b = torch.tensor([pv.distance_bucket(p - j, rel.shape[0], far) for j in js])
        kk, vv = k[js].repeat_interleave(per, dim=1), v[js].repeat_interleave(per, dim=1)
        s = torch.einsum("hd,jhd->hj", row, kk) * scale + rel[b].T
        w = torch.softmax(torch.cat([s, sink[:, None]], dim=1), dim=1)[:, :-1]
        out.append(torch.einsum("hj,jhd->hd", w, vv))
    return torch.stack(out)


def paged(rows, table, page, pages):
    """rows [T, heads, d] -> cache [pages, heads, page, d] with position j in page table[j // page] (-1: given back)."""
    cache = torch.full((pages, rows.shape[1], page, rows.shape[2]), float("nan"), dtype=rows.dtype)
    for j in range(rows.shape[0]):
        if table[j // page] >= 0:
            cache[table[j // page], :, j % page] = rows[j]
    return cache


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep,page,length", [(None, 0, 16, 400), (150, 70, 16, 620), (24, 5, 8, 400), (3, 2, 4, 50), (20, 64, 16, 700),
                                                     (40, 65, 32, 500), (130, 1, 16, 900), (64, 128, 16, 1100)])
def test_window_with_kept_positions_finds_exactly_the_planted_keys(dtype, window, keep, page, length):
    """Keys are small but for one planted key per query position; it is the first position of the window, the one right
    before it, the last kept position, the first that is not kept, a page's first, or position 0.  Pages that hold
    neither kept positions nor the last window's are given back (-1 in the table, NaN elsewhere in the cache)."""
    from tiny_llm_b200 import ops
    from tiny_llm_b200.engine import Workspace
    g = torch.Generator().manual_seed(5)
    heads, kvh, kd, vd = 4, 2, 32, 32
    k = torch.randn(length, kvh, kd, generator=g) * 0.05
    v = torch.randn(length, kvh, vd, generator=g)
    n_pages = -(-length // page)
    table = torch.randperm(n_pages + 3, generator=g)[:n_pages].tolist()
    # every query stands at the end of the sequence or near it, so that one set of given-back pages fits them all
    qpos = list(range(max(0, length - 14), length))
    if window:
        low = qpos[0] - window + 1
        for i in range(-(-keep // page), max(0, low) // page):
            table[i] = -1
    plants, q = {}, torch.randn(len(qpos), heads, kd, generator=g) * 0.05
    for i, p in enumerate(qpos):
        first = max(0, p - window + 1) if window else 0
        options = [first, first - 1, keep - 1, keep, 0, (p // page) * page, p, max(first, p - 5)]
        target = options[i % len(options)]
        if not 0 <= target <= p or (window and table[target // page] < 0):
            target = p
        plants[p] = target
        direction = torch.zeros(kd)
        direction[i] = 1.0
        k[target, 0] += 9.0 * direction
        q[i, :2] += 6.0 * direction
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    scale, far = 1.3, 90.0
    rel, tab, tab2 = rel_tables(g, 12, heads, far)
    sink = torch.tensor([0.5, 300.0, -60.0, 1.5])
    ref = attend_plain(q.double(), k.double(), v.double(), qpos, scale, rel.double(), far, window, keep, sink.double())
    for i, p in enumerate(qpos):       # the planted key decides head 0 exactly when it is visible
        visible = not window or p - plants[p] < window or plants[p] < keep
        near = float((ref[i, 0] - v[plants[p], 0].double()).abs().max()) < 0.05
        assert near == visible, (p, plants[p])
    assert float(ref[:, 1].abs().max()) < 1e-8          # a huge sink takes everything
    kc, vc = paged(k, table, page, n_pages + 3).to(DEV), paged(v, table, page, n_pages + 3).to(DEV)
    tol = 2e-5 if dtype == torch.float32 else 2.0 ** -7 * float(ref.abs().max())
    n = len(qpos)
    bt = i32([table + [-1] * 5])
    alone = SimpleNamespace(token_request=i32(list(range(n))), positions=i32(qpos), cu_q=i32(list(range(n + 1))), q_start=i32(qpos),
                            num_requests=n, max_q_len=1, max_kv_len=length)
    portion = SimpleNamespace(token_request=i32([0] * n), positions=i32(qpos), cu_q=i32([0, n]), q_start=i32([qpos[0]]), num_requests=1,
                              max_q_len=n, max_kv_len=length)
    qd = torch.cat([q.reshape(n, -1), torch.zeros(n, 40, dtype=dtype)], dim=1).to(DEV)
    got = {}
    for name, batch, tables in (("decoded", alone, bt.repeat(n, 1).contiguous()), ("portion", portion, bt)):
        for generic in (True, False):
            for ws in (None, Workspace(torch.device(DEV))):
                for out_dtype in (torch.float32, dtype):
                    out = torch.empty(n, heads * vd, dtype=out_dtype, device=DEV)
                    ops.force_generic = generic
                    try:
                        ops.paged_attention_maps(qd, heads, kvh, 1, kd, vd, kc, vc, tables, batch, out, scale, window, None, sink=sink.to(DEV),
                                                 workspace=ws, keep_first=keep, rel=tab, rel_log2=tab2)
                    finally:
                        ops.force_generic = False
                    y = out.float().cpu().view(n, heads, vd)
                    assert torch.isfinite(y).all(), (name, generic)
                    bad = ((y - ref).abs().amax(dim=(1, 2)) > (tol if out_dtype == torch.float32 else 2 * tol)).nonzero().flatten().tolist()
                    assert not bad, (name, generic, ws is not None, out_dtype, [(qpos[i], plants[qpos[i]]) for i in bad])
                    got[name, generic, out_dtype] = y
    if dtype == torch.float32:
        assert torch.equal(got["decoded", True, dtype], got["portion", True, dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kd,vd,heads,kvh,window,keep,page,buckets,far", [
    (16, 32, 4, 2, 24, 9, 8, 8, 30.0), (48, 32, 6, 1, 150, 20, 16, 32, 100.0), (128, 96, 6, 1, None, 0, 16, 16, 64.0),
    (28, 18, 5, 1, 7, 11, 4, 6, 5.0), (64, 128, 8, 8, 50, 66, 16, 64, 200.0), (24, 40, 3, 3, 50, 0, 16, 2, 40.0),
    (80, 64, 16, 2, 33, 1, 32, 20, 10.5), (32, 16, 24, 2, 64, 64, 16, 32, 600.0)])
def test_bias_window_and_sink_for_portions_of_unequal_requests(dtype, kd, vd, heads, kvh, window, keep, page, buckets, far):
    """Four requests in one step: a portion that starts far inside a sequence and crosses window and page edges, a single
    decoded token, a prompt from position 0, and a portion of two tokens right behind the kept positions."""
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(kd + vd)
    spans = [(130, 97), (211, 1), (0, 75), (keep + 2, 2)]
    lengths = [a + n for a, n in spans]
    scale = 3.0 / kd ** 0.5
    rel, tab, tab2 = rel_tables(g, buckets, heads, far)
    sink = torch.randn(heads, generator=g) * 2
    total = sum(-(-n // page) for n in lengths) + 2
    order = torch.randperm(total, generator=g).tolist()
    kc = torch.full((total, kvh, page, kd), float("nan"), dtype=dtype)
    vc = torch.full((total, kvh, page, vd), float("nan"), dtype=dtype)
    refs, tables, qs = [], [], []
    for (a, n), length in zip(spans, lengths):
        k = (torch.randn(length, kvh, kd, generator=g) * 0.7).to(dtype)
        v = torch.randn(length, kvh, vd, generator=g).to(dtype)
        q = (torch.randn(n, heads, kd, generator=g) * 0.7).to(dtype)
        table = [order.pop() for _ in range(-(-length // page))]
        for j in range(length):
            kc[table[j // page], :, j % page] = k[j]
            vc[table[j // page], :, j % page] = v[j]
        refs.append(attend_plain(q.double(), k.double(), v.double(), range(a, a + n), scale, rel.double(), far, window, keep, sink.double()))
        tables.append(table), qs.append(q)
    ref, q = torch.cat(refs), torch.cat(qs)
    width = max(len(t) for t in tables) + 2
    cu = [0]
    for _, n in spans:
        cu.append(cu[-1] + n)
    batch = SimpleNamespace(token_request=i32([r for r, (_, n) in enumerate(spans) for _ in range(n)]),
                            positions=i32([p for a, n in spans for p in range(a, a + n)]), cu_q=i32(cu), q_start=i32([a for a, _ in spans]),
                            num_requests=len(spans), max_q_len=97)
    tol = 2e-5 if dtype == torch.float32 else 2.0 ** -7 * float(ref.abs().max())
    for generic in (True, False):
        out = torch.empty(cu[-1], heads * vd, dtype=torch.float32, device=DEV)
        ops.force_generic = generic
        try:
            ops.paged_attention_maps(q.reshape(cu[-1], -1).to(DEV), heads, kvh, 1, kd, vd, kc.to(DEV), vc.to(DEV),
                                     i32([t + [-1] * (width - len(t)) for t in tables]), batch, out, scale, window, None,
                                     sink=sink.to(DEV), keep_first=keep, rel=tab, rel_log2=tab2)
        finally:
            ops.force_generic = False
        got = out.cpu().view(cu[-1], heads, vd)
        assert torch.isfinite(got).all(), generic
        bad = ((got - ref).abs().amax(dim=(1, 2)) > tol).nonzero().flatten().tolist()
        assert not bad, (generic, bad[:8])


def test_the_three_launches_of_the_32_bit_attention_give_the_same_bits():
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(11)
    heads, kvh, kd, vd, page, length = 6, 2, 20, 28, 8, 900
    rel, tab, _ = rel_tables(g, 16, heads, 200.0)
    k, v = torch.randn(length, kvh, kd, generator=g), torch.randn(length, kvh, vd, generator=g)
    table = list(range(-(-length // page)))
    kc, vc = paged(k, table, page, len(table)).to(DEV), paged(v, table, page, len(table)).to(DEV)
    pos = list(range(0, length, 37)) + [length - 1]
    n = len(pos)
    batch = SimpleNamespace(token_request=i32([0] * n), positions=i32(pos), max_q_len=n)
    q = torch.randn(n, heads * kd, generator=g).to(DEV)
    outs = []
    for window, keep in ((None, 0), (100, 0), (100, 33), (10, 300)):
        outs.append([])
        for how in (1, 0, 2):
            out = torch.empty(n, heads * vd, device=DEV)
            ops.generic_attention_split = how
            try:
                ops.paged_attention_maps(q, heads, kvh, 1, kd, vd, kc, vc, i32([table]), batch, out, 0.3, window, None, keep_first=keep, rel=tab)
            finally:
                ops.generic_attention_split = None
            outs[-1].append(out)
        assert torch.equal(outs[-1][0], outs[-1][1]) and torch.equal(outs[-1][0], outs[-1][2]), (window, keep)
    assert not torch.equal(outs[1][0], outs[2][0])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kd,vd", [(320, 256), (576, 512), (72, 300), (1000, 33)])
def test_long_key_and_value_rows(dtype, kd, vd):
    """Rows beyond 256 values (a long latent with its rotated part) run on the CUDA cores."""
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(kd)
    heads, page, length = 5, 16, 150
    rel, tab, tab2 = rel_tables(g, 8, heads, 40.0)
    k, v = (torch.randn(length, 1, kd, generator=g) * 0.3).to(dtype), torch.randn(length, 1, vd, generator=g).to(dtype)
    table = list(range(-(-length // page)))
    kc, vc = paged(k, table, page, len(table)).to(DEV), paged(v, table, page, len(table)).to(DEV)
    pos = list(range(length))
    q = (torch.randn(length, heads, kd, generator=g) * 0.3).to(dtype)
    batch = SimpleNamespace(token_request=i32([0] * length), positions=i32(pos), cu_q=i32([0, length]), q_start=i32([0]), num_requests=1, max_q_len=length)
    out = torch.empty(length, heads * vd, dtype=torch.float32, device=DEV)
    sink = torch.zeros(heads)
    ops.paged_attention_maps(q.reshape(length, -1).to(DEV), heads, 1, 1, kd, vd, kc, vc, i32([table]), batch, out, 0.4, 60, None,
                             sink=sink.to(DEV), keep_first=3, rel=tab, rel_log2=tab2)
    ref = attend_plain(q.double(), k.double(), v.double(), pos, 0.4, rel.double(), 40.0, 60, 3, sink.double())
    close(out.view(length, heads, vd), ref, dtype)


@pytest.mark.parametrize("kd,vd,heads,kvh,window,keep", [(16, 32, 4, 2, None, 0), (128, 96, 6, 1, 150, 70), (80, 48, 8, 1, 600, 0), (32, 16, 5, 5, 200, 130)])
def test_decoded_tokens_with_the_keys_in_runs_match_one_run(kd, vd, heads, kvh, window, keep):
    from tiny_llm_b200 import ops
    from tiny_llm_b200.engine import Workspace
    g = torch.Generator().manual_seed(17)
    page, contexts = 16, [1, 40, 300, 1500, 65]
    r = len(contexts)
    per = -(-max(contexts) // page)
    table = torch.arange(r * per, dtype=torch.int32).view(r, per)
    kc = (torch.randn(r * per, kvh, page, kd, generator=g) * 0.5).to(torch.bfloat16).to(DEV)
    vc = torch.randn(r * per, kvh, page, vd, generator=g).to(torch.bfloat16).to(DEV)
    q = torch.randn(r, heads * kd + 8, generator=g).to(torch.bfloat16).to(DEV)
    sink = torch.randn(heads, generator=g).to(DEV)
    _, tab, tab2 = rel_tables(g, 16, heads, 80.0)
    batch = SimpleNamespace(cu_q=i32(list(range(r + 1))), q_start=i32([c - 1 for c in contexts]), num_requests=r, max_q_len=1,
                            max_kv_len=2048, token_request=i32(list(range(r))), positions=i32([c - 1 for c in contexts]))
    for sk in (sink, None):
        one, runs = torch.empty(r, heads * vd, device=DEV), torch.empty(r, heads * vd, device=DEV)
        half = torch.empty(r, heads * vd, dtype=torch.bfloat16, device=DEV)
        kw = dict(sink=sk, keep_first=keep, rel=tab, rel_log2=tab2)
        ops.paged_attention_maps(q, heads, kvh, 1, kd, vd, kc, vc, table.to(DEV), batch, one, 0.2, window, None, **kw)
        ws = Workspace(torch.device(DEV))
        ops.paged_attention_maps(q, heads, kvh, 1, kd, vd, kc, vc, table.to(DEV), batch, runs, 0.2, window, None, workspace=ws, **kw)
        assert ws.buffers(), "the keys were not cut into runs"
        ops.paged_attention_maps(q, heads, kvh, 1, kd, vd, kc, vc, table.to(DEV), batch, half, 0.2, window, None, workspace=ws, **kw)
        assert float((one - runs).abs().max()) <= 4e-6 * max(1.0, float(one.abs().max()))
        assert torch.equal(half, runs.to(torch.bfloat16))


def test_output_bias_and_depth_average_behind_other_blocks():
    """An attention with an output bias in a pre_norm block adds it itself, and a depth average behind blocks that do not
    take it runs as a kernel of its own."""
    from tiny_llm_b200.config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
    from tiny_llm_b200.engine import StepEntry, make_runner
    from tiny_llm_b200.parts import DecoderModel
    from tiny_llm_b200.weights import random_state
    norm = PartSpec("rms_norm", {"size": 32, "eps": 1e-5, "weight_suffix": ""})
    mix = PartSpec("sink_attention", {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "key_dim": 16, "value_dim": 16, "scale": 0.25,
                                      "eps": 1e-5, "bias": True, "qk_norm": "whole", "sink": True, "gate": False, "conv": 3,
                                      "bias_max": 20.0, "window": 12, "keep_first": 2, "out_bias": True})
    layers = [LayerSpec(f"l{i}.", norm1=norm, mixer=mix, mixer_prefix="mix.", norm1_name="norm1") for i in range(3)]
    spec = ModelSpec("x", 50, 32, 256, layers, [LayerCall(i) for i in range(3)], norm, embed_name="embed", final_norm_name="fn",
                     lm_head_name="head", depth_average="dwa", embedding_scale=3.0)
    model = DecoderModel(spec)
    w = random_state(model.weight_specs(), 5, 0.2, torch.float32)
    model.load({k: t.to(DEV) for k, t in w.items()})
    runner = make_runner(model, "float32", DEV, max_tokens=64, page_size=8, max_requests=2)
    toks = torch.randint(0, 50, (41,), generator=torch.Generator().manual_seed(2)).tolist()
    runner.cache.add_request("a")
    got = [runner.step([StepEntry("a", toks[:30], list(range(30)))]).cpu().clone()]
    for t in toks[30:]:
        got.append(runner.step([StepEntry("a", [t], [0])]).cpu().clone())
    m = {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.25, "bias_max": 20.0, "mask": {"size": 12, "keep_first": 2}}
    wd = {k: t.double() for k, t in w.items()}
    x = wd["embed"][toks] * 3.0
    stages = [x]
    for i in range(3):
        x = x + pv.attention(m, wd, f"l{i}.mix.", pv.rms_unit(x, 1e-5) * wd[f"l{i}.norm1"], 1e-5, pv.no_quant)
        stages.append(x)
        x = pv.depth_average(stages, wd[f"l{i}.dwa"])
    ref = (pv.rms_unit(x, 1e-5) * wd["fn"]) @ wd["head"].T
    close(torch.cat(got), ref, torch.float32)
