"""Each new mechanism alone on the GPU against the plain implementation: layer norms without biases, the norm behind a
branch with the next norm taken along, the tanh form of GELU as a gate (element-wise and by every route of its product),
norms over all heads with a rotation behind them and the cache write, attention over a window with a sink (planted keys
at the window's edges, at page borders and on the first positions, rows rounded by the kernel), the router's groups,
renormalised weights and identity experts, SiLU * up inside the grouped products, the combine, and the soft cap."""
from types import SimpleNamespace

import pytest
import torch

import plain_lovapel as pl

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, ref, dtype, f32=2e-5, what=""):
    tol = f32 * max(1.0, float(ref.abs().max())) if dtype == torch.float32 else 2.0 ** -7 * float(ref.abs().max())
    worst = float((got.double().cpu() - ref.double()).abs().max())
    assert worst <= tol, (what, worst, tol)


# ---------------------------------------------------------------------------------------------- norms

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,h", [(1, 4), (5, 64), (33, 200), (3, 50), (7, 1), (2, 2048), (4, 5120), (2, 8192), (3, 9000), (150, 1028)])
def test_norm_behind_a_branch_takes_the_next_norm_along(dtype, n, h):
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(h)
    x, branch = torch.randn(n, h, generator=g) * 2 + 3, torch.randn(n, h, generator=g) * 5 - 20
    w, b, w2, b2 = (torch.rand(h, generator=g) + 0.5 for _ in range(4))
    for bias, bias2 in ((None, None), (b, None), (None, b2)):
        dev = lambda v: None if v is None else v.to(DEV)
        ref = x.double() + pl.layer_norm(branch.double(), w.double(), 1e-3) + (0 if bias is None else bias.double())
        plain = (x.to(DEV), branch.to(DEV))
        ops.layer_norm_add(plain[1], plain[0], dev(w), dev(bias), 1e-3)
        close(plain[0], ref, torch.float32, what="stream")
        assert float(plain[1].abs().max()) == 0.0           # handed back zeroed
        taken, copy = (x.to(DEV), branch.to(DEV)), torch.empty(n, h, dtype=torch.bfloat16, device=DEV)
        out = torch.full((n, h), float("nan"), dtype=dtype, device=DEV)
        ops.layer_norm_add(taken[1], taken[0], dev(w), dev(bias), 1e-3, copy=copy, then=(dev(w2), dev(bias2), 1e-4), out=out)
        assert torch.equal(taken[0], plain[0]) and torch.equal(taken[1], plain[1]) and torch.equal(copy, plain[0].to(torch.bfloat16))
        alone = torch.empty_like(out)
        ops.layer_norm(plain[0], dev(w2), dev(bias2), 1e-4, alone)
        assert torch.equal(out, alone)                       # the bits do not depend on which kernel took the norm
        close(out, pl.layer_norm(plain[0].double().cpu(), w2.double(), 1e-4) + (0 if bias2 is None else bias2.double()), dtype, what="next norm")
    rows = torch.randint(0, n, (n + 2,), generator=g)
    out = torch.empty(n + 2, h, dtype=dtype, device=DEV)
    ops.layer_norm(x.to(DEV), w.to(DEV), None, 1e-3, out, i32(rows.tolist()))
    close(out, pl.layer_norm(x.double()[rows], w.double(), 1e-3), dtype, what="wanted rows")


def test_layer_norm_part_adds_and_hands_on():
    from tiny_llm_b200.engine import Workspace
    from tiny_llm_b200.parts import LayerNorm, RMSNorm
    g = torch.Generator().manual_seed(2)
    x, branch, w, w2 = torch.randn(5, 64, generator=g), torch.randn(5, 64, generator=g), torch.rand(64, generator=g), torch.rand(64, generator=g)
    for dtype in DTYPES:
        ctx = SimpleNamespace(workspace=Workspace(torch.device(DEV)), dtype=dtype)
        norm, after, other = LayerNorm(64, 1e-5, has_bias=False), LayerNorm(64, 1e-4, has_bias=False), RMSNorm(64, 1e-5)
        norm.load("a", {"a": w.to(DEV)}), after.load("b", {"b": w2.to(DEV)})
        assert [s.name for s in norm.weight_specs("a")] == ["a"]
        stream = x.to(DEV)
        h = norm.add_into(ctx, branch.to(DEV), stream, then=after)
        ref = x.double() + pl.layer_norm(branch.double(), w.double(), 1e-5)
        close(stream, ref, torch.float32)
        close(h, pl.layer_norm(ref, w2.double(), 1e-4), dtype)
        assert norm.add_into(ctx, branch.to(DEV), stream, then=other) is None and norm.add_into(ctx, branch.to(DEV), stream) is None


# ---------------------------------------------------------------------------------------------- feed-forward

def test_tanh_gelu_gate_alone():
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(4)
    for m, inter, block in [(3, 24, 8), (5, 128, 128), (2, 20, 4), (7, 21, 1), (200, 256, 128)]:
        gate, up = torch.randn(m, inter, generator=g) * 2, torch.randn(m, inter, generator=g) * 3
        gate[0, 0], gate[0, 1], gate[0, 2], gate[0, 3] = 300.0, -300.0, 1e-4, -4.5
        both = torch.stack([gate.view(m, -1, block), up.view(m, -1, block)], dim=2).reshape(m, 2 * inter)
        for src, dst, consume in ((torch.float32, torch.float32, False), (torch.float32, torch.bfloat16, True),
                                  (torch.bfloat16, torch.bfloat16, False), (torch.float32, torch.bfloat16, False)):
            q = both.to(src)
            gq = q.view(m, -1, 2, block).double()
            ref = (pl.gelu_tanh(gq[:, :, 0]) * gq[:, :, 1]).reshape(m, inter)
            dev, out = q.to(DEV), torch.empty(m, inter, dtype=dst, device=DEV)
            ops.silu_mul(dev, out, block, consume=consume, act="gelu_tanh")
            close(out[1:], ref[1:], dst, what=(m, inter, src))
            close(out[0, 1:], ref[0, 1:], dst, what="extremes")
            close(out[:1, :1], ref[:1, :1], dst, what="large")
            assert not consume or float(dev.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [1, 8, 100, 129, 300])
def test_tanh_gelu_gate_behind_its_product(dtype, m):
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
        ops.linear_swiglu(a.to(DEV), w, out, block, Workspace(torch.device(DEV)), act="gelu_tanh")
        close(out, pl.gelu_tanh(a.double() @ wg.double().T) * (a.double() @ wu.double().T), dtype, what=(m, k, inter))
    ops.check_status()


def test_soft_cap():
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(3)
    for shape in [(1, 1), (3, 97), (5, 128), (64, 1001)]:
        x = torch.randn(*shape, generator=g) * 40
        for scale, cap in ((1.0, 30.0), (0.37, 2.5), (-2.0, 15.0), (3.0, None)):
            y = x.to(DEV)
            ops.soft_cap(y, scale, cap)
            z = x.double() * scale
            close(y, z if cap is None else cap * torch.tanh(z / cap), torch.float32, f32=4e-7, what=(shape, scale, cap))
    with pytest.raises(ops.KernelError):
        ops.soft_cap(y, 1.0, -1.0)


# ---------------------------------------------------------------------------------------------- whole norms, rotation, cache write

PREP = [(4, 2, 16, 32, 8, 16), (6, 3, 10, 6, 10, 4), (2, 1, 24, 8, 24, 8), (3, 3, 40, 16, 4, 16), (5, 1, 7, 9, 6, 4), (16, 4, 64, 128, 64, 16),
        (8, 1, 128, 64, 20, 8), (1, 1, 8, 8, 2, 4)]


def rotate_pairs(x, pos, dims, base):
    """x [T, heads, D]: values 2i and 2i + 1 by pos * base^(-2i / dims)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    a = pos.double()[:, None, None] * base ** (-2.0 * i / dims)
    out = x.clone()
    out[..., 0:dims:2] = x[..., 0:dims:2] * torch.cos(a) - x[..., 1:dims:2] * torch.sin(a)
    out[..., 1:dims:2] = x[..., 1:dims:2] * torch.cos(a) + x[..., 0:dims:2] * torch.sin(a)
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nq,nkv,kd,vd,dims,page", PREP)
def test_whole_norms_rotation_and_cache_write(dtype, nq, nkv, kd, vd, dims, page):
    """Two requests' tokens at scattered positions, in few tokens and in enough for the tiles of several; the norm takes
    all heads of a token at once, and heads differ in size by far, so that a norm per head shows."""
    from tiny_llm_b200 import ops
    from tiny_llm_b200.parts import pair_frequencies
    g = torch.Generator().manual_seed(kd + vd)
    nqc, nkc, nvc = nq * kd, nkv * kd, nkv * vd
    c = nqc + nkc + nvc
    wq, wk = torch.rand(nqc, generator=g) + 0.5, torch.rand(nkc, generator=g) + 0.5
    freq = pair_frequencies(dims, 300.0)
    for t in (1, 9, 700):
        rows = torch.randn(t, c, generator=g) * torch.exp(torch.randn(t, c, generator=g) * 0.5)
        rows[:, :kd] *= 6.0
        rows = rows.to(dtype)
        positions = torch.randint(0, 90, (t,), generator=g)
        positions[0] = 0
        slots = torch.randperm(t + 7, generator=g)[:t].tolist()
        pages = -(-(t + 7) // page)
        proj = torch.cat([rows, torch.full((t, -(-(c + 3) // 8) * 8 - c), float("nan"), dtype=dtype)], dim=1).to(DEV)
        half = t // 2
        batch = SimpleNamespace(cu_q=i32([0, half, t]), slots=i32([0, 1]), num_requests=2, max_q_len=t, positions=i32(positions.tolist()),
                                token_request=i32([0] * half + [1] * (t - half)))
        for pairs in (False, True):
            for mag in (1.0, 1.25):
                kc = torch.full((pages, nkv, page, kd), float("nan"), dtype=dtype, device=DEV)
                vc = torch.full((pages, nkv, page, vd), float("nan"), dtype=dtype, device=DEV)
                q = torch.empty(t, nqc, dtype=dtype, device=DEV)
                ops.conv_norm_kv_write(proj, batch, nq, nkv, kd, vd, kc, vc, i32(slots), q, norm_q=wq.to(DEV), norm_k=wk.to(DEV),
                                       eps=1e-4, freq=freq.to(DEV), rot_pairs=pairs, rot_mag=mag)
                turn = rotate_pairs if pairs else pl.rotate_halves

                def want(x, w, heads):
                    y = turn(pl.rms_norm(x.double(), w.double(), 1e-4).view(t, heads, kd), positions, dims, 300.0)
                    y[..., :dims] *= mag
                    return y
                close(q, want(rows[:, :nqc], wq, nq).reshape(t, nqc), dtype, what=("q", t, pairs))
                at = torch.tensor(slots)
                close(kc.transpose(1, 2).reshape(-1, nkv, kd)[at], want(rows[:, nqc:nqc + nkc], wk, nkv), dtype, what=("k", t, pairs))
                close(vc.transpose(1, 2).reshape(-1, nkv, vd)[at], rows[:, nqc + nkc:].double().view(t, nkv, vd), dtype, what=("v", t))
        # every token alone: the same bits
        one = torch.empty(1, nqc, dtype=dtype, device=DEV)
        for i in {0, t // 2, t - 1}:
            single = SimpleNamespace(cu_q=i32([0, 1]), slots=i32([1]), num_requests=1, max_q_len=1, positions=i32([int(positions[i])]), token_request=i32([0]))
            kc2, vc2 = kc.clone(), vc.clone()
            ops.conv_norm_kv_write(proj[i:i + 1], single, nq, nkv, kd, vd, kc2, vc2, i32([slots[i]]), one, norm_q=wq.to(DEV),
                                   norm_k=wk.to(DEV), eps=1e-4, freq=freq.to(DEV), rot_pairs=True, rot_mag=1.25)
            if dtype == torch.float32:
                assert torch.equal(one[0], q[i]) and torch.equal(kc2.nan_to_num(9.0), kc.nan_to_num(9.0)), i
            else:
                close(one[0], q[i].double().cpu(), dtype, what=i)


def test_rotation_behind_filters_and_norms():
    """The same kernel with a filter of several taps: filter, then norm, then rotation."""
    from tiny_llm_b200 import ops
    from tiny_llm_b200.parts import pair_frequencies
    g = torch.Generator().manual_seed(8)
    for nq, nkv, kd, vd, n in [(4, 2, 16, 8, 4), (3, 1, 10, 6, 3)]:
        t, c = 650, (nq + nkv) * kd + nkv * vd
        x, taps = torch.randn(t, c, generator=g), torch.randn(n, c, generator=g)
        padded = torch.cat([torch.zeros(n - 1, c), x]).double()
        y = sum(padded[j:j + t] * taps[j].double() for j in range(n))
        pos = torch.arange(t)
        ref = pl.rotate_halves(pl.rms_norm(y[:, :nq * kd], torch.ones(nq * kd), 1e-5).view(t, nq, kd), pos, 8, 50.0).reshape(t, -1)
        batch = SimpleNamespace(cu_q=i32([0, t]), slots=i32([0]), num_requests=1, max_q_len=t, positions=i32(pos.tolist()), token_request=i32([0] * t))
        kc, vc = torch.zeros(t, nkv, 1, kd, device=DEV), torch.zeros(t, nkv, 1, vd, device=DEV)
        q = torch.empty(t, nq * kd, device=DEV)
        ops.conv_norm_kv_write(x.to(DEV), batch, nq, nkv, kd, vd, kc, vc, i32(list(range(t))), q, taps=taps.to(DEV),
                               kept=torch.zeros(1, n - 1, c, device=DEV), norm_q=torch.ones(nq * kd, device=DEV),
                               norm_k=torch.ones(nkv * kd, device=DEV), eps=1e-5, freq=pair_frequencies(8, 50.0).to(DEV))
        # (the engine's angle is the 32-bit product of position and frequency: 650 * 2^-24 of a radian)
        close(q, ref, torch.float32, f32=1e-4)


# ---------------------------------------------------------------------------------------------- attention

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,page,length,kd,vd", [(None, 16, 400, 32, 32), (72, 16, 620, 64, 48), (24, 8, 400, 32, 16), (3, 4, 50, 20, 12),
                                                      (1, 16, 100, 32, 32), (64, 16, 700, 16, 64), (65, 32, 500, 48, 32), (130, 16, 900, 128, 96)])
def test_window_and_sink_find_exactly_the_planted_keys(dtype, window, page, length, kd, vd):
    """One planted key per query position: the window's first, the one right before it, a page's first, position 0, the
    token itself.  Pages behind the last window are given back (-1 in the table, NaN elsewhere in the cache).  As decoded
    tokens and as a portion, rows in 32-bit and rounded by the kernel."""
    from tiny_llm_b200 import ops
    from tiny_llm_b200.engine import Workspace
    g = torch.Generator().manual_seed(5)
    heads, kvh = 4, 2
    k, v = torch.randn(length, kvh, kd, generator=g) * 0.05, torch.randn(length, kvh, vd, generator=g)
    n_pages = -(-length // page)
    table = torch.randperm(n_pages + 3, generator=g)[:n_pages].tolist()
    qpos = list(range(max(0, length - 14), length))
    if window:
        for i in range(max(0, qpos[0] - window + 1) // page):
            table[i] = -1
    plants, q = {}, torch.randn(len(qpos), heads, kd, generator=g) * 0.05
    for i, p in enumerate(qpos):
        first = max(0, p - window + 1) if window else 0
        options = [first, first - 1, 0, (p // page) * page, p, max(first, p - 5), first - 1, first]
        target = options[i % len(options)]
        if not 0 <= target <= p or table[target // page] < 0:
            target = p
        plants[p] = target
        k[target, 0, i % kd] += 9.0
        q[i, :2, i % kd] += 6.0
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    scale, sink = 1.3, torch.tensor([0.5, 300.0, -60.0, 1.5])
    ref = pl.window_sink_attention(q.double(), k.double(), v.double(), torch.tensor(qpos), torch.arange(length), scale, sink.double(), window)
    for i, p in enumerate(qpos):       # the planted key decides head 0 exactly when it is visible
        near = float((ref[i, 0] - v[plants[p], 0].double()).abs().max()) < 0.05
        assert near == (not window or p - plants[p] < window), (p, plants[p])
    assert float(ref[:, 1].abs().max()) < 1e-8          # a huge sink takes everything
    caches = []
    for rows in (k, v):
        cache = torch.full((n_pages + 3, kvh, page, rows.shape[2]), float("nan"), dtype=dtype)
        for j in range(length):
            if table[j // page] >= 0:
                cache[table[j // page], :, j % page] = rows[j]
        caches.append(cache.to(DEV))
    n, bt = len(qpos), i32([table + [-1] * 5])
    alone = SimpleNamespace(token_request=i32(list(range(n))), positions=i32(qpos), cu_q=i32(list(range(n + 1))), q_start=i32(qpos),
                            num_requests=n, max_q_len=1, max_kv_len=length)
    portion = SimpleNamespace(token_request=i32([0] * n), positions=i32(qpos), cu_q=i32([0, n]), q_start=i32([qpos[0]]), num_requests=1,
                              max_q_len=n, max_kv_len=length)
    tol = 2e-5 if dtype == torch.float32 else 2.0 ** -7 * float(ref.abs().max())
    qd = q.reshape(n, -1).to(DEV)
    for name, batch, tables in (("decoded", alone, bt.repeat(n, 1).contiguous()), ("portion", portion, bt)):
        for generic in (True, False):
            for ws in (None, Workspace(torch.device(DEV))):
                for out_dtype in (torch.float32, dtype):
                    out = torch.empty(n, heads * vd, dtype=out_dtype, device=DEV)
                    ops.force_generic = generic
                    try:
                        ops.paged_attention_maps(qd, heads, kvh, 1, kd, vd, *caches, tables, batch, out, scale, window, None,
                                                 sink=sink.to(DEV), workspace=ws)
                    finally:
                        ops.force_generic = False
                    y = out.float().cpu().view(n, heads, vd)
                    assert torch.isfinite(y).all(), (name, generic)
                    bad = ((y - ref).abs().amax(dim=(1, 2)) > (tol if out_dtype == torch.float32 else 2 * tol)).nonzero().flatten().tolist()
                    assert not bad, (name, generic, ws is not None, out_dtype, [(qpos[i], plants[qpos[i]]) for i in bad])


# ---------------------------------------------------------------------------------------------- experts

@pytest.mark.parametrize("t,n,top,groups,keep", [(9, 6, 2, 3, 1), (70, 40, 5, 8, 3), (3, 3, 3, 1, 1), (33, 14, 3, 2, 1), (5, 7, 1, 7, 1), (40, 512, 8, 64, 5),
                                                 (6, 512, 40, 512, 100), (21, 48, 33, 4, 3), (4, 1, 1, 1, 1)])
@pytest.mark.parametrize("shift", [0.0, -3.0])
def test_router_groups_and_renormalised_weights(t, n, top, groups, keep, shift):
    """`shift` -3: every choice score is negative, so a score that counts as 0 outside the kept groups would win."""
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(n + top)
    z = torch.randn(t, n + 3, generator=g) * 2                        # further columns are ignored
    corr = torch.randn(n, generator=g) * 0.2 + shift
    ids, w = torch.empty(t, top, dtype=torch.int32, device=DEV), torch.empty(t, top, device=DEV)
    ops.moe_route(z.to(DEV), n, corr.to(DEV), 1.0, ids, w, softmax=True, renorm=True, groups=groups, keep=keep)
    rid, rw = pl.route(z[:, :n].double(), corr.double(), top, groups, keep)
    assert torch.equal(ids.cpu().long(), rid)
    close(w, rw, torch.float32, f32=2e-6)
    assert float((w.sum(dim=1) - 1).abs().max()) < 1e-5
    ops.moe_route(z.to(DEV), n, corr.to(DEV), 2.5, ids, w, softmax=True, groups=groups, keep=keep)     # not renormalised
    close(w, 2.5 * torch.gather(torch.softmax(z[:, :n].double(), dim=1), 1, rid), torch.float32, f32=2e-6)
    ops.moe_route(z.to(DEV), n, corr.to(DEV), 2.5, ids, w, softmax=True, renorm=True, groups=groups, keep=keep)
    close(w, 2.5 * rw, torch.float32, f32=2e-6)


def test_router_refuses_more_choices_than_the_groups_hold():
    from tiny_llm_b200 import ops
    z, ids, w = torch.zeros(2, 12, device=DEV), torch.empty(2, 5, dtype=torch.int32, device=DEV), torch.empty(2, 5, device=DEV)
    for groups, keep in ((3, 1), (5, 2), (3, 4), (3, 0)):
        with pytest.raises(ops.KernelError, match="groups"):
            ops.moe_route(z, 12, None, 1.0, ids, w, softmax=True, groups=groups, keep=keep)


def gated(x, wg, wu):
    y = x @ wg.T
    return y * torch.sigmoid(y) * (x @ wu.T)


@pytest.mark.parametrize("tile", [16, 64, 128])
@pytest.mark.parametrize("k,f", [(64, 40), (72, 128), (40, 8), (128, 256), (256, 200), (64, 12)])
def test_gate_inside_the_grouped_product(tile, k, f):
    from tiny_llm_b200 import ops
    from tiny_llm_b200.parts import interleave_gate_up
    from tiny_llm_b200.parts.feed_forward import gate_up_block
    g = torch.Generator().manual_seed(k + f)
    experts, t, top = 5, 61, 3
    x = torch.randn(t, k, generator=g).to(torch.bfloat16)
    wg, wu = ((torch.randn(experts, f, k, generator=g) * 0.3).to(torch.bfloat16) for _ in range(2))
    block = gate_up_block(f)
    w = torch.stack([interleave_gate_up(wg[e], wu[e], block) for e in range(experts)]).to(DEV)
    ids = torch.stack([torch.randperm(experts + 2, generator=g)[:top] for _ in range(t)]).to(torch.int32)     # two identity experts
    ref = torch.stack([gated(x[i].double(), wg[e].double(), wu[e].double()) if e < experts else torch.zeros(f, dtype=torch.float64)
                       for i in range(t) for e in ids[i].tolist()])
    real = (ids.flatten() < experts)
    tiles = ops.moe_max_tiles(t * top, experts, tile)
    rows, texp = torch.empty(tiles * tile, dtype=torch.int32, device=DEV), torch.empty(tiles, dtype=torch.int32, device=DEV)
    pos = torch.empty(t * top, dtype=torch.int32, device=DEV)
    ops.moe_align(ids.to(DEV), experts, tile, rows, texp, pos)
    assert torch.equal(pos.cpu() < 0, ~real) and sorted(r for r in rows.tolist() if r >= 0) == real.nonzero().flatten().tolist()
    out = torch.full((t * top, f), float("nan"), dtype=torch.bfloat16, device=DEV)
    xd = x.to(DEV)
    assert ops.moe_silu_up_fused(xd, w)
    ops.moe_linear(xd, w, rows, texp, tile, out, rows_per_input=top, silu_up_block=block)
    assert torch.isnan(out.cpu()[~real].float()).all()             # rows of identity experts are not touched
    close(out.cpu()[real], ref[real], torch.bfloat16, what="mma")
    if tile == 128 and f % 128 == 0:
        grouped, act = torch.empty(tiles * 128, k, dtype=torch.bfloat16, device=DEV), torch.zeros(tiles * 128, f, dtype=torch.bfloat16, device=DEV)
        ops.moe_gather(xd, rows, texp, 128, grouped, rows_per_input=top)
        ops.moe_linear_tc(grouped, w, texp, act, silu_up=True)
        close(act.cpu()[pos.cpu().long()[real]], ref[real], torch.bfloat16, what="tcgen05")
        ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 44, 1028, 7])
def test_combine_with_identity_experts(dtype, width):
    from tiny_llm_b200 import ops
    g = torch.Generator().manual_seed(width)
    t, top, experts = 37, 3, 4
    h = torch.randn(t, width + 4, generator=g).to(dtype)
    ids = torch.randint(0, experts + 3, (t, top), generator=g)
    ids[0] = torch.tensor([experts, experts + 1, experts + 2])
    w, y, resid = torch.rand(t, top, generator=g), torch.randn(t * top, width, generator=g), torch.randn(t, width, generator=g)
    rows = torch.where((ids < experts)[..., None], y.view(t, top, width).double(), h[:, None, :width].double())
    ref = resid.double() + (w[..., None].double() * rows).sum(dim=1)
    real = (ids < experts).flatten()
    y[~real] = float("nan")
    for h_dev in (h.to(DEV)[:, :width], h[:, :width].contiguous().to(DEV)):
        out = resid.to(DEV)
        ops.moe_combine(y.to(DEV), w.to(DEV), None, None, 0, out, ids=ids.to(torch.int32).to(DEV), num_experts=experts, h=h_dev)
        close(out, ref, torch.float32, f32=2e-6)
    order = torch.randperm(t * top, generator=g)                    # y in another order, found through pair_pos
    shuffled = torch.empty_like(y)
    shuffled[order] = y
    pos = torch.where(real, order, torch.full_like(order, -1)).to(torch.int32)
    out = resid.to(DEV)
    ops.moe_combine(shuffled.to(DEV), w.to(DEV), None, None, 0, out, pos.to(DEV), ids=ids.to(torch.int32).to(DEV), num_experts=experts, h=h_dev)
    close(out, ref, torch.float32, f32=2e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [dict(width=64, experts=6, identity=2, top=3, ff=48, shared=40, groups=(4, 2)), dict(width=72, experts=4, identity=4, top=2, ff=128, shared=None, groups=(2, 1)),
                                  dict(width=44, experts=5, identity=0, top=2, ff=10, shared=14, groups=None), dict(width=128, experts=1, identity=5, top=6, ff=256, shared=128, groups=None)])
@pytest.mark.parametrize("t", [1, 7, 200])
def test_experts_part(dtype, case, t, monkeypatch):
    """The whole part by each of its routes against the plain mixture; the choice is what the engine's own router made of
    its 32-bit logits wherever two choice scores are closer than the storage type resolves."""
    from tiny_llm_b200 import ops
    from tiny_llm_b200.engine import Workspace
    from tiny_llm_b200.parts import RoutedExperts
    g = torch.Generator().manual_seed(case["width"] + t)
    gr = case["groups"] or (1, 1)
    part = RoutedExperts(case["width"], case["experts"], case["top"], case["ff"], router="softmax", glu="silu", renorm=True, groups=gr[0], keep=gr[1],
                         identity=case["identity"], shared_size=case["shared"], shared_gate=False)
    w = {}
    for s in part.weight_specs("m."):
        v = torch.randn(*s.shape, generator=g) * (0.15 if len(s.shape) == 2 else 0.1)
        w[s.name] = v.to(dtype).float() if len(s.shape) == 2 else v
    part.load("m.", {n: (v.to(dtype) if v.dim() == 2 else v).to(DEV) for n, v in w.items()})
    h = torch.randn(t, case["width"], generator=g).to(dtype)
    n = case["experts"] + case["identity"]
    s = torch.softmax(h.double() @ w["m.router"].double().T, dim=1) + w["m.correction"].double()
    srt = s.sort(dim=1).values
    clear = torch.ones(t, dtype=torch.bool) if n == 1 else (srt[:, 1:] - srt[:, :-1]).min(dim=1).values > 1e-6
    assert clear.float().mean() > 0.9
    mlp = {"router": {"experts": case["experts"], "identity": case["identity"], "top": case["top"], "groups": {"count": gr[0], "keep": gr[1]}},
           "shared": {"ff": case["shared"]} if case["shared"] else None}
    ref = 0.25 + pl.expert_ff(h.double(), lambda name: w[name].double(), "m.", mlp)
    for rows in (0, 1):                                      # 1: every step with a pair per expert takes the contiguous order
        monkeypatch.setattr(ops, "moe_tc_rows_per_expert", rows)
        ctx = SimpleNamespace(workspace=Workspace(torch.device(DEV)), dtype=dtype)
        out = torch.full((t, case["width"]), 0.25, device=DEV)
        part.forward(ctx, h.to(DEV), out)
        close(out.cpu()[clear], ref[clear], dtype, what=(rows, case))
    ops.check_status()
