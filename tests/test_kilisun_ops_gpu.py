"""The mechanisms of the Kilisun design one at a time: each part or kernel against the plain function of the same
mechanism (float64 on the CPU), in packed batches of unequal requests, in portions down to one token, with pages in a
poisoned pool that are given back behind windows and used again, and with state slots that pass from one request to the
next.  Where random numbers would hide a fault (a far key among hundreds, a key just outside a window, a cap that is left
out, a map taken for the other), the inputs are made so that it shows."""
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_kilisun as pk
from test_ginodra_ops_gpu import DTYPES, F64, Rig, dev, i32, make_part, run_in_steps, step_batch

pytestmark = pytest.mark.gpu
EPS = 1e-5


@pytest.fixture(scope="module")
def ops():
    from nanohybrid_vlm_b200.kernels import ops
    return ops


def close(got, want, dtype, f32=2e-5, bf16=2e-2):
    """Worst difference relative to the size of the reference (float64)."""
    err = (got.to(F64) - want).abs().max().item()
    assert math.isfinite(err) and err <= (f32 if dtype == torch.float32 else bf16) * max(want.abs().max().item(), 1e-6), err


# ---------------------------------------------------------------- norms around the stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,width", [(5, 64), (3, 100), (300, 96), (2, 4096), (260, 2048), (1, 8), (4, 33), (2, 16384), (3, 6152)])
def test_a_pending_output_is_normed_added_and_the_sum_normed(dtype, T, width):
    from nanohybrid_vlm_b200.parts import NORMS, part
    from nanohybrid_vlm_b200.parts.base import Pending
    pre, post = (make_part(NORMS, part("rmsnorm", width=width, eps=e, weight_offset=1.0, source=n, own_name=True), width, dtype, s)
                 for n, e, s in (("norm2", EPS, 1), ("norm1b", 1e-3, 2)))
    g = torch.Generator().manual_seed(width)
    stream = torch.randn(T, width, generator=g) * 4
    y = (torch.randn(T, width, generator=g) * 0.1).to(dtype)
    new = stream.to(F64) + pk.norm_about_one(y.to(F64), post[1]["norm1b"], 1e-3)
    want = pk.norm_about_one(new, pre[1]["norm2"], EPS)
    s = dev(stream.clone())
    got = pre[0].forward_add(Pending(((dev(y), 1.0),), post=post[0]), s).cpu()
    close(got, want, dtype, bf16=5e-3)
    close(s.cpu(), new, torch.float32, f32=2e-6)            # the stream is never rounded to 16 bits
    rows = [T - 1, 0]
    s = dev(stream.clone())
    got = pre[0].forward_add_rows(Pending(((dev(y), 1.0),), post=post[0]), s, i32(rows)).cpu()
    close(got, want[rows], dtype, bf16=5e-3)
    assert torch.equal(s.cpu(), stream)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 100, 1032, 4096])
def test_the_stream_starts_as_the_normed_embedding(dtype, width):
    from nanohybrid_vlm_b200.parts import EMBEDDINGS, part
    norm = part("rmsnorm", width=width, eps=EPS, weight_offset=1.0, source="embed.norm", own_name=True)
    e, w = make_part(EMBEDDINGS, part("token_embedding", vocab_size=40, stream="float32", source="embed", norm=norm), width, dtype, 4)
    ids = [3, 39, 0, 3, 17]
    got = e.forward(i32(ids)).cpu()
    assert got.dtype == torch.float32
    close(got, pk.norm_about_one(w["embed"], w["embed.norm"], EPS)[ids], torch.float32, f32=2e-6)


# ---------------------------------------------------------------- heads from the projection to the cache
def lay_out(T, page, n_slots, seed):
    g = torch.Generator().manual_seed(seed)
    slots = torch.randperm(n_slots, generator=g)[:T].int()
    return slots


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,dims,pad", [(4, 2, 16, 24, 16, 0), (3, 1, 64, 128, 32, 0), (2, 2, 24, 60, 16, 16), (6, 3, 10, 22, 6, 4),
                                               (2, 1, 128, 256, 128, 0), (5, 5, 8, 8, 0, 8), (1, 1, 40, 80, 24, 0)])
def test_maps_are_normed_turned_and_laid_side_by_side(ops, dtype, H, G, d, dv, dims, pad):
    g = torch.Generator().manual_seed(d * H)
    T, page, row = 11, 4, max(2 * d, dv) + pad
    qkv = torch.randn(T, 2 * d * (H + G) + G * dv, generator=g).to(dtype)
    qw, kw = ((1 + 0.3 * torch.randn(d, generator=g)).to(dtype) for _ in range(2))
    pos = torch.randint(0, 90, (T,), generator=g).int()
    slots = lay_out(T, page, 24, 7)
    slots[3] = -1
    table = None
    if dims:
        ang = torch.arange(90, dtype=F64)[:, None] * torch.tensor([50.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
        table = dev(torch.cat([ang.cos(), ang.sin()], -1).float())
    b = step_batch([T], [0], [0])
    b.positions, b.n_prefill_seqs = dev(pos), 1
    pages = torch.full((6, 2, G, page, row), float("nan"), dtype=dtype, device="cuda")
    q = torch.full((T, H * 2 * row), float("nan"), dtype=dtype, device="cuda")
    ops.heads_store(dev(qkv), q, row, pages, dev(slots), b, table, dims, H, G, d, dv, EPS, dev(qw), dev(kw), maps=2)
    x = qkv.to(F64)
    wq = pk.unit_rms(x[:, :2 * d * H].reshape(T, 2 * H, d), EPS) * qw.to(F64)
    wk = pk.unit_rms(x[:, 2 * d * H:2 * d * (H + G)].reshape(T, 2 * G, d), EPS) * kw.to(F64)
    if dims:
        wq, wk = pk.turn_halves(wq, pos, 50.0, dims), pk.turn_halves(wk, pos, 50.0, dims)
    got_q = q.cpu().reshape(T, H, 2, row)
    for m in range(2):
        mine = got_q[:, :, m, m * d:(m + 1) * d]
        close(mine, wq.reshape(T, H, 2, d)[:, :, m], dtype, bf16=5e-3)
        rest = torch.cat([got_q[:, :, m, :m * d], got_q[:, :, m, (m + 1) * d:]], -1)
        assert (rest == 0).all()
    got = pages.cpu().permute(0, 3, 1, 2, 4).reshape(24, 2, G, row)
    wv = x[:, 2 * d * (H + G):].reshape(T, G, dv)
    for t, s in enumerate(slots.tolist()):
        if s < 0:
            continue
        close(got[s, 0, :, :2 * d], wk[t].reshape(G, 2 * d), dtype, bf16=5e-3)
        close(got[s, 1, :, :dv], wv[t], dtype, bf16=5e-3)
        assert (got[s, 0, :, 2 * d:] == 0).all() and (got[s, 1, :, dv:] == 0).all()
    unused = [s for s in range(24) if s not in slots.tolist()]
    assert torch.isnan(got[unused].float()).all()
    # queries only (a layer that reads another's pages)
    q2 = torch.full_like(q, float("nan"))
    ops.heads_store(dev(qkv)[:, :2 * d * H], q2, row, None, dev(slots), b, table, dims, H, G, d, dv, EPS, dev(qw), None, maps=2)
    assert torch.equal(q, q2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,K", [(4, 2, 16, 3), (3, 3, 48, 4), (2, 1, 10, 2), (1, 1, 128, 1), (5, 1, 24, 7), (2, 2, 256, 5), (6, 2, 8, 9)])
def test_filtered_heads_in_portions_and_reused_slots(ops, dtype, H, G, d, K):
    """Portions shorter than the filter make a tap reach through several earlier steps; the first tokens of a request must
    see zeros, not the request that held the slot before; single tokens and portions move the state on differently."""
    g = torch.Generator().manual_seed(d + K)
    C = (H + G) * d
    taps = torch.randn(C, K, generator=g).to(dtype)
    qw, kw = ((1 + 0.3 * torch.randn(d, generator=g)).to(dtype) for _ in range(2))
    lengths, cuts = [23, 9, 31, 5, 12], [[1, 2, 4, 11, 12, 13, 22], [3], [16, 17, 19, 20], [], [2, 3]]
    us = [(torch.randn(L, C, generator=g) + 1).to(dtype) for L in lengths]          # an offset: a leaked input shows
    state = torch.full((2, max(1, (K - 1) * C)), float("nan"), device="cuda")
    coef, every, page = 0.7, 5, 4
    pages = torch.full((10, 2, G, page, d), float("nan"), dtype=dtype, device="cuda")
    free, slot_of = [0, 1], {}
    bounds = [[0, *c, L] for L, c in zip(lengths, cuts)]
    waiting, progress = list(range(5)), dict.fromkeys(range(5), 0)
    got = {r: [] for r in range(5)}
    while waiting or slot_of:
        while waiting and free:
            slot_of[waiting.pop(0)] = free.pop(0)
        who = sorted(slot_of)
        starts = [bounds[r][progress[r]] for r in who]
        news = [bounds[r][progress[r] + 1] - s for r, s in zip(who, starts)]
        T = sum(news)
        # the projection's rows are wider than the heads (a gate's columns follow)
        qkv = torch.cat([torch.cat([us[r][s:s + n] for r, s, n in zip(who, starts, news)]), torch.full((T, 8), 5.0).to(dtype)], 1)
        b = step_batch(news, starts, [slot_of[r] for r in who])
        b.positions = i32([p for s, n in zip(starts, news) for p in range(s, s + n)])
        b.n_prefill_seqs = sum(n > 1 for n in news)
        q = torch.full((T, H * d), float("nan"), dtype=dtype, device="cuda")
        ops.heads_store(dev(qkv), q, d, pages, i32(list(range(T))), b, None, 0, H, G, d, d, EPS, dev(qw), dev(kw),
                        values_from_keys=True, taps=dev(taps.t().contiguous()), state=state, temperature=(coef, every))
        kv = pages.cpu().permute(0, 3, 1, 2, 4).reshape(40, 2, G * d)[:T]
        at = 0
        for r, n in zip(who, news):
            got[r].append(torch.cat([q[at:at + n].cpu(), kv[at:at + n, 0], kv[at:at + n, 1]], 1))
            at += n
            progress[r] += 1
            if progress[r] == len(bounds[r]) - 1:
                free.append(slot_of.pop(r))
    for r, L in enumerate(lengths):
        y = pk.taps_over_time(us[r].to(F64), taps.to(F64))
        f = pk.query_temperature(torch.arange(L), coef, every)[:, None, None]
        q = (pk.unit_rms(y[:, :H * d].reshape(L, H, d), EPS) * qw.to(F64) * f).reshape(L, -1)
        k = (pk.unit_rms(y[:, H * d:].reshape(L, G, d), EPS) * kw.to(F64)).reshape(L, -1)
        close(torch.cat(got[r]), torch.cat([q, k, y[:, H * d:]], 1), dtype, bf16=6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,dv", [(7, 3, 16), (5, 4, 128), (2, 1, 200), (9, 2, 30), (3, 5, 512), (2, 2, 600), (300, 2, 256), (1, 8, 64)])
def test_the_second_map_is_taken_off_the_first(ops, dtype, T, H, dv):
    g = torch.Generator().manual_seed(dv)
    a = torch.randn(T, H, 2, dv, generator=g)
    a[0, :, 1] = a[0, :, 0] * 1.25                              # share 0.8: nothing is left of the first token but eps
    a = a.to(dtype)
    out = torch.full((T, H * dv), float("nan"), dtype=dtype, device="cuda")
    for share, diff in ((0.8, 0.3), (-0.4, 0.0), (1.7, 0.9)):
        ops.map_difference(out, dev(a.reshape(T, -1)), torch.tensor([share], device="cuda"), 1 - diff, EPS, H, dv)
        want = pk.maps_combined(a[:, :, 0].to(F64), a[:, :, 1].to(F64), float(torch.tensor(share)), diff, EPS).reshape(T, -1)
        if dtype == torch.float32:
            torch.testing.assert_close(out.cpu()[1:].to(F64), want[1:], rtol=2e-5, atol=2e-6)
            torch.testing.assert_close(out.cpu()[:1].to(F64), want[:1], rtol=0, atol=1e-3)
        else:
            torch.testing.assert_close(out.cpu().to(F64), want, rtol=8e-3, atol=1e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,group", [(3, 4, 16), (5, 3, 10), (2, 2, 128)])
def test_one_gate_per_head(ops, dtype, T, H, group):
    g = torch.Generator().manual_seed(group)
    wide = torch.randn(T, H * group + H, generator=g).to(dtype)
    x, gate = dev(wide)[:, :H * group], dev(wide)[:, H * group:]
    out = torch.empty(T, H * group, dtype=dtype, device="cuda")
    ops.sigmoid_mul_heads(out, x, gate, group)
    w = wide.to(F64)
    want = (w[:, :H * group].reshape(T, H, group) * torch.sigmoid(w[:, H * group:])[..., None]).reshape(T, -1)
    close(out.cpu(), want, dtype, bf16=5e-3)


# ---------------------------------------------------------------- capped scores in every attention kernel
@pytest.mark.parametrize("cap,size", [(25.0, 1.0), (2.0, 1.0), (0.3, 30.0), (50.0, 300.0), (5.0, 4.0)])
@pytest.mark.parametrize("page,nq,nkv,dk,dv,window", [
    (64, 8, 2, 128, 128, 100), (64, 4, 4, 64, 64, 0), (16, 6, 2, 96, 96, 33), (128, 4, 1, 256, 256, 65), (16, 4, 2, 32, 16, 20),
    (8, 3, 1, 48, 48, 64), (5, 2, 1, 20, 12, 7), (64, 16, 1, 128, 64, 1), (64, 34, 1, 64, 64, 70)])
def test_capped_scores(ops, page, nq, nkv, dk, dv, window, cap, size):
    """Prompt portions beside single tokens against the plain softmax, in float32 and in bfloat16 with every kernel that
    takes the shape; scores far below the cap, around it and far beyond it (both forms of the cap, and its limits)."""
    news, starts = [130, 1, 2, 1, 65, 1], [0, 200, 63, 64, 70, 0]
    ends = [a + b for a, b in zip(news, starts)]
    g = torch.Generator().manual_seed(dk + dv)
    K = [torch.randn(n, nkv, dk, generator=g).bfloat16() for n in ends]
    V = [torch.randn(n, nkv, dv, generator=g).bfloat16() for n in ends]
    Q = [torch.randn(n, nq, dk, generator=g).bfloat16() for n in news]
    scale = size / dk ** 0.5
    counts = [-(-n // page) for n in ends]
    order = torch.randperm(sum(counts) + 3, generator=g).tolist()
    pages = torch.full((sum(counts) + 3, 2, nkv, page, dk), float("nan"), dtype=torch.bfloat16)
    pages[:, 1, :, :, dv:] = 0
    table = torch.full((len(ends), max(counts)), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(ends):
        lo = max(0, starts[s] - window + 1) if window else 0
        for p in range(counts[s]):
            if (p + 1) * page <= lo:
                continue                                        # behind the window: given back
            table[s, p] = order[at]
            m = min(page, n - p * page)
            pages[order[at], 0, :, :m] = K[s][p * page:p * page + m].transpose(0, 1)
            pages[order[at], 1, :, :m, :dv] = V[s][p * page:p * page + m].transpose(0, 1)
            at += 1
    cu = [0, *np.cumsum(news).tolist()]
    b = SimpleNamespace(cu_q=i32(cu), kv_len=i32(ends), n_seqs=len(news), n_tokens=cu[-1], max_kv_len=max(ends),
                        n_prefill_tokens=sum(n for n in news if n > 1), n_prefill_seqs=3, n_decode_seqs=3)
    want = []
    for s, n in enumerate(ends):
        seen = pk.in_window(n, window or None)[starts[s]:]
        heads = []
        for h in range(nq):
            kk, vv = K[s][:, h // (nq // nkv)].to(F64), V[s][:, h // (nq // nkv)].to(F64)
            heads.append(pk.softmax_rows(pk.soft_capped(Q[s][:, h].to(F64) @ kk.T * scale, cap), seen) @ vv)
        want.append(torch.cat(heads, -1))
    want = torch.cat(want)
    q = torch.cat(Q).reshape(cu[-1], nq * dk)
    dtable = SimpleNamespace(block_tables=dev(table))
    out = torch.full((cu[-1], nq * dv), float("nan"), device="cuda")
    ops.attention_sink(out, dev(q.float()), dev(pages.float()), dtable, b, nq, nkv, dk, dv, scale, None, window, softcap=cap)
    close(out.cpu(), want, torch.float32, f32=1e-5)
    before = ops.USE_TCGEN05_ATTENTION, ops.USE_TMA_DECODE
    try:
        for wide in (True, False):
            ops.USE_TCGEN05_ATTENTION = ops.USE_TMA_DECODE = wide
            out = torch.full((cu[-1], nq * dv), float("nan"), dtype=torch.bfloat16, device="cuda")
            ops.attention_sink(out, dev(q), dev(pages), dtable, b, nq, nkv, dk, dv, scale, None, window, softcap=cap)
            close(out.cpu(), want, torch.bfloat16)
    finally:
        ops.USE_TCGEN05_ATTENTION, ops.USE_TMA_DECODE = before
    ops.raise_wait_errors()


def test_a_cap_goes_before_a_distance_term(ops):
    """Both on one layer: the cap on the product, the distance taken off the capped score."""
    T, nq, d, cap, scale = 70, 2, 64, 1.5, 0.5
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(T, n, d, generator=g).bfloat16() for n in (nq, 1, 1))
    pages = torch.zeros(2, 2, 1, 64, d, dtype=torch.bfloat16)
    for p in range(2):
        m = min(64, T - p * 64)
        pages[p, 0, 0, :m], pages[p, 1, 0, :m] = k[p * 64:p * 64 + m, 0], v[p * 64:p * 64 + m, 0]
    slopes = torch.tensor([0.05, 0.4])
    b = SimpleNamespace(cu_q=i32([0, T]), kv_len=i32([T]), n_seqs=1, n_tokens=T, max_kv_len=T, n_prefill_tokens=T,
                        n_prefill_seqs=1, n_decode_seqs=0)
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(F64)
    want = torch.cat([pk.softmax_rows(pk.soft_capped(q[:, h].to(F64) @ k[:, 0].to(F64).T * scale, cap) - slopes[h].to(F64) * dist,
                                      pk.in_window(T, None)) @ v[:, 0].to(F64) for h in range(nq)], -1)
    for dtype in DTYPES:
        out = torch.empty(T, nq * d, dtype=dtype, device="cuda")
        ops.attention_sink(out, dev(q.reshape(T, -1).to(dtype)), dev(pages.to(dtype)), SimpleNamespace(block_tables=i32([[0, 1]])), b,
                           nq, 1, d, d, scale, slopes=dev(slopes), softcap=cap)
        close(out.cpu(), want, dtype)


# ---------------------------------------------------------------- differential attention
LENGTHS, CUTS = [150, 37, 90, 5], [[40, 41, 104], [2, 30], [64, 66, 67, 68], [1, 2, 3, 4]]
MAP_CASES = [
    (dict(heads=6, kv_heads=3, dim=40, vdim=96, scale=0.2, diff=0.55, softcap=18.0, rot=dict(base=1000.0, dims=32), mask=dict(size=30)), 8),
    (dict(heads=6, kv_heads=2, dim=16, vdim=48, scale=0.4, diff=0.2, softcap=3.0, rot=dict(base=50.0, dims=8), mask=dict(size=64)), 16),
    (dict(heads=2, kv_heads=1, dim=64, vdim=128, scale=0.15, diff=0.8, softcap=50.0, rot=dict(base=9000.0, dims=32), mask=dict(size=65)), 64),
    (dict(heads=3, kv_heads=3, dim=10, vdim=14, scale=0.4, diff=0.0, softcap=1.0, rot=dict(base=7.0, dims=6), mask=dict(size=2)), 5),
    (dict(heads=5, kv_heads=1, dim=32, vdim=64, scale=0.3, diff=0.5, softcap=None, rot=dict(base=300.0, dims=32), mask=None), 64),
    (dict(heads=2, kv_heads=2, dim=128, vdim=256, scale=0.1, diff=0.4, softcap=8.0, rot=dict(base=100.0, dims=128), mask=dict(size=40)), 64),
    (dict(heads=1, kv_heads=1, dim=24, vdim=20, scale=0.3, diff=1.0 - 2 ** -3, softcap=15.0, rot=dict(base=100.0, dims=16), mask=dict(size=1)), 16),
    (dict(heads=2, kv_heads=1, dim=144, vdim=80, scale=0.1, diff=0.3, softcap=15.0, rot=dict(base=100.0, dims=0), mask=dict(size=33)), 16),
]


def map_part(m, W, dtype, seed, keep=None, own=True):
    from nanohybrid_vlm_b200.parts import MIXERS, part
    rope = part("rope_banded", theta=m["rot"]["base"], rotary_dim=m["rot"]["dims"]) if m["rot"]["dims"] else None
    size = pk.window_size(m)
    return make_part(MIXERS, part("differential_attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                  v_head_dim=m["vdim"], scale=m["scale"], position=rope, eps=EPS, diff=m["diff"],
                                  softcap=m["softcap"], window=size, keep_window=keep or size, own_kv=own), W, dtype, seed,
                     scale={n: 0.5 / m["dim"] ** 0.25 for n in ("lq1", "lk1", "lq2", "lk2")})


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,page", MAP_CASES)
def test_differential_attention_and_a_layer_that_reads_its_keys(dtype, m, page):
    """Two layers on different inputs: one with keys of its own, one with other weights, more heads and a wider window that
    reads them.  The pool has room for little more than the windows."""
    W = 64
    wide = dict(m, heads=2 * m["heads"], diff=0.1, softcap=4.0, mask=None if m["mask"] is None else dict(size=m["mask"]["size"] + 9))
    (own, w0), (reader, w1) = map_part(m, W, dtype, 5, pk.window_size(wide)), map_part(wide, W, dtype, 6, own=False)
    assert own.cache_need() == reader.cache_need()
    x = [[torch.randn(n, W, generator=torch.Generator().manual_seed(10 * n + i)).to(dtype) for n in LENGTHS] for i in range(2)]
    from nanohybrid_vlm_b200.parts.base import SharedPagesNeed
    rig = Rig([own.cache_need(), SharedPagesNeed()], cache_from={1: 0}, page_size=page, num_pages=-(-300 // page) + 4, dtype=dtype)

    def step(b, rows):
        return torch.cat([p.forward(dev(torch.cat([x[i][r][s:s + n] for r, s, n in rows])), b, rig.view(i, b))
                          for i, p in enumerate((own, reader))], -1)

    got = run_in_steps(rig, LENGTHS, CUTS, step)
    for r in range(len(LENGTHS)):
        h = [x[i][r].to(F64) for i in range(2)]
        kv = pk.map_keys_values(h[0], m, w0, "", EPS)
        close(got[r][:, :W], pk.differential_attention(h[0], m, w0, "", EPS, kv), dtype, f32=1e-4, bf16=5e-2)
        close(got[r][:, W:], pk.differential_attention(h[1], wide, w1, "", EPS, kv), dtype, f32=1e-4, bf16=5e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [150, 1, 7])
@pytest.mark.parametrize("window,page", [(1, 16), (16, 16), (33, 8), (64, 64), (65, 64)])
def test_keys_just_inside_and_just_outside_a_window_of_both_maps(ops, dtype, window, page, portion):
    """Zeros but for one key per map that stands out for every query: the first map's at one place, the second's at
    another.  The outputs step exactly where the window leaves them, and each map sees its own key only."""
    T, d, dv, first, second = 150, 16, 32, 20, 37
    from nanohybrid_vlm_b200.parts.base import PagedKVNeed
    k = torch.zeros(T, 1, 2, d)
    k[first, 0, 0, 0] = k[second, 0, 1, 0] = 8.0
    v = torch.zeros(T, 1, dv)
    v[first, 0, 0], v[second, 0, 1] = 1.0, 1.0
    q = torch.zeros(T, 2, 2 * d)
    q[:, 0, 0] = q[:, 1, d] = 2.0                               # padded queries of the two maps
    rig = Rig([PagedKVNeed(1, 2 * d, window, v_head_dim=dv)], page_size=page, num_pages=-(-T // page) + 2, dtype=dtype)
    got, done = [], 0
    while done < T:
        n = min(portion, T - done)
        b = rig.batch([("r", done, n)])
        view = rig.view(0, b)
        slots = view.tables.slot_mapping.long()[:n]
        pg, off = slots // page, slots % page
        view.pages[pg, 0, 0, off] = dev(k[done:done + n].reshape(n, 2 * d).to(dtype))
        view.pages[pg, 1, 0, off] = dev(v[done:done + n, 0].to(dtype))
        out = torch.empty(n, 2 * dv, dtype=dtype, device="cuda")
        ops.attention_sink(out, dev(q[done:done + n].reshape(n, -1).to(dtype)), view.pages, view.tables, b, 2, 1, 2 * d, dv, 1.0,
                           window=window, softcap=10.0)
        got.append(out.float().cpu())
        done += n
        rig.after_step()
    a = torch.cat(got).reshape(T, 2, dv)
    seen = pk.in_window(T, window)
    for m, (at, col) in enumerate(((first, 0), (second, 1))):
        s = pk.soft_capped((q[:, m].to(F64) @ k.reshape(T, 2 * d).to(F64).T), 10.0)
        close(a[:, m], pk.softmax_rows(s, seen) @ v[:, 0].to(F64), dtype)
        assert a[at + window - 1, m, col] > 0.9
        if window > 1:
            assert a[at + window, m, col] == 0 and a[at - 1, m, col] == 0


# ---------------------------------------------------------------- attention over filtered keys
FULL_CASES = [
    (dict(heads=9, kv_heads=3, dim=48, vdim=48, scale=0.25, conv=3, q_temp=dict(coef=0.25, every=16)), 8),
    (dict(heads=4, kv_heads=4, dim=64, vdim=64, scale=0.2, conv=4, q_temp=dict(coef=1.0, every=50)), 64),
    (dict(heads=3, kv_heads=1, dim=10, vdim=10, scale=0.5, conv=2, q_temp=dict(coef=0.5, every=1)), 5),
    (dict(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.1, conv=8, q_temp=None), 64),
    (dict(heads=8, kv_heads=2, dim=32, vdim=32, scale=0.3, conv=1, q_temp=dict(coef=-0.2, every=7)), 16),
    (dict(heads=2, kv_heads=2, dim=24, vdim=24, scale=0.3, conv=0, q_temp=dict(coef=0.4, every=3)), 16),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,page", FULL_CASES)
def test_attention_over_filtered_keys_that_are_the_values(dtype, m, page):
    from nanohybrid_vlm_b200.parts import MIXERS, part
    W = 64
    qt = m["q_temp"]
    p, w = make_part(MIXERS, part("sink_attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                  scale=m["scale"], position=None, unit_norm_eps=EPS, qk_norm_weight=True,
                                  qk_norm_order="before_rotation", sink=False, values="keys", output_gate="sigmoid_head",
                                  conv_taps=m["conv"], query_temperature=None if qt is None else (qt["coef"], qt["every"])),
                     W, dtype, 8)
    x = [torch.randn(n, W, generator=torch.Generator().manual_seed(n)).to(dtype) for n in LENGTHS]
    rig = Rig([p.cache_need()], page_size=page, num_pages=-(-300 // page) + 4, slots=4, dtype=dtype)
    got = run_in_steps(rig, LENGTHS, CUTS, lambda b, rows: p.forward(dev(torch.cat([x[r][s:s + n] for r, s, n in rows])), b, rig.view(0, b)))
    for r in range(len(LENGTHS)):
        close(got[r], pk.attention(x[r].to(F64), m, w, "", EPS), dtype, f32=1e-4, bf16=4e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_among_hundreds(dtype):
    """One early token's input is aligned with every query's: its key stands out at any distance, in a prompt and decoded
    one by one, and a temperature that is left out would show in how much."""
    from nanohybrid_vlm_b200.parts import MIXERS, part
    W, T, far = 32, 400, 3
    m = dict(heads=2, kv_heads=1, dim=32, vdim=32, scale=1.0, conv=2, q_temp=dict(coef=0.15, every=64))
    p, w = make_part(MIXERS, part("sink_attention", num_heads=2, num_kv_heads=1, head_dim=32, scale=0.22, position=None,
                                  unit_norm_eps=EPS, qk_norm_weight=True, qk_norm_order="before_rotation", sink=False,
                                  values="keys", output_gate="sigmoid_head", conv_taps=2, query_temperature=(0.15, 64)), W, dtype, 9)
    m["scale"] = 0.22
    g = torch.Generator().manual_seed(2)
    x = torch.randn(T, W, generator=g) * 0.3
    # the key of the far token along the last query's direction: solve through the two projections
    Wq, Wk = w["q"][:32] * w["q.conv"][:32, 1:], w["k"] * w["k.conv"][:, 1:]
    x[far] = (torch.linalg.lstsq(Wk, Wq @ x[T - 1].to(F64)).solution * 4).float()
    x = x.to(dtype)
    want = pk.attention(x.to(F64), m, w, "", EPS)
    without = pk.attention(torch.cat([x[:far], x[:1] * 0, x[far + 1:]]).to(F64), m, w, "", EPS)
    assert (want[T - 1] - without[T - 1]).norm() > 0.2 * want[T - 1].norm()            # the far key matters
    for cuts in ([], [T - 30 + i for i in range(30)]):
        rig = Rig([p.cache_need()], page_size=16, num_pages=26, slots=1, dtype=dtype)
        got = run_in_steps(rig, [T], [cuts], lambda b, rows: p.forward(dev(torch.cat([x[s:s + n] for _, s, n in rows])), b, rig.view(0, b)))
        close(got[0], want, dtype, f32=1e-4, bf16=4e-2)


# ---------------------------------------------------------------- router and experts
@pytest.mark.parametrize("T,E,top,count,keep", [(40, 14, 2, 2, 1), (33, 8, 3, 4, 2), (9, 6, 2, 6, 3), (64, 128, 8, 8, 4), (5, 4, 4, 1, 1), (7, 9, 1, 3, 3)])
@pytest.mark.parametrize("shift", [0.0, -3.0])
def test_groups_scored_by_their_two_best(ops, T, E, top, count, keep, shift):
    """``shift`` makes every choice score negative: closed groups must count as minus infinity, not as zero."""
    g = torch.Generator().manual_seed(E + top)
    z, c = torch.randn(T, E, generator=g) * 2, torch.randn(E, generator=g) * 0.4 + shift
    ids, w = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    ops.moe_route(ids, w, dev(z), dev(c), E, count, keep, scores="sigmoid", renorm=False, group_best=2, factor=2.5)
    r = dict(experts=E, top=top, groups=dict(count=count, keep=keep), scale=2.5)
    want_ids, want_w = pk.route(z.to(F64), torch.eye(E, dtype=F64), c.to(F64), r)
    order, worder = torch.sort(ids.cpu().long(), -1), torch.sort(want_ids, -1)
    assert torch.equal(order.values, worder.values)
    torch.testing.assert_close(torch.gather(w.cpu().to(F64), 1, order.indices), torch.gather(want_w, 1, worder.indices), rtol=1e-5, atol=1e-6)


def test_the_best_expert_may_stand_in_a_closed_group(ops):
    z = torch.logit(torch.tensor([[0.95, 0.05, 0.6, 0.55]]))
    ids, w = torch.empty(1, 1, dtype=torch.int32, device="cuda"), torch.empty(1, 1, device="cuda")
    ops.moe_route(ids, w, dev(z), torch.zeros(4, device="cuda"), 4, 2, 1, scores="sigmoid", renorm=False, group_best=2, factor=0.5)
    assert ids.item() == 2 and abs(w.item() - 0.3) < 1e-6
    ops.moe_route(ids, w, dev(z), torch.zeros(4, device="cuda"), 4, 2, 1, scores="sigmoid", renorm=False, group_best=1, factor=0.5)
    assert ids.item() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,top,count,keep,ff,shared", [(1, 64, 6, 2, 3, 2, 32, 48), (50, 100, 4, 3, 2, 2, 18, 26), (300, 128, 8, 1, 4, 1, 72, None),
                                                            (700, 64, 8, 4, 2, 1, 136, 24)])
def test_mixture_with_limits_of_its_own_for_the_shared_expert(dtype, T, W, E, top, count, keep, ff, shared):
    from nanohybrid_vlm_b200.parts import FEED_FORWARDS, part
    mlp = dict(router=dict(experts=E, top=top, groups=dict(count=count, keep=keep), scale=1.7), expert=dict(ff=ff, limit=0.4),
               shared=None if shared is None else dict(ff=shared, limit=1.1))
    sh = None if shared is None else part("clamped_glu", intermediate_size=shared, limit=1.1, alpha=1.702)
    p, w = make_part(FEED_FORWARDS, part("routed_moe", experts=E, top=top, groups=count, keep=keep, group_best=2, scores="sigmoid",
                                         renorm=False, weight_factor=1.7, correction=True, intermediate_size=ff, limit=0.4,
                                         alpha=1.702, shared=sh, shared_gate=sh is not None), W, dtype, 31, scale={"correction": 0.3})
    w = {k: v[0] if v.dim() == 3 else v for k, v in w.items()}
    h = torch.randn(T, W, generator=torch.Generator().manual_seed(T)).to(dtype)
    got = p.forward(dev(h), None).cpu()
    x = h.to(F64)
    want = pk.mixture(x, mlp, w, "")
    # tokens whose choice does not hang on rounding: moving every score a little changes nothing
    sure = torch.ones(T, dtype=torch.bool)
    ids = pk.route(x, w["router"], w["correction"], mlp["router"])[0].sort(-1).values
    for s in range(4):
        nudge = torch.randn(E, generator=torch.Generator().manual_seed(s), dtype=F64) * (0.004 if dtype == torch.bfloat16 else 1e-5)
        sure &= (pk.route(x, w["router"], w["correction"] + nudge, mlp["router"])[0].sort(-1).values == ids).all(-1)
    assert sure.float().mean() > 0.8
    close(got[sure], want[sure], dtype, f32=3e-5, bf16=3e-2)
