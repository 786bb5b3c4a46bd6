"""The mechanisms of the Vozorax design one at a time: each part or kernel against the plain function of the same
mechanism (float64 on the CPU), in packed batches of unequal requests, in portions down to one token, with pages in a
poisoned pool that are given back behind windows and used again.  Where random numbers would hide a fault (a key just
outside a window, a sink that is left out), the inputs are made so that it shows."""
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_vozorax as pv
from test_ginodra_ops_gpu import DTYPES, F64, Rig, dev, i32, make_part, run_in_steps, tol

pytestmark = pytest.mark.gpu
EPS = 1e-5


@pytest.fixture(scope="module")
def ops():
    from nanohybrid_vlm_b200.kernels import ops
    return ops


def rounded(t, dtype):
    return t.to(dtype).to(F64)


def close(got, want, dtype, f32=2e-5, bf16=2e-2):
    """Worst difference relative to the size of the reference (float64)."""
    err = (got.to(F64) - want).abs().max().item()
    assert math.isfinite(err) and err <= (f32 if dtype == torch.float32 else bf16) * max(want.abs().max().item(), 1e-6), err


# ---------------------------------------------------------------- several copies of the residual stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,width,T", [(1, 64, 5), (2, 96, 3), (3, 1032, 9), (4, 4096, 2), (5, 100, 7), (7, 33, 4), (8, 2048, 3),
                                       (9, 64, 5), (16, 260, 3), (4, 50, 6), (6, 6148, 2)])
def test_streams_are_mixed_written_read_and_normed(ops, dtype, S, width, T):
    g = torch.Generator().manual_seed(S * 1000 + width)
    x = torch.randn(T, S, width, generator=g, dtype=torch.float32) * 3
    y = torch.randn(T, width, generator=g).to(dtype)
    mix, write, read = (torch.randn(*s, generator=g) for s in ((S, S), (S,), (S,)))
    w = (1 + 0.3 * torch.randn(width, generator=g)).to(dtype)
    X = x.to(F64).transpose(0, 1)
    new = pv.write_streams(X, mix.to(F64), write.to(F64), y.to(F64))
    want = pv.unit_rms(pv.read_streams(new, read.to(F64)), EPS) * w.to(F64)
    for in_place in (True, False):
        src = dev(x.clone())
        dst = src if in_place else torch.full_like(src, float("nan"))
        out = torch.empty(T, width, dtype=dtype, device="cuda")
        ops.streams_rmsnorm(out, dst, src, dev(w), EPS, dev(y), dev(mix), dev(write), dev(read))
        close(out.cpu(), want, dtype, bf16=5e-3)
        close(dst.cpu(), new.transpose(0, 1), torch.float32, f32=2e-6)
    # the last norm of a model: the plain sum, at some rows only, nothing written
    rows = [T - 1, 0]
    src = dev(x.clone())
    out = torch.empty(2, width, dtype=dtype, device="cuda")
    ops.streams_rmsnorm(out, None, src, dev(w), EPS, dev(y), dev(mix), dev(write), None, i32(rows))
    close(out.cpu(), (pv.unit_rms(new.sum(0), EPS) * w.to(F64))[rows], dtype, bf16=5e-3)
    assert torch.equal(src.cpu(), x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,width", [(3, 72), (4, 31), (1, 64), (12, 40)])
def test_streams_that_are_still_equal_are_one_row(ops, dtype, S, width):
    g = torch.Generator().manual_seed(5)
    T = 6
    e = torch.randn(T, 1, width, generator=g)
    y = torch.randn(T, width, generator=g).to(dtype)
    mix, write, read = (torch.randn(*s, generator=g) for s in ((S, S), (S,), (S,)))
    w = (1 + 0.3 * torch.randn(width, generator=g)).to(dtype)
    X = e.to(F64)[:, 0][None].repeat(S, 1, 1)
    out = torch.empty(T, width, dtype=dtype, device="cuda")
    ops.streams_rmsnorm(out, None, dev(e), dev(w), EPS, read=dev(read), n_streams=S)
    close(out.cpu(), pv.unit_rms(pv.read_streams(X, read.to(F64)), EPS) * w.to(F64), dtype, bf16=5e-3)
    dst = torch.full((T, S, width), float("nan"), device="cuda")
    ops.streams_rmsnorm(out, dst, dev(e), dev(w), EPS, dev(y), dev(mix), dev(write), dev(read), n_streams=S)
    new = pv.write_streams(X, mix.to(F64), write.to(F64), y.to(F64))
    close(dst.cpu(), new.transpose(0, 1), torch.float32, f32=2e-6)
    close(out.cpu(), pv.unit_rms(pv.read_streams(new, read.to(F64)), EPS) * w.to(F64), dtype, bf16=5e-3)


def test_the_mixing_matrix_is_indexed_from_to(ops):
    """A permutation: copy 0 goes to place 2, 1 to 0, 2 to 1."""
    x = torch.arange(3.0)[None, :, None].repeat(1, 1, 8)
    mix = torch.zeros(3, 3)
    mix[0, 2] = mix[1, 0] = mix[2, 1] = 1.0
    src, out = dev(x), torch.empty(1, 8, device="cuda")
    ops.streams_rmsnorm(out, src, src, torch.ones(8, device="cuda"), EPS, torch.zeros(1, 8, device="cuda"), dev(mix),
                        torch.zeros(3, device="cuda"), torch.ones(3, device="cuda"))
    assert src[0, :, 0].tolist() == [1.0, 2.0, 0.0]


@pytest.mark.parametrize("dtype", DTYPES)
def test_block_over_streams(dtype):
    """Two layers (the second without a feed-forward) of parts that compute simple things, the embedding as one row to
    start from, the last norm at some rows."""
    from nanohybrid_vlm_b200.parts import CONNECTIONS, NORMS, part
    from nanohybrid_vlm_b200.parts.base import BLOCKS
    S, W, T = 3, 40, 7
    g = torch.Generator().manual_seed(8)

    class Product:                                          # stands for a mixer: a product with a fixed matrix
        def __init__(self, m):
            self.m = m

        def forward(self, x, batch, cache=None):
            return (x.float() @ self.m.cuda().float()).to(dtype)

    def connection(name, seed):
        return make_part(CONNECTIONS, part("hyper_connection", streams=S, source=name), W, torch.float32, seed)

    def norm(seed):
        return make_part(NORMS, part("rmsnorm", width=W, eps=EPS, source="norm1", own_name=True), W, dtype, seed)

    mats = [(torch.randn(W, W, generator=g) / W ** 0.5) for _ in range(3)]
    (n1, nw1), (n2, nw2), (n3, nw3), (nf, nwf) = (norm(s) for s in (1, 2, 3, 4))
    (c1, cw1), (c2, cw2), (c3, cw3) = (connection(n, s) for n, s in (("hc1", 5), ("hc2", 6), ("hc1", 7)))
    cls = BLOCKS.get("hyper_connections")
    b1 = cls(part("hyper_connections"), dict(mixer=Product(mats[0]), mixer_norm=n1, mixer_connection=c1, ffn=Product(mats[1]),
                                             ffn_norm=n2, ffn_connection=c2))
    b2 = cls(part("hyper_connections"), dict(mixer=Product(mats[2]), mixer_norm=n3, mixer_connection=c3))
    e = torch.randn(T, W, generator=g)
    h, res = b1.forward(dev(e), None, None, None)
    h, res = b2.forward(h, res, None, None)
    rows = [0, T - 1, 2]
    got = nf.forward_add_rows(h, res, i32(rows)).cpu()
    X = e.to(F64)[None].repeat(S, 1, 1)
    for m, nw, cw, name in ((mats[0], nw1, cw1, "hc1"), (mats[1], nw2, cw2, "hc2"), (mats[2], nw3, cw3, "hc1")):
        y = (pv.unit_rms(pv.read_streams(X, cw[name + ".in"]), EPS) * nw["norm1"]) @ m.to(F64)
        X = pv.write_streams(X, cw[name + ".mix"], cw[name + ".out"], y)
    close(got, (pv.unit_rms(X.sum(0), EPS) * nwf["norm1"])[rows], dtype)
    with pytest.raises(ValueError, match="connection"):
        cls(part("hyper_connections"), dict(mixer=Product(mats[0]), mixer_norm=n1, mixer_connection=c1, ffn=Product(mats[1])))


# ---------------------------------------------------------------- latent attention in a window
LENGTHS, CUTS = [150, 37, 90, 5], [[40, 41, 104], [2, 30], [64, 66, 67, 68], [1, 2, 3, 4]]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,page", [
    (dict(heads=4, dim=16, rot_dim=8, vdim=16, q_rank=24, kv_rank=40, scale=0.2, rot=dict(base=1000.0, dims=8), mask=dict(size=20)), 8),
    (dict(heads=3, dim=48, rot_dim=16, vdim=32, q_rank=40, kv_rank=64, scale=0.15, rot=dict(base=50.0, dims=16), mask=dict(size=65)), 16),
    (dict(heads=2, dim=24, rot_dim=10, vdim=40, q_rank=17, kv_rank=30, scale=0.25, rot=dict(base=300.0, dims=10), mask=dict(size=1)), 5),
    (dict(heads=17, dim=8, rot_dim=4, vdim=12, q_rank=16, kv_rank=24, scale=0.3, rot=dict(base=7.0, dims=4), mask=dict(size=64)), 64),
    (dict(heads=2, dim=96, rot_dim=32, vdim=128, q_rank=32, kv_rank=128, scale=0.1, rot=dict(base=10000.0, dims=32), mask=None), 16),
])
@pytest.mark.parametrize("expand", [True, False])
def test_latent_attention_in_a_window(ops, dtype, m, page, expand, monkeypatch):
    """In portions and token by token, each request against itself whole; both forms of the bfloat16 prompt step."""
    from nanohybrid_vlm_b200.parts import MIXERS, latent_attention, part
    monkeypatch.setattr(latent_attention, "EXPAND_PROMPT_PORTIONS", expand)
    W = 64
    size = None if m["mask"] is None else m["mask"]["size"]
    mixer, w = make_part(MIXERS, part(
        "latent_attention", num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], v_head_dim=m["vdim"],
        q_rank=m["q_rank"], kv_rank=m["kv_rank"], scale=m["scale"], eps=EPS, sink=False, window=size,
        rope_layout="interleaved", position=part("rope_banded", theta=m["rot"]["base"], rotary_dim=m["rot"]["dims"])),
        W, dtype, 11)
    x = [torch.randn(n, W, generator=torch.Generator().manual_seed(n)).to(dtype) for n in LENGTHS]
    rig = Rig([mixer.cache_need()], page_size=page, num_pages=-(-300 // page) + 4, dtype=dtype)

    def step(b, rows):
        return mixer.forward(dev(torch.cat([x[r][s:s + n] for r, s, n in rows])), b, rig.view(0, b))

    got = run_in_steps(rig, LENGTHS, CUTS, step)
    for r, h in enumerate(x):
        close(got[r], pv.latent_attention(h.to(F64), m, w, "", EPS), dtype, f32=1e-4, bf16=4e-2)


def standing_out(T, H, dk, first, second):
    """Queries of ones and keys of zeros but for two positions that outweigh all others; values that tell them apart."""
    q = torch.ones(T, H * dk)
    k = torch.zeros(T, dk)
    k[first], k[second] = 9.0 / dk, 12.0 / dk
    return q, k


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [7, 64, 65, 100])
@pytest.mark.parametrize("portion", [1, 2, 30])
def test_keys_just_inside_and_just_outside_a_latent_window(ops, dtype, window, portion):
    """Two keys outweigh all others; the later tokens see both, then one, then neither as the window passes them."""
    from nanohybrid_vlm_b200.parts import PagedKVNeed
    H, rank, dr, page = 3, 32, 8, 16
    row, T = rank + dr, 240
    at = 70
    q, k = standing_out(T, H, row, at, at + 1)
    rig = Rig([PagedKVNeed(1, row, window, v_head_dim=rank, planes=1)], page_size=page, num_pages=20, dtype=dtype)
    got, done = [], 0
    while done < T:
        n = min(portion if done >= 60 else 60, T - done)
        b = rig.batch([("r", done, n)])
        pages = rig.view(0, b).pages
        slots = rig.view(0, b).tables.slot_mapping.long()
        pages.view(-1, row)[slots] = dev(k[done:done + n].to(dtype))
        out = torch.empty(n, H * rank, dtype=dtype, device="cuda")
        ops.latent_attention(out, dev(q[done:done + n].to(dtype)), pages, rig.view(0, b).tables, b, H, rank, row, 1.0, None, window)
        got.append(out.float().cpu())
        done += n
        rig.after_step()
    got = torch.cat(got)
    kr = rounded(k, dtype)
    s = rounded(q, dtype).reshape(T, H, row)[:, 0] @ kr.T
    want = pv.softmax_rows(s, pv.in_window(T, window)) @ kr[:, :rank]
    close(got, want.repeat(1, H), dtype)
    # the steps of the window show: both keys, the later one alone, neither
    a, b_, c = (got[at + window + i - 1, 0].item() for i in (0, 1, 2))
    assert c < 0.2 * b_ and abs(a - b_) > 0.005 * b_


# ---------------------------------------------------------------- attention with rows normed whole and mixed values
ATTN_CASES = [
    (dict(heads=6, kv_heads=3, dim=64, vdim=24, scale=0.2, mask=dict(size=30)), 8),
    (dict(heads=6, kv_heads=2, dim=16, vdim=48, scale=0.3, mask=dict(size=64)), 16),
    (dict(heads=2, kv_heads=1, dim=128, vdim=64, scale=0.1, mask=dict(size=65)), 64),
    (dict(heads=3, kv_heads=3, dim=10, vdim=14, scale=0.4, mask=dict(size=2)), 5),
    (dict(heads=5, kv_heads=1, dim=80, vdim=80, scale=0.15, mask=None), 16),
    (dict(heads=2, kv_heads=2, dim=64, vdim=128, scale=0.2, mask=dict(size=40)), 64),
    (dict(heads=4, kv_heads=4, dim=24, vdim=24, scale=0.2, mask=dict(size=17)), 16),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,page", ATTN_CASES)
def test_attention_with_whole_norms_sinks_and_mixed_values(ops, dtype, m, page):
    """Three layers on different inputs: the source of the values, one that mixes them in, one that does neither."""
    from nanohybrid_vlm_b200.parts import MIXERS, part
    W = 64
    size = None if m["mask"] is None else m["mask"]["size"]
    made = [make_part(MIXERS, part("sink_attention", num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                                   v_head_dim=m["vdim"], scale=m["scale"], position=None, unit_norm_eps=EPS,
                                   qk_norm_weight=True, qk_norm_scope="projection", sink=True, window=size, value_mix=vm),
                      W, dtype, 20 + i, scale={"sink": 2.0}) for i, vm in enumerate(("source", "mixed", None))]
    x = [[torch.randn(n, W, generator=torch.Generator().manual_seed(10 * n + i)).to(dtype) for n in LENGTHS] for i in range(3)]
    rig = Rig([p.cache_need() for p, _ in made], page_size=page, num_pages=-(-300 // page) + 4, dtype=dtype)

    def step(b, rows):
        return torch.cat([p.forward(dev(torch.cat([x[i][r][s:s + n] for r, s, n in rows])), b, rig.view(i, b))
                          for i, (p, _) in enumerate(made)], -1)

    got = run_in_steps(rig, LENGTHS, CUTS, step)
    for r in range(len(LENGTHS)):
        h = [x[i][r].to(F64) for i in range(3)]
        y0, own = pv.attention(h[0], m, made[0][1], "", EPS)
        y1, _ = pv.attention(h[1], m, made[1][1], "", EPS, own)
        y2, _ = pv.attention(h[2], m, made[2][1], "", EPS)
        for i, want in enumerate((y0, y1, y2)):
            close(got[r][:, i * W:(i + 1) * W], want, dtype, f32=1e-4, bf16=4e-2)


def test_a_layer_that_mixes_needs_a_source_of_its_size():
    from nanohybrid_vlm_b200.parts import MIXERS, part
    p, _ = make_part(MIXERS, part("sink_attention", num_heads=2, num_kv_heads=1, head_dim=16, scale=0.2, unit_norm_eps=EPS,
                                  qk_norm_weight=True, qk_norm_scope="projection", value_mix="mixed"), 32, torch.float32, 1)
    rig = Rig([p.cache_need()])
    b = rig.batch([("r", 0, 3)])
    with pytest.raises(ValueError, match="leaves values"):
        p.forward(torch.zeros(3, 32, device="cuda"), b, rig.view(0, b))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("dk,dv,dims", [(32, 16, 24), (10, 12, 6), (64, 64, 64)])
def test_rows_normed_whole_and_then_rotated(ops, dtype, interleaved, dk, dv, dims):
    """The store's rotation, which the design leaves out: after the norm, per head, both layouts; padded query heads."""
    nq, nkv, T, page = 4, 2, 9, 4
    D = -(-max(dk, dv) // 16) * 16
    g = torch.Generator().manual_seed(3)
    qkv = torch.randn(T, (nq + nkv) * dk + nkv * dv, generator=g).to(dtype)
    qw, kw = (1 + 0.3 * torch.randn(n * dk, generator=g) for n in (nq, nkv))
    qw, kw = qw.to(dtype), kw.to(dtype)
    first = torch.randn(T, nkv * dv, generator=g).to(dtype)
    share = torch.tensor([0.3])
    pos = torch.tensor([5, 0, 31, 7, 8, 9, 1, 2, 40])
    freq = torch.tensor([100.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    ang = torch.arange(64, dtype=F64)[:, None] * freq[None]
    table = torch.cat([ang.cos(), ang.sin()], -1).float()
    slots = [3, 0, 1, -1, 9, 2, 15, 14, 8]
    pages = torch.full((4, 2, nkv, page, D), float("nan"), dtype=dtype, device="cuda")
    q_out = torch.full((T, nq * D), float("nan"), dtype=dtype, device="cuda")
    ops.row_norm_store(dev(qkv), q_out, D, pages, i32(slots), i32(pos.tolist()), dev(table), dims, nq, nkv, dk, dv, EPS, dev(qw),
                       dev(kw), interleaved=interleaved, v_first=dev(first), v_share=dev(share))

    def turned(x):
        if interleaved:
            return torch.cat([pv.turn_neighbours(x[..., :dims], pos, 100.0), x[..., dims:]], -1)
        half = dims // 2
        c, s = (f(pos.to(F64)[:, None] * freq)[:, None] for f in (torch.cos, torch.sin))
        a, b = x[..., :half], x[..., half:dims]
        return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], -1)

    full = qkv.to(F64)
    q = turned((pv.unit_rms(full[:, :nq * dk], EPS) * qw.to(F64)).reshape(T, nq, dk))
    k = turned((pv.unit_rms(full[:, nq * dk:(nq + nkv) * dk], EPS) * kw.to(F64)).reshape(T, nkv, dk))
    v = pv.mixed_values(full[:, (nq + nkv) * dk:], first.to(F64), float(share)).reshape(T, nkv, dv)
    got_q = q_out.cpu().reshape(T, nq, D)
    close(got_q[..., :dk], q, dtype, bf16=5e-3)
    assert (got_q[..., dk:] == 0).all()
    got = pages.cpu().permute(0, 3, 1, 2, 4).reshape(16, 2, nkv, D)
    for t, s in enumerate(slots):
        if s >= 0:
            close(got[s, 0, :, :dk], k[t], dtype, bf16=5e-3)
            close(got[s, 1, :, :dv], v[t], dtype, bf16=5e-3)
            assert (got[s, 0, :, dk:] == 0).all() and (got[s, 1, :, dv:] == 0).all()
    unused = [s for s in range(16) if s not in slots]
    assert torch.isnan(got[unused].float()).all()


@pytest.mark.parametrize("page,nq,nkv,dk,dv,window", [
    (64, 9, 3, 64, 32, 0), (64, 8, 1, 128, 64, 100), (16, 4, 4, 64, 40, 33), (64, 6, 2, 192, 128, 70), (128, 2, 2, 256, 64, 64),
    (16, 3, 1, 48, 16, 20), (16, 5, 5, 96, 24, 0), (64, 2, 1, 192, 72, 1), (64, 24, 1, 64, 8, 300), (64, 2, 2, 128, 128, 65)])
def test_value_heads_smaller_than_key_heads_on_the_tensor_cores(ops, page, nq, nkv, dk, dv, window):
    """Prompt portions beside single tokens, sinks, windows, against the plain softmax; every kernel that takes the
    shape (tcgen05 and TMA with pages of 64, mma.sync with others and with those switched off)."""
    news, starts = [130, 1, 2, 1, 65, 1], [0, 200, 63, 64, 70, 0]
    ends = [a + b for a, b in zip(news, starts)]
    g = torch.Generator().manual_seed(dk + dv)
    K = [torch.randn(n, nkv, dk, generator=g).bfloat16() for n in ends]
    V = [torch.randn(n, nkv, dv, generator=g).bfloat16() for n in ends]
    Q = [torch.randn(n, nq, dk, generator=g).bfloat16() for n in news]
    sinks = torch.randn(nq, generator=g) * 2
    scale = 1.5 / dk ** 0.5
    for n, s in zip(K, starts):
        n[max(0, s - max(window, 1)):max(0, s - max(window, 1)) + 2] *= 3          # keys at the window's edge stand out
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
        seen = pv.in_window(n, window or None)[starts[s]:]
        heads = []
        for h in range(nq):
            kk, vv = K[s][:, h // (nq // nkv)].to(F64), V[s][:, h // (nq // nkv)].to(F64)
            heads.append(pv.softmax_rows(Q[s][:, h].to(F64) @ kk.T * scale, seen, sinks[h].to(F64)) @ vv)
        want.append(torch.cat(heads, -1))
    want = torch.cat(want)
    q = dev(torch.cat(Q).reshape(cu[-1], nq * dk))
    dpages, dtable = dev(pages), SimpleNamespace(block_tables=dev(table))
    before = ops.USE_TCGEN05_ATTENTION, ops.USE_TMA_DECODE
    try:
        for wide in (True, False):
            ops.USE_TCGEN05_ATTENTION = ops.USE_TMA_DECODE = wide
            out = torch.full((cu[-1], nq * dv), float("nan"), dtype=torch.bfloat16, device="cuda")
            ops.attention_sink(out, q, dpages, dtable, b, nq, nkv, dk, dv, scale, dev(sinks), window)
            close(out.cpu(), want, torch.bfloat16)
    finally:
        ops.USE_TCGEN05_ATTENTION, ops.USE_TMA_DECODE = before
    ops.raise_wait_errors()


# ---------------------------------------------------------------- router and experts
@pytest.mark.parametrize("T,E,top", [(1, 8, 3), (33, 5, 5), (70, 64, 6), (9, 3, 1), (6, 130, 8)])
def test_router_softmax_over_the_chosen_with_a_bias(ops, T, E, top):
    g = torch.Generator().manual_seed(E)
    z, b = torch.randn(T, E, generator=g) * 30, torch.randn(E, generator=g) * 20
    ids, w = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    ops.moe_route(ids, w, dev(z), dev(b), E, 1, 1, scores="chosen_softmax")
    want_ids, want_w = pv.route(z.to(F64), torch.eye(E, dtype=F64), b.to(F64), top)
    assert torch.equal(ids.cpu().long(), want_ids)
    torch.testing.assert_close(w.cpu().to(F64), want_w, rtol=1e-5, atol=1e-6)
    torch.testing.assert_close(w.sum(-1).cpu(), torch.ones(T), rtol=1e-5, atol=1e-5)


def moe_part(dtype, W, E, top, ff, shared, seed):
    from nanohybrid_vlm_b200.parts import FEED_FORWARDS, part
    sh = None if shared is None else part("dense_mlp", intermediate_size=shared, activation="relu2")
    p, w = make_part(FEED_FORWARDS, part("routed_moe", experts=E, top=top, unit="relu2", scores="chosen_softmax", correction=True,
                                         correction_source="router.b", intermediate_size=ff, limit=None, shared=sh,
                                         shared_gate=sh is not None), W, dtype, seed)
    return p, {k: v[0] if v.dim() == 3 else v for k, v in w.items()}


def same_choice(h, w, mlp):
    """Tokens whose choice does not hang on rounding: the last chosen logit well above the first that is not."""
    z = torch.sort(h @ w["router"].T + w["router.b"], -1, descending=True).values
    top, E = mlp["router"]["top"], mlp["router"]["experts"]
    return torch.ones(h.shape[0], dtype=torch.bool) if top == E else (z[:, top - 1] - z[:, top]) > 0.02


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,top,ff,shared", [(1, 64, 6, 2, 32, 48), (50, 100, 5, 3, 18, 26), (300, 128, 4, 1, 72, None),
                                                 (700, 64, 8, 4, 136, 24), (17, 72, 3, 3, 40, 8)])
def test_mixture_without_gates(ops, dtype, T, W, E, top, ff, shared):
    mlp = dict(router=dict(experts=E, top=top), expert=dict(ff=ff), shared=None if shared is None else dict(ff=shared))
    p, w = moe_part(dtype, W, E, top, ff, shared, 31)
    assert "gate" not in {d.name for d in p.params()}
    h = torch.randn(T, W, generator=torch.Generator().manual_seed(T)).to(dtype)
    got = p.forward(dev(h), None).cpu()
    want = pv.mixture(h.to(F64), mlp, w, "")
    sure = same_choice(h.to(F64), w, mlp)
    assert sure.float().mean() > 0.8
    close(got[sure], want[sure], dtype, f32=3e-5, bf16=3e-2)


@pytest.mark.parametrize("tile", [16, 64, 128, "tcgen05", "simt"])
@pytest.mark.parametrize("T,W,E,ff", [(90, 128, 3, 200), (300, 72, 5, 64), (40, 256, 2, 8)])
def test_every_form_of_the_experts_products(ops, tile, T, W, E, ff, monkeypatch):
    """relu(up x)^2 and down over rows ordered by expert, with factors on the experts' inputs too."""
    g = torch.Generator().manual_seed(ff)
    x = torch.randn(T, W, generator=g).bfloat16()
    up, down = (torch.randn(E, ff, W, generator=g) / W ** 0.5).bfloat16(), (torch.randn(E, W, ff, generator=g) / ff ** 0.5).bfloat16()
    ids = torch.stack([torch.randperm(E, generator=g)[:2] for _ in range(T)]).int()
    scale = torch.rand(T, 2, generator=g) + 0.5
    monkeypatch.setattr(ops, "MOE_TCGEN05", tile == "tcgen05")
    monkeypatch.setattr(ops, "MOE_ON_TENSOR_CORES", tile != "simt")
    if isinstance(tile, int):
        monkeypatch.setattr(ops, "MOE_TILE", tile)
    for row_scale in (None, dev(scale)):
        y, pos = ops.moe_experts(dev(x), None, dev(up), dev(down), dev(ids), float("inf"), 1.0, 0.0, row_scale)
        got = y.cpu()[pos.cpu().long()].reshape(T, 2, W)
        for k in range(2):
            xs = x.to(F64) * (1.0 if row_scale is None else scale[:, k:k + 1].to(F64))
            a = torch.relu(torch.einsum("tw,tfw->tf", xs, up.to(F64)[ids[:, k].long()])) ** 2
            want = torch.einsum("tf,twf->tw", a, down.to(F64)[ids[:, k].long()])
            close(got[:, k], want, torch.bfloat16)
    ops.raise_wait_errors()
