"""Kernels of the Nezalorn layers alone: windowed attention with one key that stands out just inside and just
outside the windows, at page, tile and range borders; side-by-side products; the recurrences against double
precision."""
import ctypes as C
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import nezalorn_oracle as oracle  # noqa: E402

pytestmark = pytest.mark.gpu
BS = 16
i32 = lambda x: torch.tensor(np.asarray(x).tolist(), dtype=torch.int32, device="cuda")


def _soft(s, first, last):
    w = torch.full_like(s, 0.0)
    w[first:last + 1] = torch.softmax(s[first:last + 1], 0)
    return w


# ------------------------------------------------------------------------------------ prompts
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 128, 129, 200, 0])
@pytest.mark.parametrize("hq,dq,dv", [(3, 40, 24), (2, 96, 64), (2, 128, 128), (5, 16, 72)])
def test_windowed_prefill_attention(hq, dq, dv, window):
    """Keys at every window's edge are made loud: the first one a query still sees, and the one before it."""
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    g = torch.Generator().manual_seed(dq + window)
    rn = lambda *s: torch.randn(*s, generator=g)
    lens, starts = [150, 2, 130, 33], [0, 128, 127, 240]
    wide = window or 1000
    lo = [max(0, s - wide + 1) // 3 * 2 for s in starts]       # keys from somewhere before the window on
    ctx = [a + b for a, b in zip(lens, starts)]
    rows = [c - a for c, a in zip(ctx, lo)]
    kv0 = np.concatenate([[0], np.cumsum(rows)])
    ldkv = hq * (dq + dv) + 8
    kv = rn(int(kv0[-1]), ldkv) * 0.5
    q = [0.3 * rn(l, hq, dq) for l in lens]
    d = rn(hq, dq)
    d = d / d.norm(dim=1, keepdim=True)
    scale, loud = 0.5, []
    for s in range(4):
        # two loud keys, one apart: for one query they lie on either side of its window's edge
        t = min(lens[s] // 2, lens[s] - 1)
        edge = starts[s] + t - wide + 1
        for p in (edge, edge - 1):
            if lo[s] <= p < ctx[s]:
                kv[int(kv0[s]) + p - lo[s], :hq * dq] = (9.0 * d).reshape(-1)
        q[s] = q[s] + 4.0 * d
        loud.append([t + x for x in (-1, 0, 1)])
    qb, kb = torch.cat(q).reshape(-1, hq * dq).cuda().bfloat16().contiguous(), kv.cuda().bfloat16()
    n = qb.shape[0]
    out = torch.full((n, hq * dv + 8), 7.0, device="cuda", dtype=torch.bfloat16)
    tiles = [(s, t) for s in range(4) for t in range(-(-lens[s] // 128))]
    call("flash_fwd_window", qb, qb.stride(0), kb, kb[:, hq * dq:], ldkv, kb.shape[0], out, out.stride(0),
         i32(np.concatenate([[0], np.cumsum(lens)])), i32(kv0), i32(lo), i32(ctx), i32([t[0] for t in tiles]),
         i32([t[1] for t in tiles]), len(tiles), n, hq, hq, dq, dv, scale, window, None, 0, stream_ptr())
    check_error()
    got, qf, kf = out.cpu().double(), qb.cpu().double(), kb.cpu().double()
    assert bool((got[:, hq * dv:] == 7.0).all())
    row = 0
    for s in range(4):
        k = kf[int(kv0[s]):int(kv0[s + 1])]
        for t in {0, 1, lens[s] // 3, lens[s] - 1, *(x for x in loud[s] if 0 <= x < lens[s])}:
            last = starts[s] + t - lo[s]
            first = max(starts[s] + t - wide + 1, 0) - lo[s] if window else 0
            for h in range(hq):
                sc = k[:, h * dq:(h + 1) * dq] @ qf[row + t, h * dq:(h + 1) * dq] * scale
                want = _soft(sc, max(first, 0), last) @ k[:, hq * dq + h * dv:hq * dq + (h + 1) * dv]
                err = (got[row + t, h * dv:(h + 1) * dv] - want).abs().max()
                assert err < 0.03, (s, t, h, float(err))
        row += lens[s]


# ------------------------------------------------------------------------------------ decoding on latent pages
def _latent_case(hq, rank, rot, ctx, window, seed, dtype):
    from brain_b200.serve import hybrid_native as hn
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g)
    width, B = rank + rot, len(ctx)
    mb = max(-(-c // BS) for c in ctx) + 1
    blocks = B * mb + 3
    pages = torch.full((blocks * BS, width), 30.0)             # what no sequence owns would win every score
    perm, tables, keys, at = torch.randperm(blocks, generator=g), torch.full((B, mb), -1, dtype=torch.int32), [], 0
    d = rn(width)
    d = d / d.norm()
    for s, c in enumerate(ctx):
        k = rn(c, width)
        for p in (c - window, c - window - 1, 0, c // 2) if window else (0, c // 2):
            if 0 <= p < c:
                k[p] = 6.0 * d + 0.5 * rn(width)
        k = k.to(dtype).float()
        keys.append(k)
        for b in range(-(-c // BS)):
            blk = int(perm[at]); at += 1
            tables[s, b] = blk
            n = min(BS, c - b * BS)
            pages[blk * BS:blk * BS + n] = k[b * BS:b * BS + n]
    q = (0.3 * rn(B, hq, width) + 3.0 * d).to(dtype).float()
    qd = torch.zeros(B, hq * width + 16)
    qd[:, :hq * width] = q.reshape(B, -1)
    t = dict(pages=pages.cuda().to(dtype), tables=tables.cuda(), q=qd.cuda().to(dtype), pos=i32([c - 1 for c in ctx]),
             seq=i32(range(B)), out=torch.full((B, hq * rank + 8), 7.0, device="cuda", dtype=dtype),
             po=torch.empty(B * hq * 16 * rank, device="cuda"), pm=torch.empty(B * hq * 16 * 2, device="cuda"))
    cfg, L, b, w = hn.Cfg(), hn.Layer(), hn.Batch(), hn.Work()
    cfg.dtype, cfg.block_size = int(dtype == torch.float32), BS
    L.hq, L.kvrp, L.rotp, L.scale, L.window, L.kc = hq, rank, rot, 0.25, window, t["pages"].data_ptr()
    b.pos, b.tables, b.row_seq, b.max_blocks, b.n, b.ns = (*(t[k].data_ptr() for k in ("pos", "tables", "seq")), mb, B, B)
    w.qa, w.ld_qa, w.ol, w.ld_ol, w.pool_blocks = t["q"].data_ptr(), qd.shape[1], t["out"].data_ptr(), t["out"].shape[1], blocks
    w.part_o, w.part_ml, w.splits = t["po"].data_ptr(), t["pm"].data_ptr(), 16
    want = torch.empty(B, hq, rank, dtype=torch.double)
    for s, c in enumerate(ctx):
        k = keys[s].double()
        first = max(c - window, 0) if window else 0
        for h in range(hq):
            want[s, h] = _soft(k @ q[s, h].double() * 0.25, first, c - 1) @ k[:, :rank]
    return t, (cfg, L, b, w), want


@pytest.mark.parametrize("window", [1, 5, 64, 65, 130, 0])
@pytest.mark.parametrize("hq,rank,rot", [(8, 48, 16), (40, 256, 32), (5, 24, 8), (130, 64, 64), (16, 512, 64), (3, 320, 32)])
@pytest.mark.parametrize("splits", [1, 3, 16])
def test_latent_decode_attention(hq, rank, rot, window, splits):
    from brain_b200.ops._cuda import check_error, lib, stream_ptr
    ctx = [1, 2, 15, 16, 17, 64, 65, 66, 129, 200, 333]
    t, (cfg, L, b, w), want = _latent_case(hq, rank, rot, ctx, window, hq + window, torch.bfloat16)
    w.splits = splits
    assert lib().bb_hy_latent_decode(C.byref(cfg), C.byref(L), C.byref(w), C.byref(b), 0, stream_ptr()) == 0
    check_error()
    got = t["out"].cpu().double()
    assert bool((got[:, hq * rank:] == 7.0).all())
    err = (got[:, :hq * rank].view(-1, hq, rank) - want).abs().amax((1, 2))
    assert float(err.max()) < 0.04, [(c, round(float(e), 4)) for c, e in zip(ctx, err)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hq,rank,rot,window", [(4, 48, 16, 33), (2, 512, 64, 16), (3, 704, 32, 0), (6, 160, 8, 1)])
def test_latent_rows_attention(hq, rank, rot, window, dtype):
    from brain_b200.ops._cuda import lib, stream_ptr
    ctx = [1, 2, 15, 16, 17, 33, 34, 35, 129, 200]
    t, (cfg, L, b, w), want = _latent_case(hq, rank, rot, ctx, window, rank, dtype)
    assert lib().bb_hy_latent_attn(C.byref(cfg), C.byref(L), C.byref(w), C.byref(b), 0, len(ctx), stream_ptr()) == 0
    got = t["out"].cpu().double()[:, :hq * rank].view(-1, hq, rank)
    assert float((got - want).abs().max()) < (3e-5 if dtype == torch.float32 else 0.04)


# ------------------------------------------------------------------------------------ side-by-side products
@pytest.mark.parametrize("M,N,K,G", [(1, 8, 8, 3), (130, 136, 72, 4), (64, 256, 64, 9), (300, 40, 200, 2), (129, 512, 256, 10)])
def test_side_by_side_products(M, N, K, G):
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    g = torch.Generator().manual_seed(M + N)
    a, b = torch.randn(M, G * (K + 8), generator=g), torch.randn(G, N, K, generator=g)
    for dtype, name, tol in ((torch.bfloat16, "gemm_bf16_groups", 0.02), (torch.float32, "sgemm_groups", 2e-6)):
        ad, bd = a.cuda().to(dtype), b.cuda().to(dtype)
        out = torch.full((M, G * (N + 16)), 7.0, device="cuda", dtype=dtype)
        call(name, ad, bd, out, M, N, K, G, ad.stride(0), K + 8, out.stride(0), N + 16, stream_ptr())
        check_error()
        got = out.cpu().double().view(M, G, N + 16)
        want = torch.einsum("mgk,gnk->mgn", ad.cpu().double().view(M, G, K + 8)[:, :, :K], bd.cpu().double())
        assert (got[:, :, :N] - want).abs().max() < tol * want.abs().max() and bool((got[:, :, N:] == 7.0).all())


# ------------------------------------------------------------------------------------ recurrences
def _delta_setup(H, D, lens, starts, seed, dtype, slots):
    from brain_b200.serve import hybrid_native as hn
    pp = hn.pad8(D)
    g = torch.Generator().manual_seed(seed)
    n, ns = sum(lens), len(lens)
    ld = 5 * H * pp + 8
    t = dict(proj=torch.randn(n, ld, generator=g).cuda().to(dtype), low=(torch.randn(n, H * pp, generator=g) * 2).cuda().to(dtype),
             w0=torch.linspace(-9, 0, H * pp).cuda(), ab=(torch.rand(H * pp, generator=g) * 3 - 2).cuda(),
             gain=(1 + 0.1 * torch.randn(H * pp, generator=g)).cuda(),
             init=(0.3 * torch.randn(ns + 2, H, D, D, generator=g)).cuda(), row0=i32(np.concatenate([[0], np.cumsum(lens)])),
             pos0=i32(starts), slots=i32(slots), pos=i32(np.concatenate([np.arange(s, s + l) for s, l in zip(starts, lens)])),
             cat=torch.zeros(n, H * pp, device="cuda", dtype=dtype), y=torch.zeros(n, H * pp, device="cuda", dtype=dtype))
    cfg, L, b, w = hn.Cfg(), hn.Layer(), hn.Batch(), hn.Work()
    cfg.dtype, cfg.eps = int(dtype == torch.float32), 1e-6
    L.heads, L.p, L.pp = H, D, pp
    L.off_r, L.off_kk, L.off_vv, L.off_gg, L.off_a = (i * H * pp for i in range(5))
    L.w0, L.a_b, L.gnorm = (t[k].data_ptr() for k in ("w0", "ab", "gain"))
    b.seq_row0, b.seq_pos0, b.seq_slot, b.pos = (t[k].data_ptr() for k in ("row0", "pos0", "slots", "pos"))
    b.n = b.n_pre = n
    b.ns = b.ns_pre = ns
    w.proj, w.ld_proj, w.aux, w.ld_aux = t["proj"].data_ptr(), ld, t["low"].data_ptr(), H * pp
    w.y, w.ld_y, w.cat, w.ld_cat = t["y"].data_ptr(), H * pp, t["cat"].data_ptr(), H * pp
    return t, (cfg, L, b, w)


def _delta_want(t, H, D, lens, starts, slots):
    pp = t["w0"].numel() // H
    heads = lambda x: x.double().cpu().numpy().reshape(-1, H, pp)[:, :, :D]
    part = lambda i: heads(t["proj"][:, i * H * pp:(i + 1) * H * pp])
    r, k, v, a = part(0), part(1), part(2), oracle.sigmoid(part(4) + heads(t["ab"][None]))
    w = np.exp(-np.exp(-0.5) * oracle.sigmoid(heads(t["low"]) + heads(t["w0"][None])))
    out, states, at = [], t["init"].double().cpu().numpy().copy(), 0
    for l, st, sl in zip(lens, starts, slots):
        o, S = oracle.delta_rule(*(x[at:at + l] for x in (r, k, v, w, a)), states[sl] if st else None)
        out.append(o)
        states[sl] = S
        at += l
    return np.concatenate(out), states


@pytest.mark.parametrize("H,D", [(3, 64), (40, 64), (4, 32), (2, 24), (5, 8), (1, 128), (20, 128), (2, 100), (2, 37)])
def test_delta_scan_keeps_fp32_state(H, D):
    """Both forms of the scan against double precision: portions of many lengths, from zero and from carried
    states, in slots that hold something else."""
    from brain_b200.ops._cuda import check_error, lib, stream_ptr
    lens, starts, slots = [2, 70, 16, 17, 1], [0, 0, 5, 640, 0], [3, 1, 0, 5, 6]
    for dtype, anys in ((torch.bfloat16, (0, 1)), (torch.float32, (0,))):
        t, (cfg, L, b, w) = _delta_setup(H, D, lens, starts, H + D, dtype, slots)
        want, states = _delta_want(t, H, D, lens, starts, slots)
        for form in anys:
            st = t["init"].clone()
            L.ssm_state = st.data_ptr()
            assert lib().bb_hy_delta_scan(C.byref(cfg), C.byref(L), C.byref(w), C.byref(b), form, stream_ptr()) == 0
            check_error()
            y = t["y"].double().cpu().numpy().reshape(-1, H, L.pp)[:, :, :D]
            assert np.abs(st.cpu().numpy() - states).max() < 2e-5 * np.abs(states).max(), (dtype, form)
            assert np.abs(y - want).max() < (2 ** -7 if dtype == torch.bfloat16 else 2e-5) * np.abs(want).max(), (dtype, form)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,D", [(3, 64), (4, 32), (2, 24), (5, 8), (4, 128), (2, 100), (2, 37), (1, 160)])
def test_delta_decode_step(H, D, dtype):
    from brain_b200.ops._cuda import check_error, lib, stream_ptr
    lens, starts, slots = [1] * 5, [0, 7, 1, 300, 0], [3, 1, 0, 5, 6]
    t, (cfg, L, b, w) = _delta_setup(H, D, lens, starts, H + D, dtype, slots)
    b.n_pre = b.ns_pre = 0
    want, states = _delta_want(t, H, D, lens, starts, slots)
    st = t["init"].clone()
    L.ssm_state = st.data_ptr()
    assert lib().bb_hy_delta(C.byref(cfg), C.byref(L), C.byref(w), C.byref(b), stream_ptr()) == 0
    check_error()
    assert np.abs(st.cpu().numpy() - states).max() < 2e-5 * np.abs(states).max()
    pp = L.pp
    heads = lambda x: x.double().cpu().numpy().reshape(-1, H, pp)[:, :, :D]
    gate = oracle.sigmoid(heads(t["proj"][:, 3 * H * pp:4 * H * pp]))
    ref = oracle.rms(want, 1e-6) * heads(t["gain"][None]) * gate
    assert np.abs(heads(t["cat"]) - ref).max() < (0.02 if dtype == torch.bfloat16 else 3e-5) * np.abs(ref).max()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("blocks,bw,taps", [(3, 32, 4), (1, 80, 2), (5, 13, 3), (2, 136, 1)])
def test_gated_linear_recurrence(blocks, bw, taps, dtype):
    """Portions longer and shorter than a block's 128 tokens and single tokens, against double precision, with
    decays from fast to within 1e-5 of one; the kept convolution inputs."""
    from brain_b200.ops._cuda import check_error, lib, stream_ptr
    from brain_b200.serve import hybrid_native as hn
    bwp, g = hn.pad8(bw), torch.Generator().manual_seed(bw)
    chp = blocks * bwp
    lens, starts, slots = [300, 2, 128, 129, 7, 1, 1], [0, 9, 128, 0, 640, 0, 33], [3, 1, 0, 5, 6, 2, 8]
    n, ns, ns_pre = sum(lens), len(lens), 5
    rn = lambda *s: torch.randn(*s, generator=g)
    mask = (torch.arange(chp) % bwp < bw).float()
    dev = lambda x: x.cuda().to(dtype)
    t = dict(proj=dev(rn(n, 2 * chp)), u=dev(rn(n, chp) * mask), gates=dev(rn(n, 2 * chp)), yb=(0.3 * rn(chp)).cuda(),
             rb=rn(chp).cuda(), ib=rn(chp).cuda(), lam=(torch.logspace(-5, 1, chp) * mask).cuda(),
             st=rn(ns + 2, chp).cuda(), ring=dev(rn(ns + 2, max(taps - 1, 1), chp)), cat=torch.zeros(n, chp, device="cuda", dtype=dtype),
             row0=i32(np.concatenate([[0], np.cumsum(lens)])), pos0=i32(starts), slots=i32(slots),
             pos=i32(np.concatenate([np.arange(s, s + l) for s, l in zip(starts, lens)])))
    state0, ring0 = t["st"].double().cpu().numpy(), t["ring"].float().cpu().numpy()
    cfg, L, b, w = hn.Cfg(), hn.Layer(), hn.Batch(), hn.Work()
    cfg.dtype = int(dtype == torch.float32)
    L.blocks, L.bw, L.bwp, L.chp, L.taps, L.off_y, L.off_xbc = blocks, bw, bwp, chp, taps, 0, chp
    L.y_b, L.r_b, L.i_b, L.lam, L.ssm_state, L.conv_state = (t[k].data_ptr() for k in ("yb", "rb", "ib", "lam", "st", "ring"))
    b.seq_row0, b.seq_pos0, b.seq_slot, b.pos = (t[k].data_ptr() for k in ("row0", "pos0", "slots", "pos"))
    b.n, b.n_pre, b.ns, b.ns_pre = n, sum(lens[:ns_pre]), ns, ns_pre
    w.proj, w.ld_proj, w.xbc, w.ld_xbc, w.aux, w.ld_aux = t["proj"].data_ptr(), 2 * chp, t["u"].data_ptr(), chp, t["gates"].data_ptr(), 2 * chp
    w.cat, w.ld_cat = t["cat"].data_ptr(), chp
    assert lib().bb_hy_rglru(C.byref(cfg), C.byref(L), C.byref(w), C.byref(b), stream_ptr()) == 0
    check_error()
    f = lambda k: t[k].double().cpu().numpy()
    gate = f("gates").reshape(n, blocks, 2, bwp)
    r = oracle.sigmoid(gate[:, :, 0].reshape(n, chp) + f("rb"))
    i = oracle.sigmoid(gate[:, :, 1].reshape(n, chp) + f("ib"))
    x = f("lam") * r
    y = oracle.gelu_tanh(f("proj")[:, :chp] + f("yb"))
    at, tol = 0, (3e-5, 3e-5) if dtype == torch.float32 else (5e-5, 2 ** -7)
    for l, s, sl in zip(lens, starts, slots):
        S = state0[sl] if s else np.zeros(chp)
        for k in range(l):
            e = np.expm1(-x[at + k])
            S = S + e * S + np.sqrt(-e * (2 + e)) * i[at + k] * f("u")[at + k]
            want = S * y[at + k]
            assert np.abs(f("cat")[at + k] - want).max() < tol[1] * max(np.abs(want).max(), 1.0), (l, s, k)
        assert np.abs(f("st")[sl] - S).max() < tol[0] * max(np.abs(S).max(), 1.0), (l, s)
        raw = t["proj"].float().cpu().numpy()[at:at + l, chp:]
        for p in range(max(s + l - (taps - 1), 0), s + l):
            ring = t["ring"].float().cpu().numpy()[sl, p % (taps - 1)]
            assert np.array_equal(ring, raw[p - s] if p >= s else ring0[sl, p % (taps - 1)])
        at += l
