"""Kernels of the hybrid decoders alone: attention over scattered pages with one key that stands out, at page,
tile and split borders, with keys just outside what a query sees made loud; fp32 GEMM; fp32 heads."""
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

pytestmark = pytest.mark.gpu
BS = 16


def _pools(k, v, ctx, n_seq, hk, dtype, seed):
    """Pages of several sequences, scattered over the pool; every place no sequence owns holds a key that
    would win every score, and values that would show."""
    dk, dv = k[0].shape[-1], v[0].shape[-1]
    mb = max(-(-c // BS) for c in ctx) + 1
    n_blocks = n_seq * mb + 3
    g = torch.Generator().manual_seed(seed)
    perm = torch.randperm(n_blocks, generator=g)
    kc = torch.full((n_blocks, hk, BS, dk), 30.0)
    vc = torch.full((n_blocks, hk, BS, dv), 100.0)
    tables = torch.full((n_seq, mb), -1, dtype=torch.int32)
    at = 0
    for s in range(n_seq):
        nb = -(-ctx[s] // BS)
        for b in range(nb):
            blk = int(perm[at]); at += 1
            tables[s, b] = blk
            n = min(BS, ctx[s] - b * BS)
            kc[blk, :, :n] = k[s][b * BS:b * BS + n].permute(1, 0, 2)
            vc[blk, :, :n] = v[s][b * BS:b * BS + n].permute(1, 0, 2)
    return kc.to("cuda", dtype), vc.to("cuda", dtype), tables.cuda(), mb


def _expect(q, k, v, pos, scale, softcap, gate):
    """One query row [hq, dk] against keys 0..pos (double precision)."""
    hq, g = q.shape[0], q.shape[0] // k.shape[1]
    out = []
    for h in range(hq):
        s = (k[:pos + 1, h // g].double() @ q[h].double()) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        out.append(torch.softmax(s, 0) @ v[:pos + 1, h // g].double() * torch.sigmoid(gate[h].double()))
    return torch.stack(out)


def _case(hq, hk, dk, dv, lens, starts, loud, seed, dtype):
    """Random requests; the key at ``loud`` of every sequence is along one direction all its queries share."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g)
    r = lambda t: t.to(dtype).float()
    ks, vs, qs, gs = [], [], [], []
    for l, st in zip(lens, starts):
        k, v, q = rn(st + l, hk, dk), rn(st + l, hk, dv), 0.3 * rn(l, hq, dk)
        q += rn(1, 1, dk) if loud is None else 0
        if loud is not None and loud < st + l:
            d = rn(dk)
            d = d / d.norm()
            q = q + 4.0 * d
            k[loud] = 12.0 * d
        ks.append(r(k)); vs.append(r(v)); qs.append(r(q)); gs.append(r(rn(l, hq)))
    return qs, ks, vs, gs


SHAPES = [(6, 2, 40, 24), (8, 1, 56, 72), (4, 4, 128, 64), (6, 3, 64, 128), (5, 1, 72, 88)]


@pytest.mark.parametrize("softcap", [0.0, 20.0])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("loud", [0, 1, 15, 16, 63, 64, 127, 128, 129, 255, None])
def test_prefill_attention(shape, loud, softcap):
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    hq, hk, dk, dv = shape
    scale = 0.35
    lens, starts = [150, 2, 130, 33], [0, 128, 127, 240]
    ctx = [a + b for a, b in zip(lens, starts)]
    for dtype in (torch.bfloat16, torch.float32):
        qs, ks, vs, gs = _case(hq, hk, dk, dv, lens, starts, loud, 7, dtype)
        kc, vc, tables, mb = _pools(ks, vs, ctx, 4, hk, dtype, 11)
        q, gate = torch.cat(qs).reshape(-1, hq * dk), torch.cat(gs)
        n = q.shape[0]
        ldg = 16
        gp = torch.zeros(n, ldg)
        gp[:, :hq] = gate
        dq, dg = q.to("cuda", dtype).contiguous(), gp.to("cuda", dtype)
        out = torch.full((n, hq * dv + 8), 7.0, device="cuda", dtype=dtype)
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
        if dtype == torch.bfloat16:
            tiles = [(s, t) for s in range(4) for t in range(-(-lens[s] // 128))]
            call("flash_fwd_paged_x", dq, dq.stride(0), kc, vc, out, out.stride(0), tables, mb, BS, kc.shape[0],
                 i32(np.concatenate([[0], np.cumsum(lens)]).tolist()), i32(ctx), i32([t[0] for t in tiles]),
                 i32([t[1] for t in tiles]), len(tiles), n, hq, hk, dk, dv, scale, softcap, dg, ldg, 0, 1.0, 0, stream_ptr())
        else:
            pos = np.concatenate([np.arange(s, s + l) for s, l in zip(starts, lens)])
            seq = np.repeat(np.arange(4), lens)
            call("attn_rows", 1, dq, dq.stride(0), kc, vc, i32(pos.tolist()), i32(seq.tolist()), tables, mb, BS, out,
                 out.stride(0), dg, ldg, n, hq, hk, dk, dv, dk, dv, scale, softcap, 0, 1.0, 0, stream_ptr())
        check_error()
        got = out.cpu().float()
        assert bool((got[:, hq * dv:] == 7.0).all())
        row = 0
        for s in range(4):
            for t in (0, 1, lens[s] // 2, lens[s] - 1):
                want = _expect(qs[s][t], ks[s], vs[s], starts[s] + t, scale, softcap, gs[s][t]).reshape(-1)
                err = (got[row + t, :hq * dv].double() - want).abs().max()
                assert err < (0.03 if dtype == torch.bfloat16 else 2e-5), (dtype, s, t, float(err))
            row += lens[s]


@pytest.mark.parametrize("softcap", [0.0, 20.0])
@pytest.mark.parametrize("shape", SHAPES + [(14, 2, 8, 8), (3, 1, 16, 120)])
@pytest.mark.parametrize("splits", [1, 3, 16])
def test_decode_attention(shape, splits, softcap):
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    hq, hk, dk, dv = shape
    scale = 0.35
    ctx = [1, 2, 15, 16, 17, 64, 65, 128, 200, 333]
    for loud in (0, 1, 16, 31, 32, 64, 127, 199, None):
        for dtype in (torch.bfloat16, torch.float32):
            starts = [c - 1 for c in ctx]
            qs, ks, vs, gs = _case(hq, hk, dk, dv, [1] * len(ctx), starts, loud, 3, dtype)
            kc, vc, tables, mb = _pools(ks, vs, ctx, len(ctx), hk, dtype, 5)
            B = len(ctx)
            dq = torch.cat(qs).reshape(B, -1).to("cuda", dtype).contiguous()
            gp = torch.zeros(B, 16)
            gp[:, :hq] = torch.cat(gs)
            dg = gp.to("cuda", dtype)
            out = torch.zeros(B, hq * dv, device="cuda", dtype=dtype)
            i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
            if dtype == torch.bfloat16:
                po = torch.empty(B * hq * splits * (64 if dv <= 64 else 128), device="cuda")
                pm = torch.empty(B * hq * splits * 2, device="cuda")
                call("paged_decode_x", dq, dq.stride(0), kc, vc, tables, mb, i32(ctx), out, out.stride(0), po, pm, B, hq,
                     hk, dk, dv, BS, splits, scale, softcap, dg, 16, 0, 1.0, 0, stream_ptr())
            else:
                call("attn_rows", 1, dq, dq.stride(0), kc, vc, i32(starts), i32(list(range(B))), tables, mb, BS, out,
                     out.stride(0), dg, 16, B, hq, hk, dk, dv, dk, dv, scale, softcap, 0, 1.0, 0, stream_ptr())
            check_error()
            got = out.cpu()
            for s in range(B):
                want = _expect(qs[s][0], ks[s], vs[s], starts[s], scale, softcap, gs[s][0]).reshape(-1)
                err = (got[s].double() - want).abs().max()
                assert err < (0.03 if dtype == torch.bfloat16 else 2e-5), (dtype, loud, ctx[s], float(err))


@pytest.mark.parametrize("M,N,K", [(1, 8, 8), (70, 130, 50), (64, 64, 16), (257, 36, 300)])
def test_fp32_gemm_is_fp32(M, N, K):
    from brain_b200.ops._cuda import call, stream_ptr
    g = torch.Generator().manual_seed(M)
    a, b, c = (torch.randn(*s, generator=g) for s in ((M, K), (N, K), (M, N)))
    for acc in (0, 1):
        out = c.cuda()
        call("sgemm", a.cuda(), b.cuda(), out, M, N, K, K, K, N, 0.7, acc, stream_ptr())
        want = 0.7 * (a.double() @ b.double().t()) + (c.double() if acc else 0)
        assert (out.cpu().double() - want).abs().max() < 3e-6 * K ** 0.5 * 4


def test_fp32_argmax_and_topk():
    from brain_b200.ops import functional as F
    g = torch.Generator().manual_seed(0)
    lg = torch.randn(5, 1032, generator=g)
    lg[0, 77] = lg[0, 900] = 9.0          # the lowest index wins a tie
    lg[1, 3] = 5.0
    lg[1, 4] = 5.0 + 1e-6                 # closer than bf16 can tell
    view = lg.cuda()[:, :1000]
    assert F.argmax_rows(view).cpu().tolist() == [77, 4] + lg[2:, :1000].argmax(1).tolist()
    idx, val = F.topk_rows(view, 20)
    tv = torch.topk(lg[:, :1000], 20).values
    assert torch.equal(val.cpu(), tv) and idx[0, :2].cpu().tolist() == [77, 900]


@pytest.mark.parametrize("segments", [False, True])
@pytest.mark.parametrize("H,P,N,G", [(4, 64, 128, 1), (2, 128, 128, 2), (6, 16, 24, 3), (3, 40, 64, 1), (2, 72, 72, 1),
                                     (8, 32, 8, 4), (5, 8, 120, 5)])
def test_chunked_recurrence_keeps_fp32_state(H, P, N, G, segments):
    """The tensor-core chunks against the token-by-token fp32 scan on the same bf16 inputs: portions of
    many lengths, from zero and from carried states, in slots that hold something else; with and without
    scratch to run a portion's segments side by side."""
    import ctypes as C
    from brain_b200.ops._cuda import check_error, lib, stream_ptr
    from brain_b200.serve import hybrid_native as hn
    g = torch.Generator().manual_seed(H * P + N)
    lens, starts = [2, 300, 128, 129, 15, 1500, 7], [0, 0, 5, 640, 64, 128, 0]
    ns, n = len(lens), sum(lens)
    inner, ch = H * P, H * P + 2 * G * N
    ldx = (ch + 7) // 8 * 8 + 8
    xbc = torch.randn(n, ldx, generator=g).to("cuda", torch.bfloat16)
    dt = torch.nn.functional.softplus(torch.randn(n, H, generator=g) - 1.0).cuda()
    a = -torch.exp(torch.rand(H, generator=g) * 5 - 4).cuda()
    d = torch.randn(H, generator=g).cuda()
    init = torch.randn(ns + 2, H, N, P, generator=g).cuda()
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    row0, pos0 = i32(np.concatenate([[0], np.cumsum(lens)]).tolist()), i32(starts)
    slots = i32([3, 1, 0, 5, 8, 2, 4])
    cfg, L, b, w = hn.Cfg(), hn.Layer(), hn.Batch(), hn.Work()
    L.heads, L.p, L.n, L.groups, L.inner, L.ch = H, P, N, G, inner, ch
    L.a, L.d_skip = a.data_ptr(), d.data_ptr()
    b.seq_row0, b.seq_pos0, b.seq_slot, b.n_pre, b.ns_pre, b.ns, b.n = \
        row0.data_ptr(), pos0.data_ptr(), slots.data_ptr(), n, ns, ns, n
    w.xbc, w.ld_xbc, w.dt, w.ld_dt, w.ld_y = xbc.data_ptr(), ldx, dt.data_ptr(), H, inner
    seg = torch.full((4 << 20,), float("nan"), device="cuda")
    b.max_len = max(lens)
    if segments:
        w.seg, w.seg_floats = seg.data_ptr(), seg.numel()
    out = {}
    for name in ("bb_ssd_chunk", "bb_hy_ssm_scan"):
        y, st = torch.zeros(n, inner, device="cuda", dtype=torch.bfloat16), init.clone()
        L.ssm_state, w.y = st.data_ptr(), y.data_ptr()
        assert getattr(lib(), name)(C.byref(cfg), C.byref(L), C.byref(w), C.byref(b), stream_ptr()) == 0
        check_error()
        out[name] = (y.float().cpu(), st.cpu())
    (y1, s1), (y2, s2) = out["bb_ssd_chunk"], out["bb_hy_ssm_scan"]
    assert (s1 - s2).abs().max() < 3e-5 * s2.abs().max()
    untouched = [i for i in range(ns + 2) if i not in slots.tolist()]
    assert torch.equal(s1[untouched], init.cpu()[untouched])
    assert (y1 - y2).abs().max() < 2 ** -7 * y2.abs().max()
    # two roundings of the same value to bf16: almost every output is bit-equal
    assert (y1 != y2).float().mean() < 0.02
