"""Kernels of the Povipel layers alone: windowed attention over scattered pages with pooled blocks behind the window, loud
keys and blocks on either side of what a query sees, sinks and outputs turned back; norms, rotations and block means per
head; decaying memories token by token and in chunks against double precision; residual streams; routing by sigmoids."""
import ctypes as C
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import povipel_oracle as oracle  # noqa: E402
from test_hybrid_kernels_gpu import BS, _pools  # noqa: E402

pytestmark = pytest.mark.gpu
i32 = lambda x: torch.tensor(np.asarray(x).tolist(), dtype=torch.int32, device="cuda")
f64 = lambda t: t.double().cpu().numpy()


# ------------------------------------------------------------------------------------ attention
def _request(hq, hk, dk, dv, l, start, window, pool, rn, dtype):
    """Queries that share a direction; the first token of a query's window and the last block it sees have keys along it,
    the token before and the block behind even louder ones."""
    r = lambda t: t.to(dtype).float()
    d = rn(dk)
    d = d / d.norm()
    n = start + l
    k, v, q = 0.5 * rn(n, hk, dk), rn(n, hk, dv), 0.2 * rn(l, hq, dk) + 4.0 * d
    t = l // 2
    i = start + t
    edge = i - window + 1
    seen = edge // pool if edge > 0 else 0               # blocks this query sees
    for b, x in ((seen - 1, 9.0), (seen, 11.0)):
        if 0 <= b and (b + 1) * pool <= n:
            k[b * pool:(b + 1) * pool] = x * d
    for p, x in ((edge, 9.5), (edge - 1, 12.0)):
        if 0 <= p < n:
            k[p] = x * d
    return r(q), r(k), r(v), sorted({0, l - 1, *(x for x in (t - 1, t, t + 1) if 0 <= x < l)})


def _means(k, pool, dtype):
    n = k.shape[0] // pool
    return k[:n * pool].reshape(n, pool, *k.shape[1:]).mean(1).to(dtype).float()


def _expect(q, k, v, pos, scale, window, pool, sink, base, dtype):
    """One query row (double precision) over the keys and means as the cache holds them."""
    hq, g = q.shape[0], q.shape[0] // k.shape[1]
    toks, blocks = oracle.seen(pos, window, pool)
    kk, vv = (f64(torch.cat([x[toks], _means(x, pool, dtype)[blocks]])) for x in (k, v))
    out = []
    for h in range(hq):
        s = kk[:, h // g] @ f64(q[h]) * scale
        top = max(s.max(), sink[h])
        e = np.exp(s - top)
        out.append(e @ vv[:, h // g] / (e.sum() + np.exp(sink[h] - top)))
    o = np.stack(out)[None]
    return oracle.rotate(o, np.array([pos]), o.shape[2], base, True, back=True)[0].reshape(-1)


def _pooled(hk, dk, dv, ks, vs, tables, pool, base, dtype, ctx0, sink):
    """(BbPooled, what it points to): means in the pages of their blocks' last tokens, and as rows; every place that holds
    none has means that would win."""
    from brain_b200.serve import hybrid_native as hn
    rows = -(-BS // pool)
    nb = int(tables.max()) + 4
    pkc, pvc = torch.full((nb, hk, rows, dk), 30.0), torch.full((nb, hk, rows, dv), 100.0)
    total = sum(k.shape[0] for k in ks)
    pk = torch.full((max(total // pool, 1) + 5, hk * (dk + dv)), 30.0)
    tab = tables.cpu()
    for s, (k, v) in enumerate(zip(ks, vs)):
        mk, mv = _means(k, pool, dtype), _means(v, pool, dtype)
        for b in range(mk.shape[0]):
            e = (b + 1) * pool - 1
            pkc[tab[s, e // BS], :, e % BS // pool], pvc[tab[s, e // BS], :, e % BS // pool] = mk[b], mv[b]
            pk[ctx0[s] // pool + b] = torch.cat([mk[b].reshape(-1), mv[b].reshape(-1)])
    ang = torch.arange(600).double()[:, None] * torch.tensor([base ** (-2.0 * i / dv) for i in range(dv // 2)], dtype=torch.float64)
    hold = [t.to("cuda", dtype).contiguous() for t in (pkc, pvc, pk)] + [ang.cos().float().cuda(), ang.sin().float().cuda(), i32(ctx0),
                                                                         torch.tensor(sink, dtype=torch.float32, device="cuda")]
    p = [t.data_ptr() for t in hold]
    x = hn.Pooled(pool, rows, p[0], p[1], p[2], hold[2].shape[1], hold[2].shape[0], p[5], p[6], p[3], p[4], dv)
    return x, hold


BORDERS = [(1, 1), (2, 3), (16, 16), (17, 5), (40, 12), (63, 16), (64, 64), (127, 2), (130, 33), (20, 100)]


@pytest.mark.parametrize("window,pool", BORDERS)
@pytest.mark.parametrize("shape", [(6, 2, 40, 24), (8, 1, 56, 72), (4, 4, 128, 64), (2, 1, 72, 128)])
def test_pooled_prompt_attention(shape, window, pool):
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    hq, hk, dk, dv = shape
    lens, starts = [150, 2, 130, 33], [0, 128, 127, 340]
    ctx = [a + b for a, b in zip(lens, starts)]
    ctx0 = np.concatenate([[0], np.cumsum(ctx)])
    g = torch.Generator().manual_seed(3)
    rn = lambda *s: torch.randn(*s, generator=g)
    sink = (2.0 + 3.0 * rn(hq)).tolist()
    for dtype in (torch.bfloat16, torch.float32):
        qs, ks, vs, rows = zip(*(_request(hq, hk, dk, dv, l, s, window, pool, rn, dtype) for l, s in zip(lens, starts)))
        kc, vc, tables, mb = _pools(ks, vs, ctx, 4, hk, dtype, 5)
        x, hold = _pooled(hk, dk, dv, ks, vs, tables, pool, 70.0, dtype, ctx0, sink)
        ext = C.c_void_p(C.addressof(x))
        q = torch.cat(qs).reshape(-1, hq * dk).to("cuda", dtype).contiguous()
        n = q.shape[0]
        out = torch.full((n, hq * dv + 8), 7.0, device="cuda", dtype=dtype)
        if dtype == torch.bfloat16:
            tiles = [(s, t) for s in range(4) for t in range(-(-lens[s] // 128))]
            call("flash_fwd_paged_p", q, q.stride(0), kc, vc, out, out.stride(0), tables, mb, BS, kc.shape[0],
                 i32(np.concatenate([[0], np.cumsum(lens)])), i32(ctx), i32([t[0] for t in tiles]), i32([t[1] for t in tiles]),
                 len(tiles), n, hq, hk, dk, dv, 0.35, 0.0, None, 0, 0, 1.0, window, ext, stream_ptr())
        else:
            pos = np.concatenate([np.arange(s, s + l) for s, l in zip(starts, lens)])
            call("attn_rows_p", 1, q, q.stride(0), kc, vc, i32(pos), i32(np.repeat(np.arange(4), lens)), tables, mb, BS, out,
                 out.stride(0), None, 0, n, hq, hk, dk, dv, dk, dv, 0.35, 0.0, 0, 1.0, window, ext, stream_ptr())
        check_error()
        got, at = f64(out), 0
        assert (got[:, hq * dv:] == 7.0).all()
        for s in range(4):
            for t in rows[s]:
                want = _expect(qs[s][t], ks[s], vs[s], starts[s] + t, 0.35, window, pool, sink, 70.0, dtype)
                err = np.abs(got[at + t, :hq * dv] - want).max()
                assert err < (0.03 if dtype == torch.bfloat16 else 3e-5), (dtype, s, t, float(err))
            at += lens[s]


@pytest.mark.parametrize("splits", [1, 3, 16])
@pytest.mark.parametrize("window,pool", BORDERS)
@pytest.mark.parametrize("shape", [(6, 2, 40, 24), (8, 1, 56, 72), (3, 1, 128, 128)])
def test_pooled_decode_attention(shape, window, pool, splits):
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    hq, hk, dk, dv = shape
    ctx = [1, 2, 16, 17, 64, 65, 128, 130, 200, 333]
    B, starts = len(ctx), [c - 1 for c in ctx]
    g = torch.Generator().manual_seed(4)
    rn = lambda *s: torch.randn(*s, generator=g)
    sink = (2.0 + 3.0 * rn(hq)).tolist()
    dtype = torch.bfloat16
    qs, ks, vs, _ = zip(*(_request(hq, hk, dk, dv, 1, s, window, pool, rn, dtype) for s in starts))
    kc, vc, tables, mb = _pools(ks, vs, ctx, B, hk, dtype, 5)
    x, hold = _pooled(hk, dk, dv, ks, vs, tables, pool, 70.0, dtype, np.concatenate([[0], np.cumsum(ctx)]), sink)
    q = torch.cat(qs).reshape(B, -1).to("cuda", dtype).contiguous()
    out = torch.zeros(B, hq * dv, device="cuda", dtype=dtype)
    po, pm = torch.empty(B * hq * splits * (64 if dv <= 64 else 128), device="cuda"), torch.empty(B * hq * splits * 2, device="cuda")
    call("paged_decode_p", q, q.stride(0), kc, vc, tables, mb, i32(ctx), out, out.stride(0), po, pm, B, hq, hk, dk, dv, BS, splits,
         0.35, 0.0, None, 0, 0, 1.0, window, C.c_void_p(C.addressof(x)), stream_ptr())
    check_error()
    for s in range(B):
        want = _expect(qs[s][0], ks[s], vs[s], starts[s], 0.35, window, pool, sink, 70.0, dtype)
        assert np.abs(f64(out[s]) - want).max() < 0.03, ctx[s]


# ------------------------------------------------------------------------------------ calls on a layer's structures
class Layer:
    def __init__(self, dtype, eps=1e-3):
        from brain_b200.serve import hybrid_native as hn
        self.L, self.b, self.w, self.cfg = hn.Layer(), hn.Batch(), hn.Work(), hn.Cfg()
        self.dtype, self.hold = dtype, []
        self.cfg.dtype, self.cfg.eps, self.cfg.block_size = int(dtype == torch.float32), eps, BS

    def put(self, where, **tensors):
        for name, t in tensors.items():
            self.hold.append(t)
            setattr(where, name, t.data_ptr())
        return self

    def call(self, name, *args):
        from brain_b200.ops._cuda import check_error, lib, stream_ptr
        fn = getattr(lib(), name)
        fn.restype, fn.argtypes = C.c_int, None
        rc = fn(C.byref(self.cfg), *(C.byref(a) if isinstance(a, C.Structure) else a for a in args), stream_ptr())
        check_error()
        return rc

    def batch(self, lens, starts, dec=0, slots=None):
        b, ns, n = self.b, len(lens), sum(lens)
        b.ns, b.ns_pre, b.n, b.n_pre, b.max_len = ns, ns - dec, n, n - dec, max(lens)
        ctx = [a + s for a, s in zip(lens, starts)]
        b.max_ctx = max(ctx[:ns - dec], default=0)
        tiles = [(s, t) for s in range(ns - dec) for t in range(-(-lens[s] // 128))][::-1]
        b.n_tiles = len(tiles)
        return self.put(b, tile_seq=i32([t[0] for t in tiles]), tile_qt=i32([t[1] for t in tiles]), seq_row0=i32(np.concatenate([[0], np.cumsum(lens)])), seq_pos0=i32(starts), seq_ctx=i32(ctx),
                        seq_slot=i32(slots or range(ns)), pos=i32(np.concatenate([np.arange(s, s + l) for s, l in zip(starts, lens)])),
                        row_seq=i32(np.repeat(np.arange(ns), lens)), ctx_row0=i32(np.concatenate([[0], np.cumsum(ctx)])))


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("hq,hk,dk,dv,rot,pool", [(6, 2, 40, 24, 16, 6), (2, 1, 128, 64, 128, 16), (3, 3, 21, 14, 6, 1),
                                                  (5, 1, 264, 136, 8, 40), (16, 4, 64, 128, 64, 3)])
def test_heads_and_block_means(hq, hk, dk, dv, rot, pool, dtype):
    """Norms, rotations, pages, and the means of blocks that portions and single tokens end, next to blocks of earlier steps."""
    from brain_b200.serve.hybrid_native import pad8
    g = torch.Generator().manual_seed(6)
    rn = lambda *s: torch.randn(*s, generator=g)
    lens, starts = [37, 2, 70, 1, 1, 1], [0, 39, 51, 0, 47, 2 * pool - 1]
    dkp, dvp, n = pad8(dk), pad8(dv), sum(lens)
    padded = lambda heads, size, sizep: torch.nn.functional.pad(rn(n, heads, size), (0, sizep - size)).reshape(n, -1)
    q, k, v = padded(hq, dk, dkp), padded(hk, dk, dkp), padded(hk, dv, dvp)
    proj = torch.cat([rn(n, 8), q, k, v], 1).to("cuda", dtype).contiguous()
    before = f64(proj)
    t = Layer(dtype).batch(lens, starts, dec=3)
    L, b, w, base, window = t.L, t.b, t.w, 90.0, 9
    ns = len(lens)
    mb = max(-(-(a + s) // BS) for a, s in zip(lens, starts))
    tables = torch.randperm(ns * mb, generator=g).reshape(ns, mb)
    gain = (1.0 + 0.2 * rn(2, dk))
    angles = lambda d: torch.arange(512).double()[:, None] * torch.tensor([base ** (-2.0 * i / d) for i in range(d // 2)], dtype=torch.float64)
    old_k, old_v = rn(ns * mb, hk, BS, dkp).to("cuda", dtype), rn(ns * mb, hk, BS, dvp).to("cuda", dtype)
    rows = -(-BS // pool)
    kc, vc = old_k.clone(), old_v.clone()
    pkc, pvc = (torch.full((ns * mb, hk, rows, d), 7.0, device="cuda", dtype=dtype) for d in (dkp, dvp))
    pk = torch.full((sum(lens) + sum(starts), hk * (dkp + dvp)), 7.0, device="cuda", dtype=dtype)
    L.hq, L.hk, L.dk, L.dv, L.dkp, L.dvp, L.rot, L.head_norm, L.pool, L.pool_rows, L.window = hq, hk, dk, dv, dkp, dvp, rot, 1, pool, rows, window
    L.off_q, L.off_k, L.off_v = 8, 8 + hq * dkp, 8 + (hq + hk) * dkp
    pad = lambda x: torch.nn.functional.pad(x, (0, dkp - dk)).cuda().contiguous()
    t.put(L, q_norm=pad(gain[0]), k_norm=pad(gain[1]), cos_t=angles(rot).cos().float().cuda(), sin_t=angles(rot).sin().float().cuda(),
          vcos_t=angles(dv).cos().float().cuda(), vsin_t=angles(dv).sin().float().cuda(), kc=kc, vc=vc, pkc=pkc, pvc=pvc)
    t.put(b, tables=tables.to("cuda", torch.int32).contiguous()).put(w, proj=proj, pk=pk)
    b.max_blocks, w.ld_proj, w.ld_pk, w.pk_rows = mb, proj.shape[1], pk.shape[1], pk.shape[0]
    assert t.call("bb_hy_heads", L, w, b) == 0
    assert t.call("bb_hy_pool", L, w, b, 1) == 0
    tol = 1e-2 if dtype == torch.bfloat16 else 2e-6
    at, off = 0, lambda p, h, size: before[:, p:p + h * size].reshape(n, h, size)
    want_q = off(8, hq, dkp)[..., :dk]
    want_k, want_v = off(8 + hq * dkp, hk, dkp)[..., :dk], off(8 + (hq + hk) * dkp, hk, dvp)[..., :dv]
    want_q, want_k = (oracle.rms(x, 1e-3) * f64(g_) for x, g_ in ((want_q, gain[0]), (want_k, gain[1])))
    got_q = f64(proj)[:, 8:8 + hq * dkp].reshape(n, hq, dkp)
    assert np.array_equal(f64(proj)[:, :8], before[:, :8]) and (got_q[..., dk:] == 0).all()
    ctx0 = 0
    for s, (l, st) in enumerate(zip(lens, starts)):
        pos = np.arange(st, st + l)
        turn = lambda x, d: oracle.rotate(x[at:at + l], pos, d, base, True)
        wq, wk, wv = turn(want_q, rot), turn(want_k, rot), turn(want_v, dv)
        assert np.abs(got_q[at:at + l, :, :dk] - wq).max() < tol * 4
        gather = lambda pages, lo, hi: np.stack([f64(pages[tables[s, p // BS], :, p % BS]) for p in range(lo, hi)])
        gk, gv = gather(kc, 0, st + l), gather(vc, 0, st + l)
        assert np.abs(gk[st:, :, :dk] - wk).max() < tol * 4 and np.abs(gv[st:, :, :dv] - wv).max() < tol * 4
        assert (gk[st:, :, dk:] == 0).all() and (gv[st:, :, dv:] == 0).all()
        if st:
            assert np.array_equal(gk[:st], gather(old_k, 0, st)) and np.array_equal(gv[:st], gather(old_v, 0, st))
        for blk in range((st + l) // pool):
            e = (blk + 1) * pool - 1
            mk, mv = (x[blk * pool:e + 1].mean(0) for x in (gk, gv))
            page, place = tables[s, e // BS], e % BS // pool
            if e >= st:                              # ends in this step
                assert np.abs(f64(pkc[page, :, place]) - mk).max() < tol and np.abs(f64(pvc[page, :, place]) - mv).max() < tol
            else:
                assert (pkc[page, :, place] == 7.0).all() and (pvc[page, :, place] == 7.0).all()
            if s < 3 and e <= st + l - 1 - window:   # a query of the portion sees it
                row = torch.cat([pkc[page, :, place].reshape(-1), pvc[page, :, place].reshape(-1)])
                assert torch.equal(pk[ctx0 // pool + blk], row)
        at += l
        ctx0 += st + l


# ------------------------------------------------------------------------------------ decaying memories
LENS, STARTS = [2, 300, 128, 129, 15, 700, 7], [0, 0, 5, 640, 64, 128, 0]


class Memory(Layer):
    """Random projections and states of a layer of linear attention; ``decay``: one per head, or None for a token's own."""

    def __init__(self, H, N, P, lens, starts, dtype, decay=None, root=0.2, rot=0, seed=1, dec=0, bias=2.0, slots=None,
                 eps=1e-3):
        from brain_b200.serve.hybrid_native import Lin, pad8
        super().__init__(dtype, eps)
        g = torch.Generator().manual_seed(seed)
        rn = lambda *s: torch.randn(*s, generator=g)
        self.batch(lens, starts, dec, slots)
        self.H, self.N, self.P, self.lens, self.starts, self.slots = H, N, P, lens, starts, slots or list(range(len(lens)))
        np_, pp, n, R = pad8(N), pad8(P), sum(lens), 16
        self.np, self.pp, self.n, self.rot, self.base = np_, pp, n, rot, 40.0
        head = lambda size, sizep: torch.nn.functional.pad(rn(n, H, size), (0, sizep - size)).reshape(n, -1)
        k, q, v, gate = head(N, np_), head(N, np_), head(P, pp), head(P, pp)
        low, w2, w0 = rn(n, R), rn(H, np_, R) / 4, bias + rn(H, np_)
        self.proj = torch.cat([rn(n, 8), k, q, v, gate, low], 1).to("cuda", dtype).contiguous()
        rounded = f64(self.proj)
        cut = lambda o, size, sizep: rounded[:, o:o + H * sizep].reshape(n, H, sizep)[:, :, :size]
        o = [8, 8 + H * np_, 8 + 2 * H * np_, 8 + 2 * H * np_ + H * pp, 8 + 2 * H * (np_ + pp)]
        self.k, self.q, self.v, self.g = cut(o[0], N, np_), cut(o[1], N, np_), cut(o[2], P, pp), cut(o[3], P, pp)
        L, w = self.L, self.w
        L.heads = L.groups = H
        L.n, L.p, L.np, L.pp, L.q_scale = N, P, np_, pp, N ** -0.5
        L.off_kk, L.off_q, L.off_vv, L.off_gg, L.off_w1 = o
        self.init = rn(len(lens) + 2, H, N, P)
        self.state = self.init.cuda()
        self.gain = 1.0 + 0.2 * rn(P)
        self.y = torch.full((n, H * pp + 8), 7.0, device="cuda", dtype=dtype)
        self.cat = self.y.clone()
        self.put(L, ssm_state=self.state, gnorm=torch.nn.functional.pad(self.gain.repeat(H, 1), (0, pp - P)).reshape(-1).cuda())
        self.put(w, proj=self.proj, y=self.y, cat=self.cat)
        w.ld_proj, w.ld_y, w.ld_cat = self.proj.shape[1], self.y.shape[1], self.cat.shape[1]
        if decay is None:
            w2 = w2.to(dtype)
            L.decay_root, L.wr, L.wrp = root, R, R
            z = torch.tensor(rounded[:, o[4]:]) @ w2.double().reshape(-1, R).T
            self.z = torch.cat([z.float(), torch.full((n, H * np_), 7.0)], 1).cuda().contiguous()
            w.ld_f32 = self.z.shape[1]
            slots = self.b.n_pre // 128 + self.b.ns_pre
            self.flags = i32(np.full(slots * H, 9))
            self.put(w, chunks=torch.full((slots * H * N * P,), float("nan"), device="cuda"), chunk_flags=self.flags)
            w.chunk_floats, w.chunk_marks = slots * H * N * P, slots * H
            dev = w2.cuda().contiguous()
            self.put(w, f32=self.z).put(L, w0=w0.float().reshape(-1).cuda())
            self.hold.append(dev)
            L.w2 = Lin(dev.data_ptr(), H * np_, R)
            self.w0, self.root = w0.float(), root
            self.decays()
        else:
            d = np.asarray(decay, dtype=np.float64)
            self.put(L, keep_less=torch.tensor(d - 1.0).float().cuda(), a=torch.tensor(np.log(d)).float().cuda())
            self.alpha = np.broadcast_to(d[None, :, None], (n, H, N))
        if rot:
            ang = torch.arange(2048).double()[:, None] * torch.tensor([self.base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
            L.rot = rot
            self.put(L, cos_t=ang.cos().float().cuda(), sin_t=ang.sin().float().cuda())

    def decays(self):
        z = (self.z[:, :self.H * self.np].cpu() + self.w0.reshape(-1)).double().reshape(self.n, self.H, self.np)[:, :, :self.N].numpy()
        self.alpha = np.exp(-np.logaddexp(0.0, -z) * np.float32(self.root))

    def b_rows(self, s):
        return sum(self.lens[:s]), sum(self.lens[:s + 1])

    def check(self, rows, tol, state_tol, first=0):
        """Finished rows and states of the sequences from ``first`` on, against double precision."""
        ys, ends, at = [], [], 0
        for s, l in enumerate(self.lens):
            pos = np.arange(self.starts[s], self.starts[s] + l)
            turn = lambda x: oracle.rotate(x[at:at + l], pos, self.rot, self.base, True)
            S = f64(self.init[self.slots[s]]) if self.starts[s] else None
            o, end = oracle.decayed_memory(turn(self.q) * self.N ** -0.5, turn(self.k), self.v[at:at + l], self.alpha[at:at + l], S)
            ys.append(o)
            ends.append(end)
            at += l
        want = oracle.rms(np.concatenate(ys), self.cfg.eps) * f64(self.gain) * oracle.silu(self.g)
        lo = sum(self.lens[:first])
        got = f64(rows)[:, :self.H * self.pp].reshape(self.n, self.H, self.pp)
        scale = np.maximum(np.abs(want[lo:]).max(axis=(1, 2), keepdims=True), 0.5)
        assert (np.abs(got[lo:, :, :self.P] - want[lo:]) / scale).max() < tol
        assert (got[lo:, :, self.P:] == 0).all() and (f64(rows)[:, self.H * self.pp:] == 7.0).all()
        for s in range(first, len(self.lens)):
            x = f64(self.state[self.slots[s]])
            assert np.abs(x - ends[s]).max() < state_tol * np.abs(ends[s]).max(), s
        rest = [i for i in range(len(self.lens) + 2) if i not in self.slots]
        assert torch.equal(self.state.cpu()[rest], self.init[rest])


SIZES = [(3, 24, 40), (2, 128, 128), (5, 13, 21), (2, 8, 8), (1, 200, 24), (1, 300, 16), (4, 64, 64), (1, 16, 520), (40, 40, 72)]
SLOTS = [3, 1, 0, 5, 8, 2, 4]


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,N,P", SIZES)
def test_scan_with_a_tokens_own_decays(H, N, P, dtype):
    m = Memory(H, N, P, LENS, STARTS, dtype, slots=SLOTS)
    assert m.call("bb_hy_linear_scan", m.L, m.w, m.b, 0) == 0
    m.check(m.cat, 0.02 if dtype == torch.bfloat16 else 1e-4, 1e-5)


@pytest.mark.parametrize("bias", [-40.0, 12.0, 90.0])
def test_scan_with_decays_near_zero_and_one(bias):
    m = Memory(2, 40, 24, [900, 3], [0, 700], torch.float32, bias=bias, root=1.0)
    assert m.call("bb_hy_linear_scan", m.L, m.w, m.b, 0) == 0
    m.check(m.cat, 2e-4, 1e-5)


@pytest.mark.parametrize("root,bias", [(0.1, 2.0), (0.9, 0.0), (1e-3, 5.0)])
@pytest.mark.parametrize("H,N,P", [(3, 24, 40), (4, 64, 64), (2, 64, 128), (5, 13, 21), (2, 8, 8), (6, 40, 104), (1, 56, 72)])
def test_chunks_with_a_tokens_own_decays(H, N, P, root, bias):
    m = Memory(H, N, P, LENS, STARTS, torch.bfloat16, root=root, bias=bias, slots=SLOTS)
    assert m.call("bb_gla_chunk", m.L, m.w, m.b) == 0
    assert m.call("bb_hy_linear_scan", m.L, m.w, m.b, 1) == 0
    m.check(m.cat, 0.02, 3e-5)


def test_pairs_that_decay_too_fast_for_chunks_go_to_the_scan():
    """One head's channel decays by e^-2 a token in one sequence, another's by e^-40: chunks leave both pairs alone, portions
    too short for that much stay, and nobody else notices."""
    m = Memory(3, 24, 40, LENS, STARTS, torch.bfloat16, root=1.0, bias=3.0, slots=SLOTS)
    a, b = m.b_rows(1), m.b_rows(5)
    for rows, h, ch, z in ((a, 0, 5, -2.0), (b, 2, 0, -40.0)):
        m.z[rows[0]:rows[1], h * m.np + ch] = z - m.w0[h, ch]
    m.decays()
    assert m.call("bb_gla_chunk", m.L, m.w, m.b) == 0
    flags, slot0 = m.flags.cpu().numpy().reshape(-1, 3), [sum(LENS[:s]) // 128 + s for s in range(len(LENS))]
    marked = {(s, h) for s in range(len(LENS)) for h in range(3) if flags[slot0[s]:slot0[s] + -(-LENS[s] // 128), h].any()}
    assert marked == {(1, 0), (5, 2)}
    assert m.call("bb_hy_linear_scan", m.L, m.w, m.b, 1) == 0
    m.check(m.cat, 0.02, 3e-5)


def test_chunks_refuse_what_their_scratch_does_not_hold():
    m = Memory(3, 24, 40, LENS, STARTS, torch.bfloat16)
    m.w.chunk_floats -= 1
    assert m.call("bb_gla_chunk", m.L, m.w, m.b) == -3
    for N, P in ((72, 40), (24, 136)):
        m = Memory(1, N, P, [3], [0], torch.bfloat16)
        assert m.call("bb_gla_chunk", m.L, m.w, m.b) == -3


@pytest.mark.parametrize("segments", [False, True])
@pytest.mark.parametrize("H,N,P,rot", [(4, 24, 40, 24), (2, 128, 128, 64), (3, 64, 64, 64), (2, 72, 64, 0), (1, 64, 128, 32),
                                       (5, 13, 21, 6), (2, 8, 8, 8)])
def test_retention_in_chunks(H, N, P, rot, segments):
    """Portions of many lengths, from zero and from carried states; with and without scratch for segments side by side."""
    decay = [1.0 - 2.0 ** (-1.0 - 2.7 * h) for h in range(H)]
    m = Memory(H, N, P, LENS, STARTS, torch.bfloat16, decay=decay, rot=rot, slots=SLOTS, eps=0.2)
    if segments:
        m.put(m.w, seg=torch.full((8 << 20,), float("nan"), device="cuda"))
        m.w.seg_floats = 8 << 20
    assert m.call("bb_hy_turn", m.L, m.w, m.b) == 0
    assert m.call("bb_retention_chunk", m.L, m.w, m.b) == 0
    assert m.call("bb_hy_linear_post", m.L, m.w, m.n) == 0
    # rotated queries and keys are rounded to bf16, as in the scan below: their product may nearly cancel
    m.check(m.cat, 0.08 if rot else 0.02, 0.01 if rot else 1e-4)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,N,P,rot", [(4, 24, 40, 24), (1, 136, 9, 64), (2, 40, 200, 40)])
def test_scan_with_constant_decays(H, N, P, rot, dtype):
    m = Memory(H, N, P, LENS, STARTS, dtype, decay=[1.0 - 1e-4 * 9.0 ** h for h in range(H)], rot=rot, slots=SLOTS, eps=0.2)
    assert m.call("bb_hy_turn", m.L, m.w, m.b) == 0
    assert m.call("bb_hy_linear_scan", m.L, m.w, m.b, 0) == 0
    m.check(m.cat, 0.08 if dtype == torch.bfloat16 else 1e-4, 0.01 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("own", [True, False])
@pytest.mark.parametrize("H,N,P", [(3, 24, 40), (2, 128, 128), (5, 13, 21), (1, 300, 16), (1, 16, 520), (160, 40, 72)])
def test_decode_steps(H, N, P, own, dtype):
    """Single tokens behind a portion: fresh ones (whatever the slot holds) and others."""
    lens, starts = [5] + [1] * 6, [0, 0, 3, 1, 64, 300, 0]
    m = Memory(H, N, P, lens, starts, dtype, decay=None if own else [0.9 + 0.1 * (h + 1) / H for h in range(H)],
               rot=0 if own else N // 2 * 2, dec=6, slots=SLOTS)
    m.state[[SLOTS[1], SLOTS[6]]] = float("nan")
    assert m.call("bb_hy_linear_decode", m.L, m.w, m.b) == 0
    m.check(m.cat, 0.02 if dtype == torch.bfloat16 else 1e-4, 1e-5, first=1)


# ------------------------------------------------------------------------------------ residual streams
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 6, 16])
@pytest.mark.parametrize("source", ["embedding", "one", "two", "experts", "weighed"])
@pytest.mark.parametrize("d", [24, 100, 2056])
def test_streams(d, source, S, dtype):
    from brain_b200.serve import hybrid_native as hn
    g = torch.Generator().manual_seed(8)
    rn = lambda *s: torch.randn(*s, generator=g)
    dp, eps, scale = hn.pad8(d), 1e-3, 1.5
    lens, starts = [5, 2, 1, 1, 1], [0, 7, 0, 3, 9]
    t = Layer(dtype, eps).batch(lens, starts, dec=3, slots=[2, 0, 4, 1, 3])
    n, cfg, w, b = sum(lens), t.cfg, t.w, t.b
    few = dtype == torch.bfloat16                    # few rows of a bf16 step: results are sums in fp32
    pad = lambda x: torch.nn.functional.pad(x, (0, dp - d))
    low = lambda x: pad(x).to("cuda", dtype).contiguous()
    x, emb = pad(rn(n, S, d)).cuda().contiguous(), low(rn(11, d))
    ya, yb, ex = low(rn(n, d)), low(3.0 * rn(n, d)), low(rn(3 * n, d))
    if few:
        ya, yb = (pad(rn(n, d)).cuda().contiguous() for _ in range(2))
    ya0, yb0 = ya.clone(), yb.clone()
    gains = 1.0 + 0.3 * rn(6, d)
    cfg.width, cfg.dp, cfg.vocab, cfg.embed_scale, cfg.streams = d, dp, 11, scale, S
    layers = (hn.Layer * 2)()
    before, after, side = layers[0], layers[1], hn.Layer()
    hc = [torch.cat([rn(S) / S, rn(S), torch.eye(S).reshape(-1) + 0.3 * rn(S * S)]).cuda() for _ in range(3)]
    before.hc[0], before.hc[1], after.hc[0] = (h.data_ptr() for h in hc)
    vec = lambda v: pad(v).float().cuda().contiguous()
    shift = torch.rand(d, generator=g)
    state0 = pad(rn(6, d)).to(dtype)
    state = state0.cuda()
    h, h2 = torch.full((n, dp), 7.0, device="cuda", dtype=dtype), torch.full((n, dp), 7.0, device="cuda", dtype=dtype)
    fq = 1 if source in ("experts", "weighed") else 0
    top = 2
    rows = torch.randperm(3 * n, generator=g)[:n * top]
    pw = torch.rand(n * top, generator=g)
    if source == "two":
        t.put(before, out_gain=vec(gains[0])).put(side, out_gain=vec(gains[1]))
        before.beside = C.addressof(side)
    if fq:
        before.n_experts, before.top, before.weigh_input = 9, top, int(source == "experts")
    toks = rn(n).mul(7).long().abs() % 11
    trace = torch.zeros(n, dp, device="cuda")
    t.put(after, norm=vec(gains[2]), norm_b=vec(gains[3]), shift=vec(shift), shift_state=state)
    t.put(cfg, embed=emb, final_norm=vec(gains[4]), final_norm_b=vec(gains[5]))
    t.put(w, **({"ya32": ya, "yb32": yb} if few else {"ya": ya, "yb": yb}))
    if few:
        after.beside = C.addressof(side)             # (both results of the next sublayer are added into zeros)
    t.put(w, x=x, ex_out=ex, pair_row=i32(rows), pair_w=pw.cuda(), h=h, h2=h2, ex_count=i32(np.zeros(9)))
    t.put(b, tok=i32(toks))
    X = f64(x)[:, :, :d].transpose(1, 0, 2)
    part = lambda i: f64(hc[i])
    cut = lambda y: f64(y)[:, :d]
    if source == "embedding":
        X = np.repeat(cut(emb)[toks.numpy()][None] * scale, S, axis=0)
    else:
        y = {"one": lambda: cut(ya), "two": lambda: oracle.rms(cut(ya), eps) * f64(gains[0]) + oracle.rms(cut(yb), eps) * f64(gains[1]),
             "experts": lambda: cut(ex)[rows.numpy()].reshape(n, top, d).sum(1),
             "weighed": lambda: (cut(ex)[rows.numpy()] * f64(pw)[:, None]).reshape(n, top, d).sum(1)}[source]()
        X = oracle.streams_out(X, y, part(fq)[2 * S:].reshape(S, S), part(fq)[S:2 * S])
    want = oracle.layer_norm(oracle.streams_in(X, part(2)[:S]), f64(gains[2]), f64(gains[3]), eps)
    null = C.c_void_p(None)
    src = null if source == "embedding" else C.byref(before)
    behind = source != "embedding"
    assert t.call("bb_hy_streams", src, fq, after, 0, w, b, 0, C.c_void_p(trace.data_ptr()) if behind else null) == 0
    tol = 2e-2 if dtype == torch.bfloat16 else 1e-4
    top_abs = max(np.abs(X).max(), 1.0)
    assert np.abs(f64(x)[:, :, :d].transpose(1, 0, 2) - X).max() < 2e-5 * top_abs
    assert bool((ya == 0).all() and (yb == 0).all()) == few
    ya.copy_(ya0), yb.copy_(yb0)
    if behind:
        assert np.abs(f64(trace)[:, :d] - X.sum(0)).max() < 1e-4 * top_abs
    # rows of portions are shifted by a second kernel, single tokens at once; both leave the last input in the slot
    assert np.abs(f64(h2)[:7, :d] - want[:7]).max() < tol * 4 and (h2[7:] == 7.0).all()
    assert t.call("bb_hy_shift", after, w, b) == 0
    at = 0
    for s, l in enumerate(lens):
        slot = [2, 0, 4, 1, 3][s]
        prev = f64(state0[slot])[:d] if starts[s] else np.zeros(d)
        u = want[at:at + l]
        sh = u + (np.concatenate([prev[None], u[:-1]]) - u) * f64(shift)
        assert np.abs(f64(h)[at:at + l, :d] - sh).max() < tol * 4, s
        assert np.abs(f64(state)[slot, :d] - u[-1]).max() < tol * 4, s
        assert (f64(h)[at:at + l, d:] == 0).all()
        at += l
    assert torch.equal(state.cpu()[5], state0[5])
    # the end: wanted rows of the streams' sum, from the same sources
    last = torch.zeros(3, dp, device="cuda", dtype=dtype)
    t.put(w, hn=last).put(b, want=i32([6, 0, 9]))
    b.n_want = 3
    if behind:
        assert t.call("bb_hy_streams", src, fq, null, 0, w, b, 0, null) == 0
        X2 = oracle.streams_out(X, y, part(fq)[2 * S:].reshape(S, S), part(fq)[S:2 * S]).sum(0)[[6, 0, 9]]
        want = oracle.layer_norm(X2, f64(gains[4]), f64(gains[5]), eps)
        assert np.abs(f64(last)[:, :d] - want).max() < tol * 4


@pytest.mark.parametrize("few", [True, False])
@pytest.mark.parametrize("E,top,d", [(4, 1, 40), (10, 3, 120), (72, 8, 64), (300, 5, 64)])
def test_sigmoid_routing_and_weighed_rows(E, top, d, few):
    """Choices, weights as they are, and experts' rows that the weight multiplies."""
    from brain_b200.serve import hybrid_native as hn
    g = torch.Generator().manual_seed(9)
    n, dtype = (50 if few else 300), torch.bfloat16
    t = Layer(dtype)
    L, w, cfg = t.L, t.w, t.cfg
    cfg.width = cfg.dp = d
    h, router = torch.randn(n, d, generator=g).to("cuda", dtype), (torch.randn(hn.pad8(E), d, generator=g) / 8).to("cuda", dtype)
    router[E:] = 0
    L.n_experts, L.top, L.groups_all, L.groups_keep, L.route_scale, L.score_kind, L.weigh_input = E, top, 1, 1, 1.0, 1, 1
    L.in32 = hn.Lin(router.data_ptr(), router.shape[0], d)
    moe = 128 * (n * top // 128 + min(n * top, E))
    f32 = torch.zeros(n, router.shape[0], device="cuda")
    pe, pr, pw = i32(np.zeros(n * top)), i32(np.zeros(n * top)), torch.zeros(n * top, device="cuda")
    rows, tile = torch.zeros(moe, d, device="cuda", dtype=dtype), i32(np.zeros(moe // 64))
    part = torch.zeros(-(-d // 64) * n * router.shape[0], device="cuda")
    t.put(w, h=h, f32=f32, pair_expert=pe, pair_row=pr, pair_w=pw, ex_count=i32(np.zeros(E)), ex_in=rows, ex_tile=tile, part32=part)
    w.ld_f32, w.moe_rows, w.part32_floats = f32.shape[1], moe, part.numel()
    z = f64(h) @ f64(router[:E]).T
    if few:
        rc = t.call("bb_hy_route_row", L, w, n)
        if E > 256:
            assert rc == -3
            return
        assert rc == 0
    else:
        f32[:, :E] = torch.tensor(z[:, :E]).float().cuda()
        assert t.call("bb_hy_route", L, w, n) == 0
    assert t.call("bb_hy_expert_rows", L, w, n) == 0
    ge, gw, gr = pe.cpu().numpy().reshape(n, top), f64(pw).reshape(n, top), pr.cpu().numpy().reshape(n, top)
    for i in range(n):
        s = np.sort(z[i])[::-1]
        want = oracle.route(z[i], top)
        if top < E and s[top - 1] - s[top] > 1e-4:
            assert sorted(ge[i]) == sorted(e for e, _ in want), i
        for c in range(top):
            assert abs(gw[i, c] - oracle.sigmoid(z[i, ge[i, c]])) < 1e-5
            assert np.abs(f64(rows[gr[i, c]]) - f64(h[i]) * gw[i, c]).max() < 0.02 and tile[gr[i, c] // 128] == ge[i, c]
    assert len(set(gr.reshape(-1).tolist())) == n * top
