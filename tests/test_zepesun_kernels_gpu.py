"""Kernels of the Zepesun layers alone: windowed attention over scattered pages with a loud key on either side of a
query's window and a gate on every element; the matrix memory in chunks and token by token against double precision;
routing and the experts' rows."""
import ctypes as C
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import zepesun_oracle as oracle  # noqa: E402
from test_hybrid_kernels_gpu import BS, _pools  # noqa: E402

pytestmark = pytest.mark.gpu
i32 = lambda x: torch.tensor(np.asarray(x).tolist(), dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------------------------ windowed attention
def _windowed(hq, hk, dk, dv, lens, starts, window, seed, dtype):
    """Random requests with a key that wins where it is seen, at every place a query's window begins and one before."""
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g)
    r = lambda t: t.to(dtype).float()
    d = rn(dk)
    d = d / d.norm()
    ks, vs, qs, gs, rows = [], [], [], [], []
    for l, st in zip(lens, starts):
        k, v, q = rn(st + l, hk, dk), rn(st + l, hk, dv), 0.3 * rn(l, hq, dk) + 4.0 * d
        t = l // 2
        edge = st + t - (window or 1 << 20) + 1
        for p in (edge, edge - 1):
            if 0 <= p < st + l:
                k[p] = (9.0 if p == edge else 12.0) * d
        ks.append(r(k)); vs.append(r(v)); qs.append(r(q)); gs.append(r(rn(l, hq * dv)))
        rows.append(sorted({0, l - 1, *(x for x in (t - 1, t, t + 1) if 0 <= x < l)}))
    return qs, ks, vs, gs, rows


def _row(q, k, v, pos, scale, window, gate, factor):
    hq, n = q.shape[0], k.shape[1]
    a = max(0, pos - window + 1) if window else 0
    out = [torch.softmax(k[a:pos + 1, h // (hq // n)].double() @ q[h].double() * scale, 0) @ v[a:pos + 1, h // (hq // n)].double()
           for h in range(hq)]
    return factor * torch.cat(out) * torch.sigmoid(gate.double())


WINDOWS = [1, 2, 15, 16, 17, 63, 64, 65, 127, 128, 129, 200, 0]


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("shape", [(6, 2, 40, 24), (8, 1, 56, 72), (4, 4, 128, 64), (2, 1, 72, 128)])
def test_windowed_prompt_attention(shape, window):
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    hq, hk, dk, dv = shape
    lens, starts = [150, 2, 130, 33], [0, 128, 127, 240]
    ctx = [a + b for a, b in zip(lens, starts)]
    for dtype in (torch.bfloat16, torch.float32):
        qs, ks, vs, gs, rows = _windowed(hq, hk, dk, dv, lens, starts, window, 3, dtype)
        kc, vc, tables, mb = _pools(ks, vs, ctx, 4, hk, dtype, 5)
        q = torch.cat(qs).reshape(-1, hq * dk).to("cuda", dtype).contiguous()
        gate = torch.cat(gs).to("cuda", dtype).contiguous()
        n = q.shape[0]
        out = torch.full((n, hq * dv + 8), 7.0, device="cuda", dtype=dtype)
        if dtype == torch.bfloat16:
            tiles = [(s, t) for s in range(4) for t in range(-(-lens[s] // 128))]
            call("flash_fwd_paged_x", q, q.stride(0), kc, vc, out, out.stride(0), tables, mb, BS, kc.shape[0],
                 i32(np.concatenate([[0], np.cumsum(lens)])), i32(ctx), i32([t[0] for t in tiles]), i32([t[1] for t in tiles]),
                 len(tiles), n, hq, hk, dk, dv, 0.35, 0.0, gate, gate.stride(0), 1, 0.6, window, stream_ptr())
        else:
            pos = np.concatenate([np.arange(s, s + l) for s, l in zip(starts, lens)])
            call("attn_rows", 1, q, q.stride(0), kc, vc, i32(pos), i32(np.repeat(np.arange(4), lens)), tables, mb, BS, out,
                 out.stride(0), gate, gate.stride(0), n, hq, hk, dk, dv, dk, dv, 0.35, 0.0, 1, 0.6, window, stream_ptr())
        check_error()
        got, at = out.cpu().double(), 0
        assert bool((got[:, hq * dv:] == 7.0).all())
        for s in range(4):
            for t in rows[s]:
                want = _row(qs[s][t], ks[s], vs[s], starts[s] + t, 0.35, window, gs[s][t], 0.6)
                err = (got[at + t, :hq * dv] - want).abs().max()
                assert err < (0.02 if dtype == torch.bfloat16 else 2e-5), (dtype, s, t, float(err))
            at += lens[s]


@pytest.mark.parametrize("splits", [1, 3, 16])
@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("shape", [(6, 2, 40, 24), (8, 1, 56, 72), (3, 1, 128, 128)])
def test_windowed_decode_attention(shape, window, splits):
    from brain_b200.ops._cuda import call, check_error, stream_ptr
    hq, hk, dk, dv = shape
    ctx = [1, 2, 16, 17, 64, 65, 128, 130, 200, 333]
    B, starts = len(ctx), [c - 1 for c in ctx]
    qs, ks, vs, gs, _ = _windowed(hq, hk, dk, dv, [1] * B, starts, window, 4, torch.bfloat16)
    kc, vc, tables, mb = _pools(ks, vs, ctx, B, hk, torch.bfloat16, 5)
    q, gate = (torch.cat(x).reshape(B, -1).to("cuda", torch.bfloat16).contiguous() for x in (qs, gs))
    out = torch.zeros(B, hq * dv, device="cuda", dtype=torch.bfloat16)
    po, pm = torch.empty(B * hq * splits * (64 if dv <= 64 else 128), device="cuda"), torch.empty(B * hq * splits * 2, device="cuda")
    call("paged_decode_x", q, q.stride(0), kc, vc, tables, mb, i32(ctx), out, out.stride(0), po, pm, B, hq, hk, dk, dv, BS, splits,
         0.35, 0.0, gate, gate.stride(0), 1, 0.6, window, stream_ptr())
    check_error()
    for s in range(B):
        want = _row(qs[s][0], ks[s], vs[s], starts[s], 0.35, window, gs[s][0], 0.6)
        assert (out[s].cpu().double() - want).abs().max() < 0.02, ctx[s]


# ------------------------------------------------------------------------------------ matrix memory
class Memory:
    """Random projections, raw gates and states of one layer, and what the kernels' structures say of them."""

    def __init__(self, H, N, P, lens, starts, dtype, cap=3.0, forget=2.0, slots=None, seed=1, dec=0):
        from brain_b200.serve import hybrid_native as hn
        g = torch.Generator().manual_seed(seed)
        rn = lambda *s: torch.randn(*s, generator=g)
        self.H, self.N, self.P, self.lens, self.starts, self.dtype, self.cap = H, N, P, lens, starts, dtype, cap
        np_, pp = hn.pad8(N), hn.pad8(P)
        self.np, self.pp = np_, pp
        ns, n = len(lens), sum(lens)
        head = lambda size, sizep: torch.nn.functional.pad(rn(n, H, size), (0, sizep - size)).reshape(n, -1)
        self.k, self.q, self.v, self.g = (head(s, p).to(dtype) for s, p in ((N, np_), (N, np_), (P, pp), (P, pp)))
        self.raw = torch.cat([rn(n, 3), 1.5 * rn(n, H), 1.5 * rn(n, H)], 1)
        self.b = (rn(H), forget + 0.3 * rn(H))
        self.gain = 1.0 + 0.2 * rn(H, P)
        self.mem = -(-(N * P + N + 1) // 4) * 4 + 4
        self.init = rn(ns + 2, H, self.mem)
        self.slots = slots or list(range(ns))[::-1]
        L, b, w, cfg = hn.Layer(), hn.Batch(), hn.Work(), hn.Cfg()
        self.L, self.b_, self.w, self.cfg = L, b, w, cfg
        self.ns, self.n, self.dec = ns, n, dec
        L.heads, L.groups, L.n, L.p, L.np, L.pp, L.mem, L.gate_cap, L.q_scale = H, H, N, P, np_, pp, self.mem, cap, N ** -0.5
        L.off_kk, L.off_q, L.off_vv, L.off_gg = 8, 8 + H * np_, 8 + 2 * H * np_, 8 + 2 * H * np_ + H * pp
        L.off32_i, L.off32_f = 3, 3 + H
        cfg.dtype, cfg.eps = int(dtype == torch.float32), 1e-3
        b.ns, b.ns_pre, b.n, b.n_pre, b.max_len = ns, ns - dec, n, n - dec, max(lens)

    def tensors(self):
        pad = torch.full((self.n, 8), 3.0, dtype=self.dtype)
        t = dict(proj=torch.cat([pad, self.k, self.q, self.v, self.g, pad], 1).cuda().contiguous(), raw=self.raw.cuda(),
                 i_b=self.b[0].cuda(), f_b=self.b[1].cuda(),
                 gain=torch.nn.functional.pad(self.gain, (0, self.pp - self.P)).reshape(-1).cuda(),
                 state=self.init.cuda(), row0=i32(np.concatenate([[0], np.cumsum(self.lens)])), pos0=i32(self.starts),
                 slot=i32(self.slots), pos=i32(np.concatenate([np.arange(s, s + l) for s, l in zip(self.starts, self.lens)])),
                 y=torch.full((self.n, self.H * self.pp + 8), 7.0, device="cuda", dtype=self.dtype))
        t["cat"] = t["y"].clone()
        L, b, w = self.L, self.b_, self.w
        L.i_b, L.f_b, L.gnorm, L.ssm_state = (t[k].data_ptr() for k in ("i_b", "f_b", "gain", "state"))
        b.seq_row0, b.seq_pos0, b.seq_slot, b.pos = (t[k].data_ptr() for k in ("row0", "pos0", "slot", "pos"))
        w.proj, w.ld_proj, w.f32, w.ld_f32 = t["proj"].data_ptr(), t["proj"].shape[1], t["raw"].data_ptr(), self.raw.shape[1]
        w.y, w.ld_y, w.cat, w.ld_cat = t["y"].data_ptr(), t["y"].shape[1], t["cat"].data_ptr(), t["cat"].shape[1]
        return t

    def call(self, name, *args):
        from brain_b200.ops._cuda import check_error, lib, stream_ptr
        fn = getattr(lib(), name)
        fn.restype, fn.argtypes = C.c_int, None
        at = [C.byref(a) if isinstance(a, C.Structure) else a for a in args]
        assert fn(C.byref(self.cfg), C.byref(self.L), C.byref(self.w), *at, stream_ptr()) == 0
        check_error()

    def expect(self):
        """(outputs of the recurrence, finished rows, states (S, n, m) per sequence), in double precision."""
        d = lambda t: t.double().numpy()
        cut = lambda t, size, sizep: d(t).reshape(self.n, self.H, sizep)[:, :, :size]
        i, f = oracle.gates(d(self.raw[:, 3:3 + self.H] + self.b[0]), d(self.raw[:, 3 + self.H:3 + 2 * self.H] + self.b[1]), self.cap)
        q, k, v = cut(self.q, self.N, self.np) * self.N ** -0.5, cut(self.k, self.N, self.np), cut(self.v, self.P, self.pp)
        ys, states, at = [], [], 0
        for s, l in enumerate(self.lens):
            st = None
            if self.starts[s] > 0:
                x = d(self.init[self.slots[s]])
                NP = self.N * self.P
                st = (x[:, :NP].reshape(self.H, self.N, self.P), x[:, NP:NP + self.N], x[:, NP + self.N])
            o, end = oracle.matrix_memory(*(a[at:at + l] for a in (q, k, v, i, f)), st)
            ys.append(o)
            states.append(end)
            at += l
        y = np.concatenate(ys)
        done = oracle.rms(y, self.cfg.eps) * d(self.gain) * oracle.sigmoid(cut(self.g, self.P, self.pp))
        return y, done, states

    def check(self, t, rows, states, tol, state_tol, first=0):
        got = rows.cpu().double().numpy()[:, :self.H * self.pp].reshape(self.n, self.H, self.pp)
        y, done, want_states = self.expect()
        want = done if rows is t["cat"] else y
        lo = sum(self.lens[:first])
        scale = np.abs(want[lo:]).max(axis=(1, 2), keepdims=True)
        assert (np.abs(got[lo:, :, :self.P] - want[lo:]) / scale).max() < tol
        x = t["state"].cpu().double().numpy()
        for s in range(first, self.ns):
            S, nn, m = want_states[s]
            NP = self.N * self.P
            g = x[self.slots[s]]
            assert np.abs(g[:, :NP].reshape(S.shape) - S).max() < state_tol * np.abs(S).max(), s
            assert np.abs(g[:, NP:NP + self.N] - nn).max() < state_tol * np.abs(nn).max(), s
            assert np.abs(g[:, NP + self.N] - m).max() < state_tol * 10, s
        rest = [i for i in range(self.ns + 2) if i not in self.slots]
        assert torch.equal(t["state"].cpu()[rest], self.init[rest])


SIZES = [(4, 24, 40), (2, 128, 128), (6, 16, 16), (3, 64, 64), (2, 72, 64), (1, 64, 128), (3, 40, 104), (5, 13, 21), (2, 8, 8)]
LENS, STARTS = [2, 300, 128, 129, 15, 1100, 7], [0, 0, 5, 640, 64, 128, 0]


@pytest.mark.parametrize("segments", [False, True])
@pytest.mark.parametrize("H,N,P", SIZES)
def test_memory_in_chunks(H, N, P, segments):
    """Portions of many lengths, from zero and from carried states, in slots that hold something else; with and without
    scratch to run a portion's segments side by side."""
    m = Memory(H, N, P, LENS, STARTS, torch.bfloat16, slots=[3, 1, 0, 5, 8, 2, 4])
    t = m.tensors()
    seg = torch.full((8 << 20,), float("nan"), device="cuda")
    if segments:
        m.w.seg, m.w.seg_floats = seg.data_ptr(), seg.numel()
    m.call("bb_hy_mlstm_gates", m.n)
    m.call("bb_mlstm_chunk", m.b_)
    m.check(t, t["cat"], t["state"], 0.02, 1e-4)
    got = t["cat"].cpu().float()
    assert bool((got[:, H * m.pp:] == 7.0).all())
    assert bool((got[:, :H * m.pp].view(m.n, H, m.pp)[:, :, P:] == 0).all())


@pytest.mark.parametrize("N,P,segments", [(64, 64, True), (64, 64, False), (128, 128, True), (24, 40, False)])
@pytest.mark.parametrize("far", [0, 1, 127, 128, 255, 640])
def test_far_token_in_the_memory(far, N, P, segments):
    """One token with an open input gate and a key that later queries share, everything else nearly shut: it is found
    a thousand tokens later, over chunks, segments and a portion's end."""
    lens, starts = [700, 500], [0, 0]
    m = Memory(2, N, P, lens, starts, torch.bfloat16, cap=12.0, forget=12.0)
    m.raw[:, 3:5] = -6.0
    m.raw[:, 5:] = 12.0
    d = torch.randn(N, generator=torch.Generator().manual_seed(2))
    for r0, l in ((0, 700), (700, 500)):
        if far < l:
            m.raw[r0 + far, 3:5] = 12.0
            m.k.view(m.n, 2, -1)[r0 + far, :, :N] = d.to(m.k.dtype)
            q = m.q.view(m.n, 2, -1)
            q[r0 + far + 1:r0 + l, :, :N] = (0.2 * q[r0 + far + 1:r0 + l, :, :N].float() + d).to(q.dtype)
    t = m.tensors()
    seg = torch.zeros(8 << 20, device="cuda")
    if segments:
        m.w.seg, m.w.seg_floats = seg.data_ptr(), seg.numel()
    m.call("bb_hy_mlstm_gates", m.n)
    m.call("bb_mlstm_chunk", m.b_)
    m.check(t, t["cat"], t["state"], 0.02, 1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,N,P", SIZES + [(1, 150, 200), (2, 33, 260), (1, 300, 12)])
def test_memory_token_by_token(H, N, P, dtype):
    lens = [min(l, 150) for l in LENS]
    m = Memory(H, N, P, lens, STARTS, dtype, slots=[3, 1, 0, 5, 8, 2, 4])
    t = m.tensors()
    m.call("bb_hy_mlstm_scan", m.b_, 0, m.ns)
    m.check(t, t["y"], t["state"], 2e-5 if dtype == torch.float32 else 0.01, 2e-5)
    assert bool((t["y"].cpu().float()[:, H * m.pp:] == 7.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,N,P", SIZES + [(1, 150, 200), (2, 33, 260), (1, 300, 12), (1, 256, 512)])
def test_memory_decode(H, N, P, dtype):
    """One token per sequence behind a prompt portion, from zero and from carried states."""
    lens, starts = [5] + [1] * 6, [0, 0, 1, 77, 0, 500, 3]
    m = Memory(H, N, P, lens, starts, dtype, slots=[3, 1, 0, 5, 8, 2, 4], dec=6)
    t = m.tensors()
    m.call("bb_hy_mlstm_decode", m.b_)
    m.slots[0] = m.ns + 1          # the portion's own slot is not touched by this call
    # (random keys: a normaliser close to zero magnifies the rounding of its sum)
    m.check(t, t["cat"], t["state"], 2e-4 if dtype == torch.float32 else 0.01, 2e-5, first=1)


# ------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("E,top,groups,keep", [(12, 3, 4, 2), (8, 2, 1, 1), (5, 5, 5, 5), (64, 8, 8, 4), (72, 7, 2, 1), (256, 8, 8, 4),
                                               (300, 32, 3, 2), (1, 1, 1, 1), (1024, 6, 32, 5)])
@pytest.mark.parametrize("n", [1, 7, 300, 5000])
def test_routing_and_rows(E, top, groups, keep, n):
    from brain_b200.ops._cuda import check_error, lib, stream_ptr
    from brain_b200.serve import hybrid_native as hn
    rng = np.random.default_rng(E + n)
    z = (3.0 * rng.standard_normal((n, E))).astype(np.float32)
    if E > 2:
        z[:, E // 2] += 4.0          # one expert that most tokens choose
    dp, ldz = 40, E + 5
    for dtype in (torch.bfloat16, torch.float32):
        h = torch.randn(n, dp, device="cuda").to(dtype)
        logits = torch.zeros(n, ldz, device="cuda")
        logits[:, :E] = torch.from_numpy(z)
        L, w, cfg = hn.Layer(), hn.Work(), hn.Cfg()
        cfg.dtype, cfg.dp = int(dtype == torch.float32), dp
        L.n_experts, L.top, L.groups_all, L.groups_keep, L.route_scale, L.route_tiny = E, top, groups, keep, 1.7, 1e-20
        tiles = lib().bb_hy_moe_tiles(C.byref(L), n)
        t = dict(ex_in=torch.zeros(tiles * 128, dp, device="cuda", dtype=dtype), pair_expert=i32(np.zeros(n * top)),
                 pair_row=i32(np.zeros(n * top)), pair_w=torch.zeros(n * top, device="cuda"), ex_count=i32(np.zeros(E)),
                 ex_tile=i32(np.full(2 * tiles + 1, 99)))
        for k, v in t.items():
            setattr(w, k, v.data_ptr())
        w.h, w.f32, w.ld_f32, w.moe_rows = h.data_ptr(), logits.data_ptr(), ldz, tiles * 128
        for fn in ("bb_hy_route", "bb_hy_expert_rows"):
            f = getattr(lib(), fn)
            f.restype = C.c_int
            assert f(C.byref(cfg), C.byref(L), C.byref(w), n, stream_ptr()) == 0
        check_error()
        expert, row, weight = (t[k].cpu().numpy().reshape(n, top) for k in ("pair_expert", "pair_row", "pair_w"))
        spec = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}, "scale": 1.7}
        for i in range(n) if n < 400 else rng.integers(0, n, 200):
            want = oracle.route(z[i].astype(np.float64), spec)
            assert expert[i].tolist() == [e for e, _ in want]
            assert np.allclose(weight[i], [x for _, x in want], rtol=2e-5, atol=1e-9)
        tile = t["ex_tile"].cpu().numpy()
        assert tile[2 * tiles] == 99 and len(set(row.ravel().tolist())) == n * top and row.max() < tiles * 128
        assert np.array_equal(tile[row // 128], expert)
        assert t["ex_count"].cpu().numpy().tolist() == np.bincount(expert.ravel(), minlength=E).tolist()
        assert torch.equal(t["ex_in"][torch.from_numpy(row.ravel()).long().cuda()], h.repeat_interleave(top, 0))
        # every expert's rows lie on as many tiles as they need
        assert np.array_equal(tile[tiles:2 * tiles], np.bincount(row.ravel() // 128, minlength=tiles))
        for e in range(E):
            assert (tile[:tiles] == e).sum() == -(-int((expert == e).sum()) // 128)


@pytest.mark.parametrize("E,top,groups,keep,more", [(12, 3, 4, 2, 6), (0, 0, 1, 1, 8), (64, 8, 8, 4, 0), (200, 5, 2, 1, 10)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_products_and_routing_of_few_rows(E, top, groups, keep, more, dtype):
    from brain_b200.ops._cuda import check_error, lib, stream_ptr
    from brain_b200.serve import hybrid_native as hn
    n, dp, g = 70, 136, torch.Generator().manual_seed(E)
    outs = hn.pad8(E) + hn.pad8(more)
    h, W = (torch.randn(*s, generator=g).to(dtype) for s in ((n, dp), (outs, dp)))
    hd, wd, out = h.cuda(), W.cuda(), torch.full((n, outs + 3), 7.0, device="cuda")
    L, w, cfg = hn.Layer(), hn.Work(), hn.Cfg()
    cfg.dtype, cfg.dp = int(dtype == torch.float32), dp
    L.in32 = hn.Lin(wd.data_ptr(), outs, dp)
    L.n_experts, L.top, L.groups_all, L.groups_keep, L.route_scale, L.route_tiny = E, top, groups, keep, 0.6, 1e-20
    pe, pr, pw, count = i32(np.zeros(n * top + 1)), i32(np.zeros(n * top + 1)), torch.zeros(n * top + 1, device="cuda"), i32(np.zeros(E + 1))
    part = torch.full((-(-dp // 64) * n * outs,), float("nan"), device="cuda")
    w.h, w.f32, w.ld_f32, w.part32, w.part32_floats = hd.data_ptr(), out.data_ptr(), outs + 3, part.data_ptr(), part.numel()
    w.pair_expert, w.pair_row, w.pair_w, w.ex_count = (x.data_ptr() for x in (pe, pr, pw, count))
    fn = lib().bb_hy_route_row
    fn.restype = C.c_int
    assert fn(C.byref(cfg), C.byref(L), C.byref(w), n, stream_ptr()) == 0
    check_error()
    want = h.double() @ W.double().t()
    assert (out[:, :outs].cpu().double() - want).abs().max() < 2e-5 and bool((out[:, outs:] == 7.0).all())
    if E:
        expert, row, weight = (x[:-1].cpu().numpy().reshape(n, top) for x in (pe, pr, pw))
        z, spec = out.cpu().double().numpy(), {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}, "scale": 0.6}
        for i in range(n):
            ref = oracle.route(z[i, :E], spec)
            assert expert[i].tolist() == [e for e, _ in ref] and np.allclose(weight[i], [x for _, x in ref], rtol=2e-5)
        for e in range(E):
            assert sorted(row[expert == e].tolist()) == list(range(int(count[e])))


@pytest.mark.parametrize("G,N,K", [(3, 72, 40), (2, 8, 130), (1, 130, 8)])
def test_fp32_tiles(G, N, K):
    from brain_b200.ops._cuda import call, stream_ptr
    g = torch.Generator().manual_seed(N)
    a, b = torch.randn(512, K, generator=g), torch.randn(G, N, K, generator=g)
    tiles = [G - 1, -1, 0, G // 2]
    out = torch.full((512, N), 7.0, device="cuda")
    call("sgemm_tiles", a.cuda(), b.cuda(), out, 512, N, K, K, N, i32(tiles), stream_ptr())
    for i, e in enumerate(tiles):
        got = out[i * 128:(i + 1) * 128].cpu().double()
        want = a[i * 128:(i + 1) * 128].double() @ b[e].double().t() if e >= 0 else torch.full((128, N), 7.0).double()
        assert (got - want).abs().max() < 2e-5 * K ** 0.5
