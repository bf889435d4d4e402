"""Serving benchmark of the Zepesun decoder beside the framework's other hybrid decoders at equal width, layers and
active feed-forward parameters (random weights): ``python bench.py --workload zepesun [--hybrid-size s|m|l]``.

Throughput and kernels as in ``hybrid_bench``; each kernel names the like kernel of the other decoders."""
from __future__ import annotations

import ctypes as C

from . import hybrid_bench as hb
from . import nezalorn_bench as nb

#: windowed attention (heads of 128, kv heads), matrix memories (heads, beside attention and alone; 64 key and 128
#: value channels), latent attention, experts (number, of a token; their width times that plus the shared one's is the
#: other decoder's feed-forward); width, layers and vocabulary are those of the other decoder's size
SIZES = {
    "s": dict(hq=8, hk=4, mside=4, malone=8, heads=16, dim=64, rot=32, vdim=64, kv_rank=256, experts=32, top=4, window=1024),
    "m": dict(hq=16, hk=4, mside=8, malone=16, heads=32, dim=64, rot=32, vdim=64, kv_rank=256, experts=32, top=4, window=1024),
    "l": dict(hq=32, hk=8, mside=16, malone=32, heads=32, dim=96, rot=32, vdim=128, kv_rank=512, experts=16, top=4, window=1024),
}


def config(size: str, layers: int = 0):
    """Cycles of four layers: attention and a matrix memory side by side, a memory, latent attention, a memory; the
    first layer's feed-forward is dense."""
    from ..models.config import (AttentionSpec, ClampedGluSpec, GeluGluSpec, HybridConfig, HybridLayer, LatentAttentionSpec,
                                 MlstmSpec, ParallelSpec, RotarySpec, RoutedSpec)
    s, base = SIZES[size], hb.SIZES[size]
    attn = AttentionSpec(s["hq"], s["hk"], 128, 128, 128 ** -0.5, window=s["window"], qk_norm=False, bias=True, gate="element")
    lat = LatentAttentionSpec(s["heads"], s["dim"], s["rot"], s["vdim"], s["kv_rank"], 0, (s["dim"] + s["rot"]) ** -0.5,
                              RotarySpec(s["rot"], 10000.0), q_latent=False, head_gate=True)
    alone = MlstmSpec(s["malone"], 64, 128, 15.0)
    cycle = [ParallelSpec(attn, MlstmSpec(s["mside"], 64, 128, 15.0), 0.7, 0.7), alone, lat, alone]
    shared = base["ff"] // 3
    moe = RoutedSpec(ClampedGluSpec((base["ff"] - shared) // s["top"], 7.0), s["experts"], s["top"], 8, 4, 2.5,
                     ClampedGluSpec(shared, 7.0))
    mixers = [cycle[i % 4] for i in range(layers or 2 * base["pairs"])]
    out = [HybridLayer(m, moe if i else GeluGluSpec(base["ff"])) for i, m in enumerate(mixers)]
    return HybridConfig(vocab=base["vocab"], width=base["width"], layers=out, eps=1e-6, design="Zepesun",
                        max_position_embeddings=8192)


def kernels(eng, entries, phase, timer, peaks):
    from ..ops import _cuda
    from ..ops._cuda import stream_ptr
    lib = _cuda.lib()
    sc, b, blob = eng._prepare(entries)
    cfg, w, bb = C.byref(eng.ccfg), C.byref(sc.work), C.byref(b)
    n, d, P = b.n, eng.dp, C.c_void_p
    ld = eng.ld
    lens = [len(e.tokens) for e in entries]
    ctxs = [e.start + len(e.tokens) for e in entries]
    out = []
    # a whole step: buffers hold what its kernels leave behind
    eng._run(sc, b)

    def t(fn, *args):
        f = getattr(lib, fn)
        f.restype = C.c_int

        def go():
            rc = f(*args, stream_ptr())
            if rc:
                raise RuntimeError(f"{fn} failed with code {rc}")
        return timer(go)

    def row(name, us, like, gbytes=None, tflop=None):
        hb._row(out, phase, name, us, gbytes, tflop, peaks, like)

    at = lambda buf, off=0: P(getattr(sc, buf).data_ptr() + 2 * off)

    def gemm(name, like, a, lda, lin, y, ldy, rows=n, mode=0):
        us = t("bb_gemm_bf16", a, P(lin.w), y, P(None), rows, lin.n, lin.k, lda, lin.k, ldy, 0, 0, mode, C.c_float(1.0), 0, 0)
        row(name, us, like, (rows * lin.k * 2 + lin.n * lin.k * 2 + rows * lin.n * (0, 4, 8)[mode]) / 1e9 +
            (rows * lin.n * 2 / 1e9 if mode == 0 else 0), 2e-12 * rows * lin.n * lin.k)

    def groups(name, like, a, lda, xs, wt, y, ldy, ys, G, N, K, rows=n):
        us = t("bb_gemm_bf16_groups", a, P(wt), y, rows, N, K, G, lda, xs, ldy, ys)
        row(name, us, like, 2 * (rows * G * (K + N) + G * N * K) / 1e9, 2e-12 * rows * G * N * K)

    L = eng.layer_list
    both, alone, lat = L[0] if len(L) < 5 else L[4], L[1], L[2]
    side = next(m for m in eng.mixers if both.beside and C.addressof(m) == both.beside)
    last = eng.layer_list.index(lat)
    # the start of a layer behind experts
    us = t("bb_hy_start", cfg, last, w, bb, 0, P(None))
    row("sum of experts, norm", us, "norm", n * d * (4 + 4 + 2 + 2 * alone.top) / 1e9)
    for tag, l in (("both", both), ("memory", alone), ("latent", lat)):
        gemm(f"{tag}: input projections", "input projections", at("h"), d, l.inp, at("proj"), ld["proj"])
    few = n <= 128
    if not few:
        gemm("router and gates (fp32)", "input projections", at("h"), d, alone.in32, P(sc.f32.data_ptr()), ld["f32"], mode=1)
    for tag, l in (("both", both), ("memory", alone), ("latent", lat)):
        gemm(f"{tag}: output projections + residual", "output projections", at("cat"), ld["cat"], l.out, P(sc.x.data_ptr()), d,
             mode=2)
    sc.x.zero_()
    eng._run(sc, b)
    # experts
    le = C.byref(alone)
    reset = lambda: sc.ex_count.zero_()
    reset()

    def route():
        rc = (lib.bb_hy_route_row if few else lib.bb_hy_route)(cfg, le, w, n, stream_ptr())
        assert rc == 0
    both_us = timer(lambda: (reset(), route()))
    extra = (alone.in32.n + n) * d * 2 if few else 0
    row("router and gates (fp32), routing" if few else "experts: routing", max(both_us - timer(reset), 0.1),
        "input projections" if few else "attention post", (n * (alone.n_experts * 4 + alone.top * 12) + extra) / 1e9)
    rows_ = sc.pair_row.clone()
    reset()
    route()

    def expert_rows():
        sc.pair_row.copy_(rows_)
        rc = lib.bb_hy_expert_rows(cfg, le, w, n, stream_ptr())
        assert rc == 0
    rows_ = sc.pair_row.clone()
    us = timer(expert_rows) - timer(lambda: sc.pair_row.copy_(rows_))
    row("experts: rows", max(us, 0.1), "attention post", n * d * 2 * (1 + alone.top) / 1e9)
    tiles = lib.bb_hy_moe_tiles(le, n)
    used = int((sc.ex_tile[:tiles] >= 0).sum())
    live = int((sc.ex_count > 0).sum())
    pairs = n * alone.top
    sms = eng.sm_count

    def width(N):
        full = tiles * -(-N // 256) >= sms and N >= 256
        return 256 if full else (128 if N >= 128 and tiles * -(-N // 128) >= sms // 2 else 64)
    for tag, like, wt, a, lda, y, ldy, N, K in (
            ("experts: gate and up", "input projections", alone.w_egu, "ex_in", d, "ex_gu", ld["gu"], 2 * alone.effp, d),
            ("experts: down", "output projections", alone.w_edown, "ex_act", ld["act"], "ex_out", d, d, alone.effp)):
        us = t("bb_gemm_bf16_grouped", at(a), P(wt), at(y), tiles * 128, N, K, lda, K, ldy, 0, 0, 1, P(sc.ex_tile.data_ptr()), N,
               alone.n_experts * N, P(None), 0, C.c_long(0), width(N))
        row(tag, us, like, 2 * (pairs * (N + K) + live * N * K) / 1e9, 2e-12 * pairs * N * K)
    us = t("bb_hy_expert_glu", cfg, le, w, n)
    row("experts: gated product", us, "post (glu)", used * 128 * alone.effp * 6 / 1e9)
    us = t("bb_hy_glu", cfg, le, w, n)
    row("shared expert: gated product", us, "post (glu)", n * alone.ff * 6 / 1e9)
    # attention
    la, q = C.byref(both), at("proj", both.off_q)
    gate = at("proj", both.off_g)
    qkv = both.hq * both.dkp + both.hk * (both.dkp + both.dvp)
    us = t("bb_hy_kv_post", cfg, la, w, bb)
    row("attention: biases, pages, glu", us, "attention post", n * (2 * qkv + 3 * both.ff) * 2 / 1e9)
    win = both.window
    ext = (gate, ld["proj"], 1, C.c_float(both.out_scale), win)
    if b.n_pre:
        us = t("bb_flash_fwd_paged_x", q, ld["proj"], P(both.kc), P(both.vc), at("cat"), ld["cat"], P(b.tables), b.max_blocks,
               eng.block_size, eng.num_blocks + 1, P(b.seq_row0), P(b.seq_ctx), P(b.tile_seq), P(b.tile_qt), b.n_tiles, n,
               both.hq, both.hk, both.dkp, both.dvp, C.c_float(both.scale), C.c_float(0.0), *ext)
        keys = sum(min(p + 1, win) for l, c in zip(lens, ctxs) for p in range(c - l, c))
        row("attention: scores and values", us, "attention", tflop=2e-12 * keys * both.hq * (both.dk + both.dv))
    else:
        splits = max(1, min(16, -(-4 * eng.sm_count // (n * both.hk)), -(-win // 32)))
        us = t("bb_paged_decode_x", q, ld["proj"], P(both.kc), P(both.vc), P(b.tables), b.max_blocks, P(b.seq_ctx), at("cat"),
               ld["cat"], P(sc.part_o.data_ptr()), P(sc.part_ml.data_ptr()), n, both.hq, both.hk, both.dkp, both.dvp,
               eng.block_size, splits, C.c_float(both.scale), C.c_float(0.0), *ext)
        row("attention: scores and values", us, "attention", sum(min(c, win) for c in ctxs) * both.hk * (both.dkp + both.dvp) * 2 / 1e9)
    # matrix memories
    for tag, m in (("memory beside attention", side), ("memory", alone)):
        lm = C.byref(m)
        state = len(entries) * m.heads * m.mem * 8
        if b.n_pre:
            if m is alone:
                us = t("bb_hy_mlstm_gates", cfg, lm, w, n)
                row("memory: gates", us, "attention post", n * m.heads * 16 / 1e9)
                sc.f32.zero_()
            us = t("bb_mlstm_chunk", cfg, lm, w, bb)
            fl = 2.0 * n * m.heads * (64 * (m.n + m.p) + 2 * m.n * m.p)
            row(f"{tag}: chunks, norm, gate", us, "recurrence", (n * m.heads * (2 * m.np + 3 * m.pp) * 2 + n * m.heads * 8 + state) / 1e9,
                1e-12 * fl)
        else:
            us = t("bb_hy_mlstm_decode", cfg, lm, w, bb)
            row(f"{tag}: state step, norm, gate", us, "recurrence", (n * m.heads * (2 * m.np + 3 * m.pp) * 2 + state) / 1e9)
    # latent attention
    ll, width_, dq = C.byref(lat), lat.kvrp + lat.rotp, lat.dkp + lat.rotp
    us = t("bb_hy_latent_in", cfg, ll, w, bb)
    row("latent: norm, rotation, pages", us, "latent norms and pages", n * 2 * width_ * 2 / 1e9)
    us = t("bb_hy_latent_q", cfg, ll, w, bb, b.n_pre)
    row("latent: query rotation", us, "latent query rotation", n * lat.hq * lat.rotp * 4 / 1e9)
    ql = at("proj", lat.off_q)
    if b.n_pre:
        us = t("bb_hy_latent_gather", cfg, ll, w, bb)
        row("latent: page rows", us, "latent page rows", b.n_exp * width_ * 4 / 1e9)
        gemm("latent: keys and values", "keys and values", at("ckv"), ld["ckv"], lat.expand, at("kvx"), ld["kvx"], rows=b.n_exp)
        us = t("bb_flash_fwd_window", ql, ld["proj"], at("kvx"), at("kvx", lat.hq * dq), ld["kvx"], b.n_exp, at("cat"), ld["cat"],
               P(b.seq_row0), P(b.kv_row0), P(b.kv_pos0), P(b.seq_ctx), P(b.tile_seq), P(b.tile_qt), b.n_tiles, n, lat.hq, lat.hq,
               dq, lat.dvp, C.c_float(lat.scale), lat.window, at("proj", lat.off_g), ld["proj"])
        keys = sum(p + 1 for l, c in zip(lens, ctxs) for p in range(c - l, c))
        row("latent: scores and values", us, "attention", tflop=2e-12 * keys * lat.hq * (lat.dk + lat.rot + lat.dv))
    else:
        groups("latent: queries into latents", "input projections", ql, ld["proj"], dq, lat.w_abs, at("qa"), ld["qa"], width_,
               lat.hq, lat.kvrp, lat.dkp)
        us = t("bb_hy_latent_decode", cfg, ll, w, bb, 0)
        row("latent: scores and values", us, "attention", (sum(ctxs) * width_ * 2 + n * lat.hq * (width_ + lat.kvrp) * 2) / 1e9,
            2e-12 * sum(ctxs) * lat.hq * (width_ + lat.kvrp))
        groups("latent: values out of latents", "input projections", at("ol"), ld["ol"], lat.kvrp, lat.w_uv, at("cat"), ld["cat"],
               lat.dvp, lat.hq, lat.dvp, lat.kvrp)
    del blob
    return out


def run(size: str = "m", steps: int = 10, with_kernels: bool = True, **kw) -> dict:
    base = hb.SIZES[size]
    shape = dict(SIZES[size], width=base["width"], ff=base["ff"], layers=2 * base["pairs"])
    return hb.compare(size, shape, (("zepesun", config(size), kernels), ("pakalix", hb.hybrid_config(base), hb.hybrid_kernels),
                                    ("nezalorn", nb.config(size), nb.kernels)), steps, with_kernels, **kw)


def steps(portion: int, seqs: int, ctx: int, n: int = 3, size: str = "s") -> None:
    """``n`` equal steps of a four-layer model: prompts of ``portion`` tokens, or one token each (``portion`` 1), at
    position ``ctx``.  A small program to put under a profiler."""
    hb.equal_steps(config(size, layers=4), portion, seqs, ctx, n)


if __name__ == "__main__":
    import argparse
    ap = argparse.ArgumentParser(description="equal steps of a four-layer Zepesun decoder (for a profiler)")
    ap.add_argument("--portion", type=int, default=1024)
    ap.add_argument("--seqs", type=int, default=2)
    ap.add_argument("--ctx", type=int, default=0)
    ap.add_argument("--size", default="s", choices=sorted(SIZES))
    a = ap.parse_args()
    steps(a.portion, a.seqs, a.ctx, size=a.size)
