"""Serving benchmark of the Povipel decoder beside the framework's other hybrid decoders at equal width, layers and
active feed-forward parameters (random weights): ``python bench.py --workload povipel [--hybrid-size s|m|l]``.

Throughput and kernels as in ``hybrid_bench``; each kernel names the like kernel of the other decoders."""
from __future__ import annotations

import ctypes as C

from . import hybrid_bench as hb
from . import zepesun_bench as zb

#: windowed attention (heads of 128, kv heads), gated linear attention beside it and retention (heads of 64 key and 128
#: value channels), experts (number, of a token; their widths make up the other decoder's feed-forward); width, layers and
#: vocabulary are those of the other decoder's size
SIZES = {
    "s": dict(hq=8, hk=4, gla=4, ret=8, experts=32, top=4, window=1024, pool=16, streams=4),
    "m": dict(hq=16, hk=4, gla=8, ret=16, experts=32, top=4, window=1024, pool=16, streams=4),
    "l": dict(hq=32, hk=8, gla=16, ret=32, experts=16, top=4, window=1024, pool=16, streams=4),
}


def config(size: str, layers: int = 0):
    """Windowed attention beside gated linear attention, and retention, by turns; the first layer's feed-forward is dense."""
    from ..models.config import (AttentionSpec, GatedLinearSpec, GeluSpec, HybridConfig, HybridLayer, ParallelSpec, RetentionSpec,
                                 RotarySpec, RoutedSpec, SiluGluSpec)
    s, base = SIZES[size], hb.SIZES[size]
    attn = AttentionSpec(s["hq"], s["hk"], 128, 128, 128 ** -0.5, rot=RotarySpec(128, 10000.0, interleaved=True), window=s["window"],
                         pool=s["pool"], qk_norm="head", gate=None, sink=True, turn_values=True)
    both = ParallelSpec(attn, GatedLinearSpec(s["gla"], 64, 128, 16.0, 16), 0.5, 0.5, normed=True)
    ret = RetentionSpec(s["ret"], 64, 128, [1.0 - 2.0 ** (-5.0 - 6.0 * h / s["ret"]) for h in range(s["ret"])], RotarySpec(64, 10000.0))
    moe = RoutedSpec(SiluGluSpec(base["ff"] // s["top"]), s["experts"], s["top"], scores="sigmoid", weigh_input=True)
    mixers = [(both, ret)[i % 2] for i in range(layers or 2 * base["pairs"])]
    out = [HybridLayer(m, moe if i else GeluSpec(base["ff"] * 3 // 2)) for i, m in enumerate(mixers)]
    return HybridConfig(vocab=base["vocab"], width=base["width"], layers=out, eps=1e-6, design="Povipel", streams=s["streams"],
                        logit_softcap=30.0)


def kernels(eng, entries, phase, timer, peaks):
    from ..ops import _cuda
    from ..ops._cuda import stream_ptr
    from ..serve import hybrid_native as hn
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
        row(name, us, like, (rows * lin.k * 2 + lin.n * lin.k * 2 + rows * lin.n * (2, 4, 8, 2)[mode]) / 1e9, 2e-12 * rows * lin.n * lin.k)

    def result(name, a, lda, lin, which):           # a sublayer's result; small steps add it up in fp32
        if n <= 256:
            gemm(name, "output projections", a, lda, lin, P(getattr(sc, which + "32").data_ptr()), d, mode=2)
        else:
            gemm(name, "output projections", a, lda, lin, at(which), d)

    L = eng.layer_list
    first, both, ret = L[0], L[2 if len(L) > 2 else 0], L[1]
    side = next(m for m in eng.mixers if both.beside and C.addressof(m) == both.beside)
    S, few = eng.ccfg.streams, n <= 128
    lb, lr, ls = C.byref(both), C.byref(ret), C.byref(side)
    # between sublayers (behind a projection, two of them, experts); every stream is read and written
    stream = lambda *a: t("bb_hy_streams", cfg, *a, w, bb, 0, P(None))
    move = n * d * S * 8
    row("streams behind retention", stream(lr, 0, lr, 1), "norm", (move + n * d * 4) / 1e9)
    row("streams behind both mixers", stream(lb, 0, lb, 1), "norm", (move + n * d * 6) / 1e9)
    row("streams behind experts", stream(lr, 1, lb, 0), "norm", (move + n * d * 2 * (1 + ret.top)) / 1e9)
    sc.x.zero_()
    eng._run(sc, b)
    if b.n_pre:
        row("token shift", t("bb_hy_shift", cfg, lb, w, bb), "post (glu)", n * d * 4 / 1e9)
    gemm("both: input projections", "input projections", at("h"), d, both.inp, at("proj"), ld["proj"])
    gemm("retention: input projections", "input projections", at("h"), d, ret.inp, at("proj"), ld["proj"])
    result("attention: output projection", at("cat"), ld["cat"], both.out, "ya")
    result("gated linear: output projection", at("cat", side.off_cat), ld["cat"], side.out, "yb")
    result("retention: output projection", at("cat"), ld["cat"], ret.out, "ya")
    gemm("dense: up, gelu", "input projections", at("h"), d, first.up, at("cat"), ld["cat"], mode=3)
    result("dense: down", at("cat"), ld["cat"], first.down, "ya")
    eng._run(sc, b)
    # experts
    if not few:
        gemm("router (fp32)", "router", at("h"), d, ret.in32, P(sc.f32.data_ptr()), ld["f32"], mode=1)
    reset = lambda: sc.ex_count.zero_()
    reset()

    def route():
        rc = (lib.bb_hy_route_row if few else lib.bb_hy_route)(cfg, lr, w, n, stream_ptr())
        assert rc == 0
    us = timer(lambda: (reset(), route())) - timer(reset)
    row("router and routing (fp32)" if few else "experts: routing", max(us, 0.1), "routing",
        (n * (ret.n_experts * 4 + ret.top * 12) + ((ret.in32.n + n) * d * 2 if few else 0)) / 1e9)
    rows_ = sc.pair_row.clone()
    reset()
    route()
    rows_ = sc.pair_row.clone()

    def expert_rows():
        sc.pair_row.copy_(rows_)
        rc = lib.bb_hy_expert_rows(cfg, lr, w, n, stream_ptr())
        assert rc == 0
    us = timer(expert_rows) - timer(lambda: sc.pair_row.copy_(rows_))
    row("experts: weighed rows", max(us, 0.1), "experts: rows", n * d * 2 * (1 + ret.top) / 1e9)
    tiles = lib.bb_hy_moe_tiles(lr, n)
    used = int((sc.ex_tile[:tiles] >= 0).sum())
    live = int((sc.ex_count > 0).sum())
    pairs, sms = n * ret.top, eng.sm_count

    def width(N):
        full = tiles * -(-N // 256) >= sms and N >= 256
        return 256 if full else (128 if N >= 128 and tiles * -(-N // 128) >= sms // 2 else 64)
    for tag, wt, a, lda, y, ldy, N, K in (
            ("experts: gate and up", ret.w_egu, "ex_in", d, "ex_gu", ld["gu"], 2 * ret.effp, d),
            ("experts: down", ret.w_edown, "ex_act", ld["act"], "ex_out", d, d, ret.effp)):
        us = t("bb_gemm_bf16_grouped", at(a), P(wt), at(y), tiles * 128, N, K, lda, K, ldy, 0, 0, 1, P(sc.ex_tile.data_ptr()), N,
               ret.n_experts * N, P(None), 0, C.c_long(0), width(N))
        row(tag, us, tag, 2 * (pairs * (N + K) + live * N * K) / 1e9, 2e-12 * pairs * N * K)
    row("experts: gated product", t("bb_hy_expert_glu", cfg, lr, w, n), "experts: gated product", used * 128 * ret.effp * 6 / 1e9)
    eng._run(sc, b)
    # attention
    qkv = both.hq * both.dkp + both.hk * (both.dkp + both.dvp)
    row("attention: norms, rotation, pages", t("bb_hy_heads", cfg, lb, w, bb), "attention post", n * 2 * qkv * 2 / 1e9)
    x = hn.Pooled(both.pool, both.pool_rows, both.pkc, both.pvc, sc.work.pk, ld["pk"], sc.work.pk_rows, b.ctx_row0, both.sink, both.vcos_t,
                  both.vsin_t, both.dv)
    q, win, pool = at("proj", both.off_q), both.window, both.pool
    seen = lambda p: min(p + 1, win) + max(p + 1 - win, 0) // pool
    ext = (P(None), 0, 0, C.c_float(1.0), win, C.byref(x))
    if b.n_pre:
        row("attention: means of blocks", t("bb_hy_pool", cfg, lb, w, bb, 1), "latent page rows",
            sum(l * (1 + 2 / pool) for l in lens) * both.hk * (both.dkp + both.dvp) * 2 / 1e9)
        us = t("bb_flash_fwd_paged_p", q, ld["proj"], P(both.kc), P(both.vc), at("cat"), ld["cat"], P(b.tables), b.max_blocks,
               eng.block_size, eng.num_blocks + 1, P(b.seq_row0), P(b.seq_ctx), P(b.tile_seq), P(b.tile_qt), b.n_tiles, n,
               both.hq, both.hk, both.dkp, both.dvp, C.c_float(both.scale), C.c_float(0.0), *ext)
        keys = sum(seen(p) for l, c in zip(lens, ctxs) for p in range(c - l, c))
        row("attention: scores and values", us, "attention", tflop=2e-12 * keys * both.hq * (both.dk + both.dv))
    else:
        most = -(-(win + b.max_blocks * eng.block_size // pool) // 32)
        splits = max(1, min(16, -(-4 * eng.sm_count // (n * both.hk)), most))
        us = t("bb_paged_decode_p", q, ld["proj"], P(both.kc), P(both.vc), P(b.tables), b.max_blocks, P(b.seq_ctx), at("cat"),
               ld["cat"], P(sc.part_o.data_ptr()), P(sc.part_ml.data_ptr()), n, both.hq, both.hk, both.dkp, both.dvp,
               eng.block_size, splits, C.c_float(both.scale), C.c_float(0.0), *ext)
        row("attention: scores and values", us, "attention", sum(seen(c - 1) for c in ctxs) * both.hk * (both.dkp + both.dvp) * 2 / 1e9)
    # linear attention
    for tag, m, lm in (("gated linear", side, ls), ("retention", ret, lr)):
        state = len(entries) * m.heads * m.n * m.p * 8
        io = n * m.heads * (2 * m.np + 3 * m.pp) * 2
        if not b.n_pre:
            row(f"{tag}: state step, norm, gate", t("bb_hy_linear_decode", cfg, lm, w, bb), "recurrence", (io + state) / 1e9)
        elif m is side:
            gemm("gated linear: decays (fp32)", "router", at("proj", m.off_w1), ld["proj"], m.w2, P(sc.f32.data_ptr()), ld["f32"], mode=1)
            row("gated linear: chunks, norm, gate", t("bb_gla_chunk", cfg, lm, w, bb), "recurrence",
                (io + n * m.heads * m.np * 4 + state) / 1e9)
            row("gated linear: pairs left to the scan", t("bb_hy_linear_scan", cfg, lm, w, bb, 1), "recurrence",
                n / 128 * m.heads * 4 / 1e9)
            row("gated linear: scan, norm, gate (fallback)", t("bb_hy_linear_scan", cfg, lm, w, bb, 0), "recurrence",
                (io + n * m.heads * m.np * 4 + state) / 1e9)
        else:
            row("retention: rotation", t("bb_hy_turn", cfg, lm, w, bb), "attention post", n * m.heads * m.np * 8 / 1e9)
            row("retention: chunks", t("bb_retention_chunk", cfg, lm, w, bb), "recurrence",
                (n * m.heads * (2 * m.np + 2 * m.pp) * 2 + state) / 1e9)
            row("retention: norm, gate", t("bb_hy_linear_post", cfg, lm, w, n), "post (glu)", n * m.heads * m.pp * 6 / 1e9)
            row("retention: scan, norm, gate (fallback)", t("bb_hy_linear_scan", cfg, lm, w, bb, 0), "recurrence", (io + state) / 1e9)
    row("logits: bound", t("bb_hy_cap", cfg, w, b.n_want), "post (glu)", b.n_want * eng.vocabp * 8 / 1e9)
    del blob
    return out


def run(size: str = "m", steps: int = 10, with_kernels: bool = True, **kw) -> dict:
    base = hb.SIZES[size]
    shape = dict(SIZES[size], width=base["width"], ff=base["ff"], layers=2 * base["pairs"])
    return hb.compare(size, shape, (("povipel", config(size), kernels), ("pakalix", hb.hybrid_config(base), hb.hybrid_kernels),
                                    ("zepesun", zb.config(size), zb.kernels)), steps, with_kernels, **kw)


def steps(portion: int, seqs: int, ctx: int, n: int = 3, size: str = "s") -> None:
    """``n`` equal steps of a two-layer model: prompts of ``portion`` tokens, or one token each (``portion`` 1), at
    position ``ctx``.  A small program to put under a profiler."""
    hb.equal_steps(config(size, layers=2), portion, seqs, ctx, n)


if __name__ == "__main__":
    import argparse
    ap = argparse.ArgumentParser(description="equal steps of a two-layer Povipel decoder (for a profiler)")
    ap.add_argument("--portion", type=int, default=1024)
    ap.add_argument("--seqs", type=int, default=2)
    ap.add_argument("--ctx", type=int, default=0)
    ap.add_argument("--size", default="s", choices=sorted(SIZES))
    a = ap.parse_args()
    steps(a.portion, a.seqs, a.ctx, size=a.size)
