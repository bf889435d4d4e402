"""Serving benchmark of the Nezalorn decoder beside the framework's other hybrid decoder at equal width, layers
and feed-forward parameters (random weights): ``python bench.py --workload nezalorn [--hybrid-size s|m|l]``.

Throughput and kernels as in ``hybrid_bench``; each kernel names the other decoder's like kernel."""
from __future__ import annotations

import ctypes as C

from . import hybrid_bench as hb

#: latent attention (heads, unrotated / rotated / value sizes, latent ranks), delta-rule heads of 64, gate blocks;
#: width, layers and vocabulary are those of the other decoder's size
SIZES = {
    "s": dict(heads=16, dim=64, rot=32, vdim=64, kv_rank=256, q_rank=512, delta=16, blocks=8, window=1024),
    "m": dict(heads=32, dim=64, rot=32, vdim=64, kv_rank=256, q_rank=768, delta=32, blocks=8, window=1024),
    "l": dict(heads=32, dim=96, rot=32, vdim=128, kv_rank=512, q_rank=1536, delta=64, blocks=16, window=1024),
}


def config(size: str, layers: int = 0):
    """Cycles of four layers: latent attention, linear recurrence, delta rule, latent attention on the first
    one's latents."""
    from ..models.config import (GeneralDeltaSpec, HybridConfig, HybridLayer, LatentAttentionSpec, PolyNormSpec, RgLruSpec,
                                 RotarySpec, YarnSpec)
    s, base = SIZES[size], hb.SIZES[size]
    d = base["width"]
    rot = RotarySpec(s["rot"], 10000.0, YarnSpec(4.0, 4096.0, 32.0, 1.0), True)
    mlp = PolyNormSpec(base["ff"] * 3 // 2)       # two matrices with the parameters of the gated form's three

    def latent(kv_from):
        return LatentAttentionSpec(s["heads"], s["dim"], s["rot"], s["vdim"], s["kv_rank"], s["q_rank"],
                                   (s["dim"] + s["rot"]) ** -0.5, rot, s["window"], kv_from)
    out = []
    while len(out) < (layers or 2 * base["pairs"]):
        first = len(out)
        out += [latent(None), RgLruSpec(d, s["blocks"], 4), GeneralDeltaSpec(s["delta"], 64, 64), latent(first)]
    return HybridConfig(vocab=base["vocab"], width=d, layers=[HybridLayer(m, mlp) for m in out], eps=1e-6, design="Nezalorn")


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
        row(name, us, like, (rows * lin.k * 2 + lin.n * lin.k * 2 + rows * lin.n * (8 if mode else 2)) / 1e9,
            2e-12 * rows * lin.n * lin.k)

    def groups(name, like, a, lda, xs, wt, y, ldy, ys, G, N, K, rows=n):
        us = t("bb_gemm_bf16_groups", a, P(wt), y, rows, N, K, G, lda, xs, ldy, ys)
        row(name, us, like, 2 * (rows * G * (K + N) + G * N * K) / 1e9, 2e-12 * rows * G * N * K)

    layers = {l.kind: (i, l) for i, l in reversed(list(enumerate(eng.layer_list)))}
    (_, a), (di, dl), (_, r) = layers[2], layers[3], layers[4]
    us = t("bb_hy_mix_norm", cfg, di, w, bb, P(None))
    row(f"sum of {di + 1} results, two norms", us, "norm", n * d * (4 * (di + 1) + 4 + 4) / 1e9)
    for tag, l in (("latent", a), ("lru", r), ("delta", dl)):
        gemm(f"{tag}: input projections", "input projections", at("h"), d, l.inp, at("proj"), ld["proj"])
    gemm("feed-forward: up", "input projections", at("h2"), d, a.up, at("proj", a.off_up), ld["proj"])
    us = t("bb_hy_polynorm", cfg, C.byref(a), w, n)
    row("feed-forward: polynomial of norms", us, "post (glu)", n * a.ff * 4 / 1e9)
    for tag, l in (("latent", a), ("lru", r), ("delta", dl)):
        gemm(f"{tag}: output projections + residual", "output projections", at("cat"), ld["cat"], l.out,
             P(sc.x.data_ptr()), d, mode=2)
    sc.x.zero_()
    # latent attention
    la, width, dq = C.byref(a), a.kvrp + a.rotp, a.dkp + a.rotp
    us = t("bb_hy_latent_in", cfg, la, w, bb)
    row("latent: norms, rotation, pages", us, "attention post", n * (2 * a.qrp + 2 * width) * 2 / 1e9)
    gemm("latent: queries", "input projections", at("proj", a.off_dq), ld["proj"], a.uq, at("q"), ld["q"])
    n_in = b.n_pre
    us = t("bb_hy_latent_q", cfg, la, w, bb, n_in)
    row("latent: query rotation", us, "attention post", n * a.hq * a.rotp * 4 / 1e9)
    win = a.window
    if b.n_pre:
        us = t("bb_hy_latent_gather", cfg, la, w, bb)
        row("latent: page rows", us, "attention post", b.n_exp * width * 4 / 1e9)
        gemm("latent: keys and values", "input projections", at("ckv"), ld["ckv"], a.expand, at("kvx"), ld["kvx"], rows=b.n_exp)
        us = t("bb_flash_fwd_window", at("q"), ld["q"], at("kvx"), at("kvx", a.hq * dq), ld["kvx"], b.n_exp, at("cat"), ld["cat"],
               P(b.seq_row0), P(b.kv_row0), P(b.kv_pos0), P(b.seq_ctx), P(b.tile_seq), P(b.tile_qt), b.n_tiles, n, a.hq, a.hq,
               dq, a.dvp, C.c_float(a.scale), win, P(None), 0)
        pairs = sum(min(p + 1, win) for l, c in zip(lens, ctxs) for p in range(c - l, c))
        row("latent: scores and values", us, "attention", tflop=2e-12 * pairs * a.hq * (a.dk + a.rot + a.dv))
    else:
        groups("latent: queries into latents", "input projections", at("q"), ld["q"], dq, a.w_abs, at("qa"), ld["qa"], width,
               a.hq, a.kvrp, a.dkp)
        us = t("bb_hy_latent_decode", cfg, la, w, bb, 0)
        keys = sum(min(c, win) for c in ctxs)
        row("latent: scores and values", us, "attention", (keys * width * 2 + n * a.hq * (width + a.kvrp) * 2) / 1e9,
            2e-12 * keys * a.hq * (width + a.kvrp))
        groups("latent: values out of latents", "input projections", at("ol"), ld["ol"], a.kvrp, a.w_uv, at("cat"), ld["cat"],
               a.dvp, a.hq, a.dvp, a.kvrp)
    # linear recurrence
    lr = C.byref(r)
    us = t("bb_hy_conv_linear", cfg, lr, w, bb)
    row("lru: convolution", us, "convolution", n * r.chp * 4 / 1e9)
    groups("lru: gates", "input projections", at("xbc"), ld["xbc"], r.bwp, r.w_gate, at("aux"), ld["aux"], 2 * r.bwp, r.blocks,
           2 * r.bwp, r.bwp)
    us = t("bb_hy_rglru", cfg, lr, w, bb)
    row("lru: recurrence", us, "recurrence", (n * r.chp * 10 + len(entries) * r.chp * 8) / 1e9)
    # delta rule
    ldl = C.byref(dl)
    us = t("bb_hy_delta_tanh", cfg, ldl, w, bb)
    row("delta: tanh", us, "attention post", n * dl.wrp * 4 / 1e9)
    gemm("delta: decays", "input projections", at("proj", dl.off_w1), ld["proj"], dl.w2, at("aux"), ld["aux"])
    us = t("bb_hy_delta", cfg, ldl, w, bb)
    state = len(entries) * dl.heads * dl.p * dl.p * 8
    row("delta: recurrence, norm, gate", us, "recurrence", (n * dl.innerp * (12 if b.n_pre else 14) + state) / 1e9)
    if b.n_pre:
        us = t("bb_hy_delta_scan", cfg, ldl, w, bb, 0)
        row("delta: recurrence alone", us, "recurrence", (n * dl.innerp * 12 + state) / 1e9)
    del blob
    return out


def run(size: str = "m", steps: int = 10, with_kernels: bool = True, **kw) -> dict:
    base = hb.SIZES[size]
    shape = dict(SIZES[size], width=base["width"], ff=base["ff"] * 3 // 2, layers=2 * base["pairs"])
    return hb.compare(size, shape, (("nezalorn", config(size), kernels), ("pakalix", hb.hybrid_config(base), hb.hybrid_kernels)),
                      steps, with_kernels, **kw)


def steps(portion: int, seqs: int, ctx: int, n: int = 3, size: str = "m") -> None:
    """``n`` equal steps of a four-layer model: prompts of ``portion`` tokens, or one token each (``portion`` 1), at
    position ``ctx``.  A small program to put under a profiler."""
    hb.equal_steps(config(size, layers=4), portion, seqs, ctx, n)


if __name__ == "__main__":
    import argparse
    ap = argparse.ArgumentParser(description="equal steps of a four-layer Nezalorn decoder (for a profiler)")
    ap.add_argument("--portion", type=int, default=1024)
    ap.add_argument("--seqs", type=int, default=2)
    ap.add_argument("--ctx", type=int, default=0)
    a = ap.parse_args()
    steps(a.portion, a.seqs, a.ctx)
