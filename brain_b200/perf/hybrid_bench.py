"""Serving benchmark of the hybrid decoder beside the dense decoder of equal size (random weights):
``python bench.py --workload hybrid [--hybrid-size s|m|l]``.

Throughput: prefill (a packed step of several prompts) and decode (a replayed graph of greedy steps) through
the engines' own calls.  Kernels: device time of every kernel of a layer, each launch behind a buffer write
larger than L2, as the difference of two replayed graphs (write + kernel, write alone), with the share of
the measured copy bandwidth or tensor throughput it reaches, beside the dense decoder's like kernel."""
from __future__ import annotations

import ctypes as C
import json
import os
import statistics

import numpy as np
import torch

#: width, attention (heads, kv heads), state-space heads (64 wide, state 128), feed-forward, layers of each kind
SIZES = {
    "s": dict(width=1024, hq=16, hk=8, mh=32, ff=3072, pairs=4, vocab=32768),
    "m": dict(width=2048, hq=16, hk=4, mh=64, ff=6144, pairs=4, vocab=32768),
    "l": dict(width=4096, hq=32, hk=8, mh=128, ff=12288, pairs=2, vocab=32768),
}
HEAD = 128


def hybrid_config(s):
    from ..models.config import AttentionSpec, ClampedGluSpec, HybridConfig, HybridLayer, Mamba2Spec, RotarySpec
    attn = AttentionSpec(s["hq"], s["hk"], HEAD, HEAD, HEAD ** -0.5, 50.0, RotarySpec(HEAD, 10000.0), True)
    mamba = Mamba2Spec(s["mh"], 64, 128, 1, 4, 1)
    mlp = ClampedGluSpec(s["ff"], 7.0)
    return HybridConfig(vocab=s["vocab"], width=s["width"], layers=[HybridLayer(mamba, mlp), HybridLayer(attn, mlp)] * s["pairs"],
                        eps=1e-6, residual_mult=1.0)


def dense_config(s):
    from ..models.config import QwenConfig
    return QwenConfig(vocab=s["vocab"], block_size=8192, n_layers=2 * s["pairs"], d_model=s["width"], n_heads=s["hq"],
                      n_kv_heads=s["hk"], head_dim=HEAD, d_ff=s["ff"], tie_embeddings=False)


class KernelTimer:
    """Device microseconds of a launch behind a buffer write larger than L2: replays of (write + kernel) and of the
    write alone take turns, so both see the same clocks, and the difference counts."""

    def __init__(self, reps: int = 8, rounds: int = 7):
        self.buf = torch.empty(192 << 20, device="cuda", dtype=torch.uint8)
        self.reps, self.rounds = reps, rounds
        self.base = self._graph(lambda: None)

    def _graph(self, fn):
        fn()
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, capture_error_mode="thread_local"):
            for _ in range(self.reps):
                self.buf.zero_()
                fn()
        return g

    def __call__(self, fn) -> float:
        g = self._graph(fn)
        us = []
        for i in range(self.rounds + 2):
            ev = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
            torch.cuda.synchronize()
            ev[0].record()
            self.base.replay()
            ev[1].record()
            g.replay()
            ev[2].record()
            torch.cuda.synchronize()
            if i >= 2:
                us.append((ev[1].elapsed_time(ev[2]) - ev[0].elapsed_time(ev[1])) / self.reps * 1e3)
        return max(statistics.median(us), 0.1)


def _time_calls(fn, n: int) -> float:
    """Device seconds of ``n`` calls after three warm-up calls (their working set exceeds L2)."""
    for _ in range(3):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(n):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / 1e3


def throughput(eng, n_seq: int, T: int, B: int, ctx: int, steps: int, vocab: int):
    """(prefill tokens/s, decode tokens/s) of an engine through the calls its scheduler makes."""
    rng = np.random.default_rng(0)
    per = -(-T // eng.block_size)
    has = eng.state_slots > 0
    items = []
    for i in range(n_seq):
        bt = np.full(eng.max_blocks, -1, dtype=np.int32)
        bt[:per] = np.arange(i * per, (i + 1) * per)
        it = (rng.integers(0, vocab, T).astype(np.int32), 0, bt, True, True)
        items.append(it + ((i,) if has else ()))
    sec = _time_calls(lambda: eng.prefill_batch(items), steps) / steps
    pre = n_seq * T / sec
    win = 8
    per = -(-(ctx + win) // eng.block_size)
    bts = np.full((B, eng.max_blocks), -1, dtype=np.int32)
    for i in range(B):
        bts[i, :per] = np.arange(i * per, (i + 1) * per)
    tok = rng.integers(0, vocab, B).astype(np.int32)
    pos = np.full(B, ctx, dtype=np.int32)
    kw = {"slots": np.arange(B, dtype=np.int32)} if has else {}
    sec = _time_calls(lambda: eng.decode(tok, pos, bts, window=win, greedy=True, **kw), steps) / (steps * win)
    return pre, B / sec


def _row(out, phase, name, us, gbytes=None, tflop=None, peaks=None, like=None):
    """One kernel: the larger of its two roofline shares."""
    shares = {}
    if gbytes:
        shares["copy"] = gbytes / (us * 1e-6) / peaks["hbm_gbs"]
    if tflop:
        shares["gemm"] = tflop / (us * 1e-6) / peaks["bf16_tflops"]
    kind = max(shares, key=shares.get)
    out.append({"phase": phase, "kernel": name, "us": round(us, 2), "bound": kind, "of_measured": round(shares[kind], 3),
                "like": like})


def hybrid_kernels(eng, entries, phase, timer, peaks):
    from ..ops import _cuda
    from ..ops._cuda import stream_ptr
    lib = _cuda.lib()
    sc, b, blob = eng._prepare(entries)
    cfg, w = C.byref(eng.ccfg), C.byref(sc.work)
    n, d, P = b.n, eng.dp, C.c_void_p
    ctxs = [e.start + len(e.tokens) for e in entries]
    lens = [len(e.tokens) for e in entries]
    out = []

    def t(fn, *args):
        f = getattr(lib, fn)
        f.restype = C.c_int

        def go():
            rc = f(*args, stream_ptr())
            if rc:
                raise RuntimeError(f"{fn} failed with code {rc}")
        return timer(go)
    m = next(l for l in eng.layer_list if l.kind == 1)
    a = next(l for l in eng.layer_list if l.kind == 0)
    x, h, proj, cat = (P(getattr(sc, k).data_ptr()) for k in ("x", "h", "proj", "cat"))
    us = t("bb_hy_norm", C.c_int(0), x, P(None), P(a.norm), h, n, d, d, C.c_float(eng.cfg.eps))
    _row(out, phase, "norm", us, n * d * 6 / 1e9, peaks=peaks, like="norm")
    for tag, l in (("mamba2", m), ("attention", a)):
        us = t("bb_gemm_bf16", h, P(l.inp.w), proj, P(None), n, l.inp.n, d, d, d, eng.ld["proj"], 0, 0, 0, C.c_float(1.0), 0, 0)
        _row(out, phase, f"{tag}: input projections", us, (n * d + l.inp.n * d + n * l.inp.n) * 2 / 1e9,
             2e-12 * n * l.inp.n * d, peaks, "gemm in")
        us = t("bb_gemm_bf16", cat, P(l.out.w), x, P(None), n, d, l.out.k, eng.ld["cat"], l.out.k, d, 0, 0, 2, C.c_float(1.0),
               0, 0)
        _row(out, phase, f"{tag}: output projections + residual", us,
             (n * l.out.k * 2 + l.out.k * d * 2 + n * d * 8) / 1e9, 2e-12 * n * l.out.k * d, peaks, "gemm out")
    sc.x.zero_()
    la, lm, bb = C.byref(a), C.byref(m), C.byref(b)
    qkv = (a.hq + a.hk) * a.dkp + a.hk * a.dvp
    us = t("bb_hy_attn_post", cfg, la, w, bb)
    _row(out, phase, "attention: norms, rotation, pages, glu", us, n * (2 * qkv + 3 * a.ff) * 2 / 1e9, peaks=peaks, like="rows")
    q = P(sc.proj.data_ptr() + 2 * a.off_q)
    gate = P(sc.proj.data_ptr() + 2 * a.off_g)
    if b.n_pre:
        us = t("bb_flash_fwd_paged_x", q, eng.ld["proj"], P(a.kc), P(a.vc), cat, eng.ld["cat"], P(b.tables), b.max_blocks,
               eng.block_size, eng.num_blocks + 1, P(b.seq_row0), P(b.seq_ctx), P(b.tile_seq), P(b.tile_qt), b.n_tiles, n,
               a.hq, a.hk, a.dkp, a.dvp, C.c_float(a.scale), C.c_float(a.softcap), gate, eng.ld["proj"], 0, C.c_float(1.0), 0)
        pairs = sum(l * (c - l) + l * (l + 1) / 2 for l, c in zip(lens, ctxs))
        _row(out, phase, "attention: scores and values", us, tflop=2e-12 * pairs * a.hq * (a.dk + a.dv), peaks=peaks,
             like="attention")
        us = t("bb_hy_conv", cfg, lm, w, bb)
        _row(out, phase, "mamba2: convolution", us, n * (2 * m.ch * 2 + m.heads * 6) / 1e9, peaks=peaks, like="rows")
        us = t("bb_ssd_chunk", cfg, lm, w, bb)
        fl = 2.0 * n * m.heads * (64 * m.n / (m.heads // m.groups) + 64 * m.p + 2 * m.n * m.p)
        _row(out, phase, "mamba2: recurrence in chunks", us,
             (n * (m.ch + m.inner) * 2 + n * m.heads * 4 + len(entries) * m.heads * m.n * m.p * 8) / 1e9, 1e-12 * fl, peaks,
             "attention")
    else:
        splits = C.c_int(max(1, min(16, -(-4 * 148 // (n * a.hk)))))
        us = t("bb_paged_decode_x", q, eng.ld["proj"], P(a.kc), P(a.vc), P(b.tables), b.max_blocks, P(b.seq_ctx), cat,
               eng.ld["cat"], P(sc.part_o.data_ptr()), P(sc.part_ml.data_ptr()), n, a.hq, a.hk, a.dkp, a.dvp, eng.block_size,
               splits, C.c_float(a.scale), C.c_float(a.softcap), gate, eng.ld["proj"], 0, C.c_float(1.0), 0)
        _row(out, phase, "attention: scores and values", us, sum(ctxs) * a.hk * (a.dkp + a.dvp) * 2 / 1e9, peaks=peaks,
             like="attention")
        us = t("bb_hy_ssm_decode", cfg, lm, w, bb)
        _row(out, phase, "mamba2: convolution and state step", us, n * (m.heads * m.n * m.p * 8 + m.ch * 8) / 1e9,
             peaks=peaks, like="attention")
    us = t("bb_hy_mamba_post", cfg, lm, w, bb)
    _row(out, phase, "mamba2: gate, norm, glu", us, n * (3 * m.inner + 3 * m.ff) * 2 / 1e9, peaks=peaks, like="rows")
    del blob
    return out


def dense_kernels(eng, n_seq, T, ctx, phase, timer, peaks):
    """The dense decoder's kernels at equal rows: prompts of T tokens, or one row at context ``ctx`` each."""
    from ..ops import _cuda
    from ..ops._cuda import L as clong, stream_ptr
    lib = _cuda.lib()
    n = n_seq * T
    d, hq, hk, hd, ff = eng.cfg.d_model, eng.hq, eng.hk, eng.hd, eng.cfg.d_ff
    dev = eng.device
    z = lambda *s: torch.randn(*s, device=dev).to(torch.bfloat16)
    x, r, h, qkv, qk, o = z(n, d), z(n, d), z(n, d), z(n, (hq + 2 * hk) * hd), z(n, (hq + hk) * hd), z(n, hq * hd)
    gu, act = z(n, 2 * ff), z(n, ff)
    l = eng.layers[0]
    rstd = torch.empty(n * (hq + hk), device=dev)
    out = []
    P = lambda t: C.c_void_p(t.data_ptr())

    def t(fn, *args):
        f = getattr(lib, fn)
        f.restype = C.c_int

        def go():
            rc = f(*args, stream_ptr())
            if rc:
                raise RuntimeError(f"{fn} failed with code {rc}")
        return timer(go)
    f1 = C.c_float
    us = t("bb_rmsnorm_fwd", P(x), P(r), P(l["ln1"]), P(h), P(o if hq * hd >= d else r), P(rstd), n, d, f1(1e-6))
    _row(out, phase, "norm", us, n * d * 8 / 1e9, peaks=peaks)
    for name, lin, a, c in (("gemm in", l["qkv"], h, qkv), ("gemm in (gate/up)", l["gate_up"], h, gu),
                            ("gemm out", l["wo"], o, x), ("gemm out (down)", l["down"], act, x)):
        N, K = lin.w.shape
        us = t("bb_gemm_bf16", P(a), P(lin.w), P(c), C.c_void_p(None), n, N, K, K, K, N, 0, 0, 0, f1(1.0), 0, 0)
        _row(out, phase, name, us, (n * K + N * K + n * N) * 2 / 1e9, 2e-12 * n * N * K, peaks)
    pos = torch.arange(n, device=dev, dtype=torch.int32) % T + (0 if T > 1 else ctx)
    us = t("bb_qknorm_rope_fwd", P(qkv), qkv.shape[1], P(l["q_norm"]), P(l["k_norm"]), P(eng.cos), P(eng.sin), P(pos), P(qk),
           qk.shape[1], P(rstd), n, hq, hk, hd, f1(1e-6))
    _row(out, phase, "rows: q/k norm and rotation", us, n * (hq + hk) * hd * 4 / 1e9, peaks=peaks)
    us = t("bb_swiglu_fwd", P(gu), P(act), clong(n), ff)
    _row(out, phase, "rows: swiglu", us, n * ff * 6 / 1e9, peaks=peaks)
    per = -(-(T if T > 1 else ctx + 1) // eng.block_size)
    bts = torch.full((n_seq, eng.max_blocks), 0, dtype=torch.int32)
    for i in range(n_seq):
        bts[i, :per] = torch.arange(i * per, (i + 1) * per)
    bts = bts.to(dev)
    if T > 1:
        meta = eng._paged_prefill_meta([(i * T, T, 0, bts[i]) for i in range(n_seq)], n)
        us = timer(lambda: eng._paged_prefill_attention(0, qk[:, :hq * hd], o, meta))
        _row(out, phase, "attention", us, tflop=2e-12 * n_seq * T * (T + 1) / 2 * hq * 2 * hd, peaks=peaks)
    else:
        lens = torch.full((n,), ctx + 1, dtype=torch.int32, device=dev)
        us = timer(lambda: eng._paged_attention(0, qk[:, :hq * hd], bts, lens, out=o))
        _row(out, phase, "attention", us, n * (ctx + 1) * hk * hd * 4 / 1e9, peaks=peaks)
    return out


def run(size: str = "m", steps: int = 10, kernels: bool = True, n_seq: int = 4, T: int = 2048, B: int = 64,
        ctx: int = 2048) -> dict:
    from ..models.hybrid import HybridDecoder
    from ..models.qwen3 import Qwen3
    from ..ops import _cuda
    from ..serve.engine import make_engine
    from ..serve.hybrid import Entry
    s = SIZES[size]
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        peaks = json.load(open(os.path.join(root, "MEASURED_PEAKS.json")))
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    blocks = max(n_seq * -(-T // 16), B * -(-(ctx + 16) // 16))
    res = {"size": size, "shape": s, "prefill_tokens_per_s": {}, "decode_tokens_per_s": {}, "kernels": {}}
    timer = KernelTimer() if kernels else None
    rng = np.random.default_rng(1)
    launches0 = _cuda.launch_count
    for name in ("hybrid", "dense"):
        torch.manual_seed(0)
        if name == "hybrid":
            model = HybridDecoder(hybrid_config(s)).init_weights(0).to("cuda", torch.bfloat16)
            kw = dict(max_batch=B)
        else:
            model = Qwen3(dense_config(s)).to("cuda", torch.bfloat16)
            model.init_weights(0)
            kw = {}
        eng = make_engine(model, block_size=16, num_blocks=blocks, max_seq_len=-(-(max(T, ctx) + 16) // 16) * 16,
                          max_prefill=T, **kw)
        del model
        pre, dec = throughput(eng, n_seq, T, B, ctx, steps, s["vocab"])
        res["prefill_tokens_per_s"][name], res["decode_tokens_per_s"][name] = round(pre), round(dec)
        if kernels:
            if name == "hybrid":
                per = -(-T // 16)
                ent = [Entry(rng.integers(0, s["vocab"], T), 0, np.arange(i * per, (i + 1) * per), i, [T - 1])
                       for i in range(n_seq)]
                rows = hybrid_kernels(eng, ent, "prefill", timer, peaks)
                per = -(-(ctx + 1) // 16)
                ent = [Entry(rng.integers(0, s["vocab"], 1), ctx, np.arange(i * per, (i + 1) * per), i, [0]) for i in range(B)]
                rows += hybrid_kernels(eng, ent, "decode", timer, peaks)
            else:
                rows = dense_kernels(eng, n_seq, T, 0, "prefill", timer, peaks)
                rows += dense_kernels(eng, B, 1, ctx, "decode", timer, peaks)
            res["kernels"][name] = rows
        _cuda.check_error()
        del eng
        torch.cuda.empty_cache()
    res["gpu_launches"] = _cuda.launch_count - launches0
    return res


def compare(size: str, shape: dict, designs, steps: int = 10, with_kernels: bool = True, n_seq: int = 4, T: int = 2048,
            B: int = 64, ctx: int = 2048) -> dict:
    """Throughput and kernel tables of hybrid decoders of equal size; ``designs``: (name, configuration, kernel table)."""
    from ..models.hybrid import HybridDecoder
    from ..ops import _cuda
    from ..serve.engine import make_engine
    from ..serve.hybrid import Entry
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        peaks = json.load(open(os.path.join(root, "MEASURED_PEAKS.json")))
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    vocab = SIZES[size]["vocab"]
    blocks = max(n_seq * -(-T // 16), B * -(-(ctx + 16) // 16))
    res = {"size": size, "shape": shape, "prefill_tokens_per_s": {}, "decode_tokens_per_s": {}, "kernels": {}}
    timer = KernelTimer() if with_kernels else None
    rng = np.random.default_rng(1)
    launches0 = _cuda.launch_count
    for name, cfg, table in designs:
        with torch.device("cuda"):
            model = HybridDecoder(cfg).to(torch.bfloat16).init_weights(0)
        eng = make_engine(model, block_size=16, num_blocks=blocks, max_seq_len=-(-(max(T, ctx) + 16) // 16) * 16,
                          max_prefill=T, max_batch=B)
        del model
        pre, dec = throughput(eng, n_seq, T, B, ctx, steps, vocab)
        res["prefill_tokens_per_s"][name], res["decode_tokens_per_s"][name] = round(pre), round(dec)
        if with_kernels:
            per = -(-T // 16)
            ent = [Entry(rng.integers(0, vocab, T), 0, np.arange(i * per, (i + 1) * per), i, [T - 1]) for i in range(n_seq)]
            rows = table(eng, ent, "prefill", timer, peaks)
            per = -(-(ctx + 1) // 16)
            ent = [Entry(rng.integers(0, vocab, 1), ctx, np.arange(i * per, (i + 1) * per), i, [0]) for i in range(B)]
            res["kernels"][name] = rows + table(eng, ent, "decode", timer, peaks)
        _cuda.check_error()
        del eng
        torch.cuda.empty_cache()
    res["gpu_launches"] = _cuda.launch_count - launches0
    return res


def equal_steps(cfg, portion: int, seqs: int, ctx: int, n: int) -> None:
    """``n`` steps of ``seqs`` prompts of ``portion`` tokens each at position ``ctx``, for a profiler."""
    from ..models.hybrid import HybridDecoder
    from ..ops import _cuda
    from ..serve.engine import make_engine
    from ..serve.hybrid import Entry
    cfg.vocab = 1024
    with torch.device("cuda"):
        model = HybridDecoder(cfg).to(torch.bfloat16).init_weights(0)
    per = (portion + ctx) // 16 + 1
    eng = make_engine(model, max_batch=seqs, block_size=16, num_blocks=seqs * per, max_seq_len=portion + ctx + 16,
                      max_prefill=portion)
    rng = np.random.default_rng(0)
    for _ in range(n):
        eng.step_logits([Entry(rng.integers(0, 1024, portion), ctx, np.arange(i * per, (i + 1) * per), i, [portion - 1])
                         for i in range(seqs)])
    torch.cuda.synchronize()
    _cuda.check_error()
    print("ok")


def steps(portion: int, seqs: int, ctx: int, n: int = 3, size: str = "m") -> None:
    """``n`` equal steps of a two-layer model (one layer of each kind): prompts of ``portion`` tokens, or one
    token each (``portion`` 1), at position ``ctx``.  A small program to put under a profiler."""
    equal_steps(hybrid_config(dict(SIZES[size], pairs=1)), portion, seqs, ctx, n)


if __name__ == "__main__":
    import argparse
    ap = argparse.ArgumentParser(description="equal steps of a two-layer hybrid decoder (for a profiler)")
    ap.add_argument("--portion", type=int, default=1024)
    ap.add_argument("--seqs", type=int, default=2)
    ap.add_argument("--ctx", type=int, default=0)
    a = ap.parse_args()
    steps(a.portion, a.seqs, a.ctx)
