"""Small random hybrid decoders for the tests: configurations, weights (rounded to bf16 so that every
precision sees the same values), engines, and requests fed portion by portion."""
import numpy as np
import torch

from brain_b200.models.config import (AttentionSpec, ClampedGluSpec, HybridConfig, HybridLayer, Mamba2Spec,
                                      RotarySpec)
from brain_b200.models.hybrid import HybridDecoder

import hybrid_oracle as oracle


def attn(heads=6, kv_heads=2, dim=40, vdim=24, scale=0.2, softcap=5.0, rot=16, base=7000.0, v_mix=True):
    return AttentionSpec(heads, kv_heads, dim, vdim, scale, softcap, RotarySpec(rot, base) if rot else None, v_mix)


def mamba(heads=6, vdim=16, state=24, groups=2, conv=4, norm_groups=3):
    return Mamba2Spec(heads, vdim, state, groups, conv, norm_groups)


def glu(ff=72, limit=1.5):
    return ClampedGluSpec(ff, limit)


def make(layers, vocab=211, width=104, eps=1e-5, mult=0.6, seed=3, sharp=1.0):
    """(model, numpy weights, config dict).  ``sharp`` scales the query gains: larger scores, so that single
    keys carry the attention."""
    cfg = HybridConfig(vocab=vocab, width=width, layers=[HybridLayer(*l) for l in layers], eps=eps, residual_mult=mult)
    m = HybridDecoder(cfg).init_weights(seed)
    for n, t in m.reference_state().items():
        if n.endswith("q.norm"):
            t.mul_(sharp)
        if n.endswith("A_log"):
            t.sub_(3.0)          # slow decay and a small skip: what the state carries shows
        if n.endswith("mix.D"):
            t.mul_(0.2)
        t.copy_(t.to(torch.bfloat16).float())
    W = {n: t.numpy().astype(np.float64) for n, t in m.reference_state().items()}
    return m, W, cfg.to_json()


def mixed_model(**kw):
    """Both kinds of layer, with and without a feed-forward, sizes that differ between layers."""
    return make([(mamba(), glu()), (attn(), None), (attn(heads=4, kv_heads=2, dim=24, rot=24), glu(40, 0.8)),
                 (mamba(heads=4, vdim=12, state=16, groups=1, conv=3, norm_groups=1), None),
                 (attn(heads=3, kv_heads=1, dim=16, vdim=32, rot=0, softcap=None, v_mix=False), glu())], **kw)


def engine(m, dtype="fp32", **kw):
    from brain_b200.serve.engine import make_engine
    opts = dict(block_size=16, num_blocks=40, max_seq_len=640, max_prefill=64, state_slots=4, dtype=dtype, device="cuda:0")
    opts.update(kw)
    return make_engine(m, **opts)


def session(m, dtype="fp32", **kw):
    from brain_b200.serve.trace_run import TraceSession
    return TraceSession(engine(m, dtype, **kw))


def tokens(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def feed(s, rid, toks, sizes, end=True):
    """One request alone in portions of the given sizes (the last repeats); logits of every token."""
    out, i, k = [], 0, 0
    while i < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - i)
        out.append(s.step([(rid, toks[i:i + n], list(range(n)))]))
        i, k = i + n, k + 1
    if end:
        s.end(rid)
    return np.concatenate(out)


def error(got, want):
    """Largest root-mean-square error of a row, mean taken off, over the root mean square of all rows."""
    d = np.asarray(got, dtype=np.float64) - want
    d = d - d.mean(axis=1, keepdims=True)
    scale = np.sqrt(np.mean((want - want.mean(axis=1, keepdims=True)) ** 2))
    return float(np.sqrt((d * d).mean(axis=1)).max() / scale)


#: rounding only: fp32 through a few layers, bf16 with its 8-bit mantissa
TOL = {"fp32": 4e-5, "bf16": 0.04}
