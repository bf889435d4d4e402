"""Small random Povipel decoders for the tests (engines and requests: ``hybrid_util``)."""
import numpy as np
import torch

import hybrid_util as hu
from brain_b200.models.config import (AttentionSpec, GatedLinearSpec, GeluSpec, HybridConfig, HybridLayer, ParallelSpec,
                                      RetentionSpec, RotarySpec, RoutedSpec, SiluGluSpec)
from brain_b200.models.hybrid import HybridDecoder


def attn(heads=6, kv_heads=2, dim=40, vdim=24, scale=0.2, rot=16, base=3000.0, window=21, pool=6):
    return AttentionSpec(heads, kv_heads, dim, vdim, scale, rot=RotarySpec(rot, base, interleaved=True), window=window, pool=pool,
                         qk_norm="head", gate=None, sink=True, turn_values=True)


def gla(heads=3, dim=24, vdim=40, tau=9.0, rank=11):
    return GatedLinearSpec(heads, dim, vdim, tau, rank)


def both(left=None, right=None):
    return ParallelSpec(left or attn(), right or gla(), 0.5, 0.5, normed=True)


def ret(heads=3, dim=40, vdim=24, rot=24, base=5000.0, decay=None):
    return RetentionSpec(heads, dim, vdim, list(decay or [1.0 - 2.0 ** (-3.0 - 2.5 * h) for h in range(heads)]), RotarySpec(rot, base))


def gelu(ff=88):
    return GeluSpec(ff)


def moe(ff=40, experts=10, top=2):
    return RoutedSpec(SiluGluSpec(ff), experts, top, scores="sigmoid", weigh_input=True)


#: kinds of token that routers tell apart (the first channels of the residual streams)
KINDS = 8


def _decide(m, rng):
    """Routing without close calls, which rounding could turn: the first channels hold the token's kind, hardly anything
    is added to them, and a router's logits for a kind's experts are well above the others'."""
    cfg = m.cfg
    for n, t in m.reference_state().items():
        if n == "embed":
            t[:, :KINDS] = 6.0 / cfg.embed_scale * torch.eye(KINDS)[torch.arange(cfg.vocab) % KINDS]
        elif n.endswith((".down", ".o")):
            t[:KINDS] *= 0.03
        elif n.endswith((".left.out", ".right.out")):
            t[:KINDS] *= 0.01
        elif ".norm2" in n:
            t[:KINDS] = 0.0 if n.endswith(".b") else 1.0
        elif n.endswith("router"):
            t.mul_(0.02)
            e = t.shape[0]
            top = cfg.layers[int(n[1:n.index(".")])].mlp.top
            levels = np.concatenate([np.linspace(-1.4, -0.6, e - top), np.linspace(0.2, 0.8, top)])
            for k in range(KINDS):
                t[:, k] = torch.from_numpy(levels[rng.permutation(e)])


def make(layers, vocab=203, width=120, eps=0.01, seed=3, sharp=1.0, streams=3, loop=None, cap=9.0, embed_scale=2.0, spread=1.0):
    """(model, numpy weights, config dict).  ``sharp`` scales the queries' gain: larger scores, so that single keys carry
    the attention.  ``spread`` scales the head, for logits near their bound.  Results enter the streams damped, and norms
    have a wide epsilon: stacks of random layers otherwise double a rounding error every layer.  Weights are rounded to
    bf16, so every precision sees the same values."""
    cfg = HybridConfig(vocab=vocab, width=width, layers=[HybridLayer(*l) for l in layers], eps=eps, design="Povipel",
                       embed_scale=embed_scale, streams=streams, loop=loop, logit_softcap=cap)
    m = HybridDecoder(cfg).init_weights(seed)
    if any(l.mlp is not None and l.mlp.kind == "routed" for l in cfg.layers):
        _decide(m, np.random.default_rng(seed))
    for n, t in m.reference_state().items():
        if n.endswith(".left.q.norm"):
            t.mul_(sharp)
        if n == "head":
            t.mul_(spread)
        if n.endswith((".hc1.out", ".hc2.out")):
            t.mul_(0.3)
        if n.endswith((".hc1.in", ".hc2.in")):
            t.mul_(0.5).add_(0.5 / streams)
        t.copy_(t.to(torch.bfloat16).float())
    W = {n: t.numpy().astype(np.float64) for n, t in m.reference_state().items()}
    return m, W, cfg.to_json()


def mixed_model(**kw):
    """Every kind of layer and feed-forward, and none; sizes that differ between layers; two layers that run twice."""
    opts = dict(loop=(2, 4, 2))
    opts.update(kw)
    return make([(both(), gelu()), (ret(), moe()), (both(attn(4, 1, 24, 56, 0.3, 24, 900.0, 34, 9), gla(2, 40, 16, 5.0, 8)), moe(24, 6, 1)),
                 (ret(2, 16, 72, 8, decay=[0.9, 0.999]), None), (both(attn(3, 3, 16, 16, 0.4, 8, 50.0, 5, 17)), gelu(40))], **opts)


def borders_model(size, pool):
    """One layer whose queries all look for loud tokens (even ids), at places that a rotation does not move: a window a key
    off, or a block seen a token off, changes what is found.  (model, numpy weights, config dict, tokens): runs of loud
    tokens about as long as a block, and quiet ones between them."""
    m, W, cfg = make([(both(attn(2, 1, 24, 24, 0.7, 8, window=size, pool=pool)), None)], vocab=64)
    p = "l0.mix.left."
    look = torch.zeros(24)
    look[8:] = 1.0
    state = m.reference_state()
    state["embed"][:, 1] = torch.where(torch.arange(64) % 2 == 0, 3.0, 0.0)
    for n, v in (("l0.norm1", 0.0), ("l0.norm1.b", 2.0), ("l0.shift", 0.0)):
        state[n][0] = v                              # a channel that is the same for every token
    state["l0.shift"][1] = 0.0
    for n, c in ((p + "q", 0), (p + "k", 1)):
        w = state[n]
        w.mul_(0.3)
        w[:, :2] = 0.0
        w[:, c] = look.repeat(w.shape[0] // 24) * 2.0
    state["l0.mix.left.out"].fill_(4.0)
    state["l0.hc1.out"].fill_(1.0)
    for n, t in state.items():
        t.copy_(t.to(torch.bfloat16).float())
        W[n] = t.numpy().astype(np.float64)
    rng, toks = np.random.default_rng(7), []
    while len(toks) < 3 * (size + pool) + 40:
        for loud in (1, 0):
            toks += (2 * rng.integers(0, 32, int(rng.integers(1, pool + 3))) + 1 - loud).tolist()
    return m, W, cfg, toks


BORDERS = [(7, 5), (16, 16), (40, 9), (20, 31), (1, 3)]


def close(got, want, dtype):
    """Rounding only.  In bf16 a stack of layers has a few rows in which a norm meets a result near zero: one row in fifty may
    be over the tolerance, none over three times of it."""
    d = np.asarray(got, dtype=np.float64) - want
    d = d - d.mean(axis=1, keepdims=True)
    scale = np.sqrt(np.mean((want - want.mean(axis=1, keepdims=True)) ** 2))
    rows = np.sort(np.sqrt((d * d).mean(axis=1)) / scale)[::-1]
    tol = hu.TOL[dtype]
    return bool(rows[0] < tol if dtype == "fp32" else rows[0] < 3 * tol and rows[min(-(-len(rows) // 50), len(rows) - 1)] < tol)
