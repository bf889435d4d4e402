"""Small random Zepesun decoders for the tests (engines and requests: ``hybrid_util``)."""
import numpy as np
import torch

import hybrid_util as hu
from brain_b200.models.config import (AttentionSpec, ClampedGluSpec, GeluGluSpec, HybridConfig, HybridLayer,
                                      LatentAttentionSpec, MlstmSpec, ParallelSpec, RotarySpec, RoutedSpec)
from brain_b200.models.hybrid import HybridDecoder


def latent(heads=5, dim=24, rot=16, vdim=40, kv_rank=56, scale=0.3, base=3000.0):
    return LatentAttentionSpec(heads, dim, rot, vdim, kv_rank, 0, scale, RotarySpec(rot, base), q_latent=False, head_gate=True)


def memory(heads=3, dim=24, vdim=40, cap=2.5):
    return MlstmSpec(heads, dim, vdim, cap)


def attn(heads=6, kv_heads=3, dim=40, vdim=24, scale=0.25, window=37):
    return AttentionSpec(heads, kv_heads, dim, vdim, scale, window=window, qk_norm=False, bias=True, gate="element")


def both(left=None, right=None, ls=0.8, rs=1.25):
    return ParallelSpec(left or attn(), right or memory(), ls, rs)


def gelu(ff=88):
    return GeluGluSpec(ff)


def moe(ff=40, limit=0.9, experts=12, top=3, groups=4, keep=2, scale=1.75, shared=(56, 1.2)):
    return RoutedSpec(ClampedGluSpec(ff, limit), experts, top, groups, keep, scale, None if shared is None else ClampedGluSpec(*shared))


#: kinds of token that routers tell apart (the first channels of the residual stream)
KINDS = 8


def _decide(m, rng):
    """Routing without close calls, which rounding could turn: the first channels hold the token's kind, hardly
    anything is added to them, and a router's logits are about a whole number apart, in another order for every kind."""
    cfg, d = m.cfg, m.cfg.width
    for n, t in m.reference_state().items():
        if n == "embed":
            t[:, :KINDS] = 6.0 / cfg.embed_scale * torch.eye(KINDS)[torch.arange(cfg.vocab) % KINDS]
        elif n == "pos":
            t[:, :KINDS] = 0.0
        elif n.endswith(("down", "down.b", ".o", "o.b")):
            t[:KINDS] *= 0.03
        elif n.endswith("router"):
            t.mul_(0.2)
            for k in range(KINDS):
                t[:, k] = torch.from_numpy(rng.permutation(t.shape[0]) * 0.2 * (1.0 + d / 240.0))


def make(layers, vocab=203, width=120, eps=3e-6, seed=3, sharp=1.0, positions=640, embed_scale=7.0):
    """(model, numpy weights, config dict).  ``sharp`` scales the queries of attention: larger scores, so that single
    keys carry it.  Weights are rounded to bf16, so every precision sees the same values."""
    cfg = HybridConfig(vocab=vocab, width=width, layers=[HybridLayer(*l) for l in layers], eps=eps, design="Zepesun",
                       max_position_embeddings=positions, embed_scale=embed_scale)
    m = HybridDecoder(cfg).init_weights(seed)
    if any(l.mlp is not None and l.mlp.kind == "routed" for l in cfg.layers):
        _decide(m, np.random.default_rng(seed))
    for n, t in m.reference_state().items():
        layer = cfg.layers[int(n[1:n.index(".")])] if n[0] == "l" else None
        if layer is not None and (n.endswith(".left.q") or (n.endswith("mix.q") and layer.mixer.kind == "latent_attention")):
            t.mul_(sharp)
        t.copy_(t.to(torch.bfloat16).float())
    W = {n: t.numpy().astype(np.float64) for n, t in m.reference_state().items()}
    return m, W, cfg.to_json()


def mixed_model(**kw):
    """Every kind of layer and feed-forward, and none; sizes that differ between layers."""
    return make([(both(), gelu()), (memory(), moe()), (latent(), moe(32, 1.5, 8, 2, 1, 1, 0.6, None)),
                 (both(attn(4, 1, 24, 56, 0.4, 90), memory(2, 40, 16), 1.3, 0.4), moe(experts=6, top=1, groups=3, keep=1)),
                 (memory(heads=1, dim=16, vdim=72, cap=6.0), None), (latent(heads=3, dim=40, rot=8, vdim=16, kv_rank=24), gelu(40))],
                **kw)
