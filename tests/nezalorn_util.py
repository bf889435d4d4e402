"""Small random Nezalorn decoders for the tests (engines, requests and error measures: ``hybrid_util``)."""
import numpy as np
import torch

from brain_b200.models.config import (GeneralDeltaSpec, HybridConfig, HybridLayer, LatentAttentionSpec, PolyNormSpec,
                                      RgLruSpec, RotarySpec, YarnSpec)
from brain_b200.models.hybrid import HybridDecoder

YARN = YarnSpec(factor=5.0, original=300.0, fast=24.0, slow=1.5)


def latent(heads=5, dim=24, rot=16, vdim=40, kv_rank=48, q_rank=56, scale=0.3, window=37, base=3000.0, yarn=YARN, kv_from=None):
    return LatentAttentionSpec(heads, dim, rot, vdim, kv_rank, q_rank, scale, RotarySpec(rot, base, yarn, True), window, kv_from)


def delta(heads=3, dim=24, rank=10):
    return GeneralDeltaSpec(heads, dim, rank)


def lru(width=96, blocks=3, conv=4):
    return RgLruSpec(width, blocks, conv)


def poly(ff=88):
    return PolyNormSpec(ff)


def make(layers, vocab=203, width=120, eps=3e-6, seed=3, sharp=1.0):
    """(model, numpy weights, config dict).  ``sharp`` scales the latent queries: larger scores, so that single
    keys carry the attention.  Weights are rounded to bf16, so every precision sees the same values."""
    cfg = HybridConfig(vocab=vocab, width=width, layers=[HybridLayer(*l) for l in layers], eps=eps, design="Nezalorn")
    m = HybridDecoder(cfg).init_weights(seed)
    for n, t in m.reference_state().items():
        if n.endswith("dq.norm"):
            t.mul_(sharp)
        t.copy_(t.to(torch.bfloat16).float())
    W = {n: t.numpy().astype(np.float64) for n, t in m.reference_state().items()}
    return m, W, cfg.to_json()


def mixed_model(**kw):
    """Every kind of layer, with and without a feed-forward, sizes that differ between layers, latents shared
    with a later layer of other heads and another window."""
    return make([(lru(), poly()), (latent(), poly(40)), (delta(), None),
                 (latent(heads=3, dim=40, vdim=16, q_rank=32, window=90, kv_from=1), poly()),
                 (lru(width=60, blocks=4, conv=3), None), (delta(heads=2, dim=40, rank=16), poly(56)),
                 (latent(heads=4, dim=16, rot=8, vdim=8, kv_rank=24, q_rank=20, window=5, yarn=None), None)], **kw)
