"""Hybrid decoders: a parallel mixer + feed-forward per layer.
Pakalix mixers: soft-capped attention with rotary positions, whole-projection query / key norms, value
mixing and per-head output gates, or a Mamba-2 state-space recurrence.
Nezalorn mixers: windowed latent attention, a generalised delta rule, or a real-gated linear recurrence;
what a layer passes on is a weighted sum of all results so far.
Zepesun mixers: latent attention, a matrix memory with exponential gates, or windowed attention and a matrix
memory side by side; feed-forwards dense or a mixture of experts; learned positions.
Povipel mixers: retention, or windowed attention with pooled blocks behind the window beside gated linear attention;
several residual streams, token shifts, layers that run several times.

This is the weight container of the family (names, shapes, initial values, loading); its forward lives in
the serving engine (``serve.hybrid.HybridEngine`` over ``csrc/serve/hybrid_forward.cu``)."""
from __future__ import annotations

import math
from typing import Dict

import torch
import torch.nn as nn

from .config import HybridConfig


class HybridDecoder(nn.Module):
    family = "hybrid"

    def __init__(self, cfg: HybridConfig):
        super().__init__()
        self.cfg = cfg
        self._names = {}
        for name, shape in cfg.tensors():
            attr = name.replace(".", "__")
            self.register_parameter(attr, nn.Parameter(torch.zeros(shape), requires_grad=False))
            self._names[name] = attr

    def tensor(self, name: str) -> torch.Tensor:
        return getattr(self, self._names[name])

    @torch.no_grad()
    def init_weights(self, seed: int = 1234) -> "HybridDecoder":
        """Random values at which every mechanism works in its usual range: projections that keep the
        scale of their input, norm gains near their neutral value, step sizes between 1e-3 and 1e-1, decay
        rates between 1 and 16."""
        dev = next(self.parameters()).device
        g = torch.Generator(dev).manual_seed(seed)

        def uniform(shape, lo, hi):
            return torch.rand(shape, generator=g, device=dev) * (hi - lo) + lo

        def normal(shape):
            return torch.randn(shape, generator=g, device=dev)

        for name, shape in self.cfg.tensors():
            p = self.tensor(name)
            leaf = name.split(".", 2)[-1] if name[0] == "l" and name[1].isdigit() else name
            leaf = leaf.removeprefix("left.").removeprefix("right.")
            streams = self.cfg.streams
            if name.endswith(("hc1.in", "hc2.in")):
                v = (1.0 + 0.3 * normal(shape)) / streams
            elif name.endswith(("hc1.out", "hc2.out")):
                v = uniform(shape, 0.3, 1.2)
            elif name.endswith(("hc1.mix", "hc2.mix")):
                v = torch.eye(streams, device=dev) * 0.8 + 0.2 * normal(shape) / streams
            elif name.endswith(".shift"):
                v = uniform(shape, 0.0, 0.8)
            elif name.endswith((".norm1.b", ".norm2.b")) or name == "final.norm.b":
                v = 0.1 * normal(shape)
            elif leaf == "sink":
                v = uniform(shape, 0.0, 3.0)
            elif leaf == "a2.b":
                v = uniform(shape, -1.0, 5.0)                            # decays between fast and slow
            elif leaf == "out":
                v = 1.0 + 0.1 * normal(shape)
            elif leaf in ("embed.norm", "final.norm") or name.endswith((".norm1", ".norm2")):
                v = 1.0 - self.cfg.traits.norm_offset + 0.1 * normal(shape)
            elif leaf in ("q.norm", "k.norm", "norm", "dq.norm", "dkv.norm"):
                v = 1.0 + 0.1 * normal(shape)
            elif name.endswith(".dwa"):
                v = 0.2 * normal(shape) / shape[0]     # mostly the layer's own result
                v[-1] += 1.0
            elif leaf == "act":
                v = uniform(shape, 0.2, 0.8)
            elif leaf == "lam":
                v = uniform(shape, -5.0, -0.5)                           # decays between slow and fast
            elif leaf == "w0":
                v = uniform(shape, -8.0, 0.0)
            elif leaf == "a.b":
                v = uniform(shape, -2.0, 1.0)
            elif leaf == "f.b":
                v = uniform(shape, 2.0, 5.0)                             # most of the memory is kept
            elif leaf.endswith(".b") and leaf != "conv.b":
                v = uniform(shape, -0.3, 0.3)
            elif leaf == "vmix":
                v = uniform(shape, 0.2, 0.6)
            elif leaf == "dt_bias":
                dt = torch.exp(uniform(shape, math.log(1e-3), math.log(1e-1)))
                v = dt + torch.log(-torch.expm1(-dt))          # inverse of softplus
            elif leaf == "A_log":
                v = torch.log(uniform(shape, 1.0, 16.0))
            elif leaf == "D":
                v = uniform(shape, 0.5, 1.5)
            elif leaf == "conv":
                v = uniform(shape, -1.0, 1.0) / math.sqrt(shape[1])
            elif leaf == "conv.b":
                v = uniform(shape, -0.1, 0.1)
            elif name == "embed":
                v = normal(shape) / self.cfg.embed_scale
            elif name == "pos":
                v = 0.3 * normal(shape)
            else:
                v = normal(shape) / math.sqrt(shape[-1])
            p.copy_(v.to(p.dtype))
        return self

    # ---- checkpoint surface shared by the model families
    def reference_state(self) -> Dict[str, torch.Tensor]:
        return {n: self.tensor(n) for n, _ in self.cfg.tensors()}

    @torch.no_grad()
    def load_reference_state(self, state: Dict[str, torch.Tensor], strict: bool = True):
        mine = self.reference_state()
        missing = [n for n in mine if n not in state]
        for n, dst in mine.items():
            if n in missing:
                continue
            if state[n].numel() != dst.numel():
                raise ValueError(f"{n}: checkpoint has {tuple(state[n].shape)}, the configuration asks for {tuple(dst.shape)}")
            dst.copy_(state[n].reshape(dst.shape).to(dst.dtype))
        if strict and missing:
            raise KeyError(f"checkpoint is missing {len(missing)} tensors, e.g. {missing[:4]}")
        return missing

    def config_json(self) -> dict:
        return self.cfg.to_json()

    def flops_per_token(self, T: int, train: bool = False) -> float:
        """Matrix-product FLOPs of one token with T tokens of context, attention and recurrence included."""
        total, runs = 0.0, self.cfg.runs
        for n, s in self.cfg.tensors():
            if len(s) > 1 and n != "pos" and ".hc" not in n and (n != "embed" or self.cfg.traits.tied) and not n.endswith((".conv", "a.b", "i.b")):
                share = 1.0
                if ".mlp.e" in n:            # of a token's own experts
                    f = self.cfg.layers[int(n[1:n.index(".")])].mlp
                    share = f.top / f.experts
                if n[0] == "l" and n[1].isdigit():
                    share *= runs.count(int(n[1:n.index(".")]))
                total += 2.0 * share * math.prod(s)
        return total + sum(self.cfg.layers[i].mixer.flops(T) for i in self.cfg.runs)
