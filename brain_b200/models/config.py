"""Model configuration records and their checkpoint JSON (the ``brain.config`` metadata string).

Key names and presets follow the reference so checkpoints stay interchangeable:
Qwen ``crates/qwen3/src/config.rs:44-73,100-188,219-238``; GPT ``crates/gpt2/src/model.rs:254-260``;
toy MoE ``crates/toymoe/src/train.rs:100-167``.  The 14B dense and 30B-A3B MoE shapes are presets
added here (the reference has none)."""
from __future__ import annotations

import json
import math
from dataclasses import dataclass, field, asdict
from typing import List, Optional


@dataclass
class LoraCfg:
    rank: int = 8
    alpha: float = 16.0
    targets: List[str] = field(default_factory=lambda: ["wq", "wk", "wv", "wo"])


@dataclass
class QwenConfig:
    vocab: int = 151936
    block_size: int = 1024
    n_layers: int = 28
    d_model: int = 1024
    n_heads: int = 16
    n_kv_heads: int = 8
    head_dim: int = 128
    d_ff: int = 3072
    rope_theta: float = 1.0e6
    rms_eps: float = 1e-6
    max_position_embeddings: int = 0
    tie_embeddings: bool = True
    qk_norm: bool = True
    attn_bias: bool = False
    lora: Optional[LoraCfg] = None

    def __post_init__(self):
        if not self.max_position_embeddings:
            self.max_position_embeddings = self.block_size

    # ---- JSON (checkpoint metadata) ----
    def to_json(self) -> dict:
        v = {
            "model": "qwen", "vocab_size": self.vocab, "block_size": self.block_size,
            "n_layers": self.n_layers, "d_model": self.d_model, "n_heads": self.n_heads,
            "n_kv_heads": self.n_kv_heads, "head_dim": self.head_dim, "d_ff": self.d_ff,
            "rope_theta": self.rope_theta, "rms_norm_eps": self.rms_eps,
            "max_position_embeddings": self.max_position_embeddings,
            "tie_word_embeddings": self.tie_embeddings,
        }
        if not self.qk_norm:
            v["qk_norm"] = False
        if self.attn_bias:
            v["attn_bias"] = True
        if self.lora is not None:
            v["lora"] = {"rank": self.lora.rank, "alpha": self.lora.alpha,
                         "targets": list(self.lora.targets)}
        return v

    @staticmethod
    def from_json(c: dict) -> "QwenConfig":
        lora = None
        if c.get("lora"):
            l = c["lora"]
            lora = LoraCfg(int(l["rank"]), float(l["alpha"]), list(l.get("targets", [])))
        bs = int(c.get("block_size", 1024))
        return QwenConfig(
            vocab=int(c["vocab_size"]), block_size=bs, n_layers=int(c["n_layers"]),
            d_model=int(c["d_model"]), n_heads=int(c["n_heads"]),
            n_kv_heads=int(c.get("n_kv_heads", c["n_heads"])),
            head_dim=int(c.get("head_dim", int(c["d_model"]) // int(c["n_heads"]))),
            d_ff=int(c["d_ff"]), rope_theta=float(c.get("rope_theta", 1e6)),
            rms_eps=float(c.get("rms_norm_eps", 1e-6)),
            max_position_embeddings=int(c.get("max_position_embeddings", bs)),
            tie_embeddings=bool(c.get("tie_word_embeddings", True)),
            qk_norm=bool(c.get("qk_norm", True)), attn_bias=bool(c.get("attn_bias", False)),
            lora=lora)

    # ---- presets ----
    @staticmethod
    def tiny() -> "QwenConfig":
        return QwenConfig(vocab=23, block_size=12, n_layers=2, d_model=16, n_heads=4, n_kv_heads=2,
                          head_dim=8, d_ff=32)

    @staticmethod
    def cli_default(vocab: int, block: int) -> "QwenConfig":
        """The architecture ``brain qwen3 train`` builds (crates/cli/src/qwen_cli.rs:368-475)."""
        return QwenConfig(vocab=vocab, block_size=block, n_layers=6, d_model=384, n_heads=6,
                          n_kv_heads=2, head_dim=64, d_ff=1024)

    @staticmethod
    def preset(name: str, block_size: int = 0) -> "QwenConfig":
        shapes = {
            "0.6b": dict(n_layers=28, d_model=1024, n_heads=16, n_kv_heads=8, d_ff=3072,
                         tie_embeddings=True),
            "1.7b": dict(n_layers=28, d_model=2048, n_heads=16, n_kv_heads=8, d_ff=6144,
                         tie_embeddings=True),
            "4b": dict(n_layers=36, d_model=2560, n_heads=32, n_kv_heads=8, d_ff=9728,
                       tie_embeddings=True),
            "8b": dict(n_layers=36, d_model=4096, n_heads=32, n_kv_heads=8, d_ff=12288,
                       tie_embeddings=False),
            "14b": dict(n_layers=40, d_model=5120, n_heads=40, n_kv_heads=8, d_ff=17408,
                        tie_embeddings=False),
        }
        key = name.lower().replace("qwen3-", "")
        if key not in shapes:
            raise KeyError(f"unknown Qwen3 preset {name!r}; have {sorted(shapes)}")
        c = QwenConfig(vocab=151936, head_dim=128, rope_theta=1e6, **shapes[key])
        if block_size:
            c.block_size = block_size
            c.max_position_embeddings = block_size
        return c

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    def param_list(self):
        """(name, numel) in checkpoint order (crates/qwen3/src/config.rs:311-366)."""
        d, out = self.d_model, []
        out.append(("tok.weight", self.vocab * d))

        def lin(name, o, i, bias=False):
            out.append((f"{name}.weight", o * i))
            if bias:
                out.append((f"{name}.bias", o))
            if self.lora is not None and name.rsplit(".", 1)[-1] in self.lora.targets:
                out.append((f"{name}.lora_a", self.lora.rank * i))
                out.append((f"{name}.lora_b", o * self.lora.rank))

        for l in range(self.n_layers):
            p = f"blocks.{l}"
            out.append((f"{p}.ln1.weight", d))
            lin(f"{p}.attn.wq", self.q_dim, d, self.attn_bias)
            lin(f"{p}.attn.wk", self.kv_dim, d, self.attn_bias)
            lin(f"{p}.attn.wv", self.kv_dim, d, self.attn_bias)
            if self.qk_norm:
                out.append((f"{p}.attn.q_norm.weight", self.head_dim))
                out.append((f"{p}.attn.k_norm.weight", self.head_dim))
            lin(f"{p}.attn.wo", d, self.q_dim)
            out.append((f"{p}.ln2.weight", d))
            lin(f"{p}.mlp.gate", self.d_ff, d)
            lin(f"{p}.mlp.up", self.d_ff, d)
            lin(f"{p}.mlp.down", d, self.d_ff)
        out.append(("norm.weight", d))
        if not self.tie_embeddings:
            out.append(("lm_head.weight", self.vocab * d))
        return out

    def param_count(self) -> int:
        return sum(n for _, n in self.param_list())


@dataclass
class GptConfig:
    vocab: int = 50257
    block_size: int = 1024
    n_layers: int = 12
    d_model: int = 768
    n_heads: int = 12
    d_ff: int = 3072
    itos: Optional[List[str]] = None

    def to_json(self) -> dict:
        v = {"model": "gpt", "vocab_size": self.vocab, "block_size": self.block_size,
             "n_layers": self.n_layers, "d_model": self.d_model, "n_heads": self.n_heads,
             "d_ff": self.d_ff}
        if self.itos is not None:
            v["itos"] = list(self.itos)
        return v

    @staticmethod
    def from_json(c: dict) -> "GptConfig":
        return GptConfig(vocab=int(c["vocab_size"]), block_size=int(c["block_size"]),
                         n_layers=int(c["n_layers"]), d_model=int(c["d_model"]),
                         n_heads=int(c["n_heads"]), d_ff=int(c.get("d_ff", 4 * int(c["d_model"]))),
                         itos=c.get("itos"))

    @staticmethod
    def small() -> "GptConfig":
        return GptConfig()

    @staticmethod
    def gradcheck() -> "GptConfig":
        """The shape of the CLI gradcheck gate (crates/gradcheck/src/lib.rs:290-300)."""
        return GptConfig(vocab=23, block_size=12, n_layers=2, d_model=16, n_heads=2, d_ff=32)

    def param_list(self):
        d, ff = self.d_model, self.d_ff
        out = [("tok.weight", self.vocab * d), ("pos.weight", self.block_size * d)]
        for l in range(self.n_layers):
            p = f"blocks.{l}"
            out += [(f"{p}.ln1.weight", d), (f"{p}.ln1.bias", d),
                    (f"{p}.attn.qkv.weight", 3 * d * d), (f"{p}.attn.qkv.bias", 3 * d),
                    (f"{p}.attn.out.weight", d * d), (f"{p}.attn.out.bias", d),
                    (f"{p}.ln2.weight", d), (f"{p}.ln2.bias", d),
                    (f"{p}.mlp.fc.weight", ff * d), (f"{p}.mlp.fc.bias", ff),
                    (f"{p}.mlp.proj.weight", d * ff), (f"{p}.mlp.proj.bias", d)]
        out += [("ln.weight", d), ("ln.bias", d), ("lm_head.weight", self.vocab * d)]
        return out

    def param_count(self) -> int:
        return sum(n for _, n in self.param_list())


@dataclass
class MoeConfig:
    """Sparse top-k MoE transformer.  ``family='toymoe'`` keeps the toy model's layout (fused qkv,
    interleaved RoPE, no QK-norm, names ``token_emb``/``norm1``/``norm2``); ``family='qwen3_moe'``
    is the Qwen3-MoE decoder (GQA + QK-norm + NeoX RoPE, names as the dense Qwen3 plus
    ``blocks.{l}.moe.router`` / ``blocks.{l}.moe.experts.{e}.{w_gate,w_up,w_down}``)."""
    family: str = "qwen3_moe"
    vocab: int = 151936
    block_size: int = 4096
    n_layers: int = 48
    d_model: int = 2048
    n_heads: int = 32
    n_kv_heads: int = 4
    head_dim: int = 128
    n_experts: int = 128
    top_k: int = 8
    d_ff: int = 768
    rope_theta: float = 1.0e6
    rms_eps: float = 1e-6
    aux_coef: float = 0.001
    z_coef: float = 0.0
    norm_topk_prob: bool = True
    routed_scaling: float = 1.0
    tie_embeddings: bool = False

    def to_json(self) -> dict:
        v = asdict(self)
        v["model"] = "moe" if self.family == "toymoe" else "qwen_moe"
        v["vocab_size"] = v.pop("vocab")
        v["rms_norm_eps"] = v.pop("rms_eps")
        v["tie_word_embeddings"] = v.pop("tie_embeddings")
        return v

    @staticmethod
    def from_json(c: dict) -> "MoeConfig":
        c = dict(c)
        c.pop("model", None)
        c["vocab"] = c.pop("vocab_size")
        c["rms_eps"] = c.pop("rms_norm_eps", 1e-6)
        c["tie_embeddings"] = c.pop("tie_word_embeddings", False)
        known = {f for f in MoeConfig.__dataclass_fields__}
        return MoeConfig(**{k: v for k, v in c.items() if k in known})

    @staticmethod
    def qwen3_30b_a3b(block_size: int = 4096) -> "MoeConfig":
        return MoeConfig(block_size=block_size)

    @staticmethod
    def toy(vocab: int = 64, block: int = 32) -> "MoeConfig":
        """Defaults of ``brain toymoe train`` (crates/toymoe/src/train.rs:700-730)."""
        return MoeConfig(family="toymoe", vocab=vocab, block_size=block, n_layers=2, d_model=64,
                         n_heads=4, n_kv_heads=4, head_dim=16, n_experts=4, top_k=2, d_ff=128,
                         rope_theta=10000.0, aux_coef=0.01, z_coef=1e-4, tie_embeddings=True)

    @property
    def q_dim(self):
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self):
        return self.n_kv_heads * self.head_dim

    def param_list(self):
        d, out = self.d_model, []
        toy = self.family == "toymoe"
        out.append(("token_emb.weight" if toy else "tok.weight", self.vocab * d))
        for l in range(self.n_layers):
            p = f"blocks.{l}"
            if toy:
                out += [(f"{p}.norm1.weight", d), (f"{p}.attn.qkv.weight", 3 * d * d),
                        (f"{p}.attn.out.weight", d * d), (f"{p}.norm2.weight", d)]
            else:
                out += [(f"{p}.ln1.weight", d), (f"{p}.attn.wq.weight", self.q_dim * d),
                        (f"{p}.attn.wk.weight", self.kv_dim * d),
                        (f"{p}.attn.wv.weight", self.kv_dim * d),
                        (f"{p}.attn.q_norm.weight", self.head_dim),
                        (f"{p}.attn.k_norm.weight", self.head_dim),
                        (f"{p}.attn.wo.weight", d * self.q_dim), (f"{p}.ln2.weight", d)]
            out.append((f"{p}.moe.router.weight", self.n_experts * d))
            for e in range(self.n_experts):
                q = f"{p}.moe.experts.{e}"
                out += [(f"{q}.w_gate.weight", self.d_ff * d), (f"{q}.w_up.weight", self.d_ff * d),
                        (f"{q}.w_down.weight", d * self.d_ff)]
        out.append(("norm.weight", d))
        if not self.tie_embeddings:
            out.append(("lm_head.weight", self.vocab * d))
        return out

    def param_count(self) -> int:
        return sum(n for _, n in self.param_list())


# ------------------------------------------------------------------------------------ hybrid decoders
# A decoder described layer by layer: every layer names its mixer (attention or a state-space
# recurrence) with sizes of its own, and its feed-forward.  The records below are mechanisms with their
# constants as fields; a design is a reader of its config file (``HYBRID_DESIGNS``) that fills them in.

@dataclass
class YarnSpec:
    """Per-pair frequency interpolation: pairs that turn more than ``fast`` times over the original context
    keep their frequency, those that turn less than ``slow`` times have it divided by ``factor``, with a
    ramp in between; cos and sin grow by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass
class RotarySpec:
    dims: int                    # leading dimensions of a head that are rotated
    base: float
    scaling: Optional[YarnSpec] = None
    interleaved: bool = False    # neighbouring pairs (2i, 2i + 1) instead of half-split ones

    def frequencies(self):
        """(angle per position of every pair, factor on cos and sin), in double precision."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        y = self.scaling
        if y is None:
            return f, 1.0
        turns = lambda t: self.dims * math.log(y.original / (2 * math.pi * t)) / (2 * math.log(self.base))
        lo, hi = max(math.floor(turns(y.fast)), 0), min(math.ceil(turns(y.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [v / y.factor * r + v * (1.0 - r) for v, r in zip(f, ramp)], 0.1 * math.log(y.factor) + 1.0

    @staticmethod
    def from_json(c: dict, interleaved: bool = False) -> "RotarySpec":
        y = c.get("scaling")
        return RotarySpec(int(c["dims"]), float(c["base"]),
                          None if not y else YarnSpec(*(float(y[k]) for k in ("factor", "original", "fast", "slow"))),
                          interleaved)


@dataclass
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                     # query / key head size
    vdim: int                    # value head size
    scale: float
    softcap: Optional[float] = None
    rot: Optional[RotarySpec] = None
    v_mix: bool = False          # values mixed with those of the first layer that has this set
    window: Optional[int] = None     # keys a query sees, itself included (None: every earlier one)
    qk_norm: object = True       # root-mean-square norm of queries and keys: True over the whole projections, "head" over
                                 # every head with one gain for all of them, False none
    bias: bool = False           # on the query, key, value and output projections
    gate: Optional[str] = "head"     # sigmoid gate on the output: one value per head, or one per element
    pool: Optional[int] = None   # behind the window: one mean key and value per block of this many tokens
    sink: bool = False           # a learned number per head in the softmax's denominator
    turn_values: bool = False    # values rotated like keys (over all of a head), outputs rotated back
    kind = "attention"
    recurrent = False

    @staticmethod
    def from_json(m: dict, interleaved: bool = False, **constants) -> "AttentionSpec":
        rot, mask = m.get("rot"), m.get("mask") or {}
        return AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                             scale=float(m["scale"]), softcap=float(m["softcap"]) if m.get("softcap") else None,
                             rot=RotarySpec.from_json(rot, interleaved=interleaved) if rot else None,
                             v_mix=bool(m.get("v_mix", False)), window=int(mask["size"]) if mask.get("size") else None,
                             pool=int(mask["pool"]) if mask.get("pool") else None, **constants)

    def to_json(self) -> dict:
        m = {k: v for k, v in asdict(self).items()
             if v is not None and k not in ("window", "qk_norm", "bias", "gate", "pool", "sink", "turn_values")}
        if self.rot is not None:
            m["rot"] = {"dims": self.rot.dims, "base": self.rot.base}
        if self.window is not None:
            m["mask"] = {"size": self.window}
            if self.pool is not None:
                m["mask"]["pool"] = self.pool
        if self.qk_norm is not True:
            del m["v_mix"]
        return m

    @property
    def value_rot(self) -> Optional[RotarySpec]:
        return RotarySpec(self.vdim, self.rot.base, interleaved=self.rot.interleaved) if self.turn_values and self.rot else None

    def check(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"attention: {self.heads} heads over {self.kv_heads} key/value heads")
        if self.rot is not None and (self.rot.dims % 2 or self.rot.dims > self.dim):
            raise ValueError(f"attention: cannot rotate {self.rot.dims} of {self.dim} dimensions")
        if self.window is not None and self.window < 1:
            raise ValueError("attention: the window holds at least the token itself")
        if not self.qk_norm and (self.rot is not None or self.v_mix):
            raise ValueError("attention: rotation and value mixing come with normed queries and keys")
        if self.pool is not None and (self.pool < 1 or self.window is None):
            raise ValueError("attention: pooled blocks hold a token or more and lie behind a window")
        if self.turn_values and (self.rot is None or self.vdim % 2):
            raise ValueError(f"attention: cannot rotate values of {self.vdim} dimensions")
        if self.qk_norm == "head" and (self.softcap is not None or self.v_mix or self.bias):
            raise ValueError("attention: soft caps, value mixing and biases do not come with norms per head")
        if self.qk_norm != "head" and (self.pool is not None or self.sink or self.turn_values or self.gate is None):
            raise ValueError("attention: pooled blocks, sinks and rotated values come with norms per head")

    def tensors(self, width: int):
        out = []
        for n, rows in (("q", self.heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.kv_heads * self.vdim)):
            out.append((n, (rows, width)))
            if self.bias:
                out.append((n + ".b", (rows,)))
        if self.qk_norm == "head":
            out += [("q.norm", (self.dim,)), ("k.norm", (self.dim,))]
        elif self.qk_norm:
            out += [("q.norm", (self.heads * self.dim,)), ("k.norm", (self.kv_heads * self.dim,))]
        if self.v_mix:
            out.append(("vmix", ()))
        if self.sink:
            out.append(("sink", (self.heads,)))
        if self.gate is not None:
            out.append(("g", (self.heads * (self.vdim if self.gate == "element" else 1), width)))
        out.append(("o", (width, self.heads * self.vdim)))
        return out + [("o.b", (width,))] if self.bias else out

    def flops(self, T: int) -> float:
        keys = min(T, self.window or T)
        if self.pool is not None:
            keys += (T - keys) // self.pool
        return 2.0 * self.heads * (self.dim + self.vdim) * keys


@dataclass
class Mamba2Spec:
    heads: int
    vdim: int                    # channels of a head
    state: int
    groups: int                  # heads of a group share B and C
    conv: int                    # taps of the short convolution
    norm_groups: int
    kind = "mamba2"
    recurrent = True

    @staticmethod
    def from_json(m: dict) -> "Mamba2Spec":
        return Mamba2Spec(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]),
                          conv=int(m["conv"]), norm_groups=int(m["norm_groups"]))

    def to_json(self) -> dict:
        return asdict(self)

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def check(self):
        if self.heads % self.groups:
            raise ValueError(f"mamba2: {self.heads} heads over {self.groups} groups")
        if self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.inner} channels in {self.norm_groups} norm groups")
        if self.conv < 1:
            raise ValueError("mamba2: the convolution needs at least one tap")

    def tensors(self, width: int):
        return [("in", (self.inner + self.channels + self.heads, width)), ("conv", (self.channels, self.conv)),
                ("conv.b", (self.channels,)), ("dt_bias", (self.heads,)), ("A_log", (self.heads,)),
                ("D", (self.heads,)), ("norm", (self.inner,)), ("o", (width, self.inner))]

    def flops(self, T: int) -> float:
        return 6.0 * self.heads * self.state * self.vdim


@dataclass
class LatentAttentionSpec:
    """Attention whose keys and values are projections of one cached latent per token, plus one rotated key
    part that all heads share; queries go through a latent of their own, or straight from the input."""
    heads: int
    dim: int                     # unrotated query / key dimensions of a head
    rot_dim: int                 # rotated ones
    vdim: int
    kv_rank: int
    q_rank: int                  # 0 with q_latent: as the checkpoint has it
    scale: float
    rot: RotarySpec = None
    window: Optional[int] = None     # keys a query sees, itself included (None: every earlier one)
    kv_from: Optional[int] = None    # the layer whose latents and rotated key parts are used
    q_latent: bool = True        # queries go through a latent of their own
    head_gate: bool = False      # sigmoid gate on every head's output
    kind = "latent_attention"
    recurrent = False

    @staticmethod
    def from_json(m: dict, interleaved: bool = True, **constants) -> "LatentAttentionSpec":
        mask, j = m.get("mask") or {}, m.get("kv_from")
        rot = dict(m["rot"])
        rot.setdefault("dims", m["rot_dim"])
        return LatentAttentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                   kv_rank=int(m["kv_rank"]), q_rank=int(m.get("q_rank") or 0), scale=float(m["scale"]),
                                   rot=RotarySpec.from_json(rot, interleaved=interleaved),
                                   window=int(mask["size"]) if mask.get("size") else None,
                                   kv_from=None if j is None else int(j), **constants)

    def to_json(self) -> dict:
        m = {k: v for k, v in asdict(self).items() if k not in ("rot", "window", "kv_from", "q_latent", "head_gate")}
        if not self.q_latent:
            del m["q_rank"]
        m["rot"] = {"dims": self.rot.dims, "base": self.rot.base}
        if self.rot.scaling is not None:
            m["rot"]["scaling"] = asdict(self.rot.scaling)
        if self.window is not None:
            m["mask"] = {"size": self.window}
        if self.kv_from is not None:
            m["kv_from"] = self.kv_from
        return m

    def fill(self, shape):
        if self.q_latent:
            self.q_rank = self.q_rank or shape("dq")[0]

    def check(self):
        if self.rot.dims != self.rot_dim or self.rot_dim % 2:
            raise ValueError(f"latent attention: cannot rotate {self.rot.dims} of {self.rot_dim} dimensions")
        if self.window is not None and self.window < 1:
            raise ValueError("latent attention: the window holds at least the token itself")

    def tensors(self, width: int):
        rows = self.heads * (self.dim + self.rot_dim)
        out = [("dq", (self.q_rank, width)), ("dq.norm", (self.q_rank,)), ("uq", (rows, self.q_rank))] if self.q_latent else \
            [("q", (rows, width))]
        if self.kv_from is None:
            out += [("dkv", (self.kv_rank + self.rot_dim, width)), ("dkv.norm", (self.kv_rank,))]
        out += [("uk", (self.heads * self.dim, self.kv_rank)), ("uv", (self.heads * self.vdim, self.kv_rank))]
        if self.head_gate:
            out.append(("g", (self.heads, width)))
        return out + [("o", (width, self.heads * self.vdim))]

    def flops(self, T: int) -> float:
        return 2.0 * self.heads * (self.dim + self.rot_dim + self.vdim) * min(T, self.window or T)


@dataclass
class GeneralDeltaSpec:
    """Delta rule with a decay and a removal rate of its own for every key channel; the decay comes from a
    low-rank projection of ``decay_rank`` (0: as the checkpoint has it)."""
    heads: int
    dim: int
    decay_rank: int = 0
    kind = "general_delta"
    recurrent = True

    @property
    def inner(self) -> int:
        return self.heads * self.dim

    @staticmethod
    def from_json(m: dict) -> "GeneralDeltaSpec":
        return GeneralDeltaSpec(heads=int(m["heads"]), dim=int(m["dim"]), decay_rank=int(m.get("decay_rank") or 0))

    def to_json(self) -> dict:
        return asdict(self)

    def fill(self, shape):
        self.decay_rank = self.decay_rank or shape("w1")[0]

    def check(self):
        pass

    def tensors(self, width: int):
        n = self.inner
        return [("r", (n, width)), ("k", (n, width)), ("v", (n, width)), ("g", (n, width)), ("a", (n, width)),
                ("a.b", (n,)), ("w1", (self.decay_rank, width)), ("w2", (n, self.decay_rank)), ("w0", (n,)),
                ("norm", (n,)), ("o", (width, n))]

    def flops(self, T: int) -> float:
        return 10.0 * self.heads * self.dim * self.dim


@dataclass
class RgLruSpec:
    """Gated linear recurrence per channel behind a short convolution, its gates from block-diagonal maps,
    beside a gelu branch that multiplies its output."""
    width: int                   # channels
    blocks: int                  # equal parts of the gates' maps
    conv: int
    decay: float = 8.0           # log a = -decay r softplus(lam)
    kind = "rglru"
    recurrent = True

    @staticmethod
    def from_json(m: dict) -> "RgLruSpec":
        return RgLruSpec(width=int(m["width"]), blocks=int(m["blocks"]), conv=int(m["conv"]))

    def to_json(self) -> dict:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}

    def check(self):
        if self.blocks < 1 or self.width % self.blocks:
            raise ValueError(f"rglru: {self.width} channels in {self.blocks} blocks")
        if self.conv < 1:
            raise ValueError("rglru: the convolution needs at least one tap")

    def tensors(self, width: int):
        n, b = self.width, self.width // self.blocks
        return [("y", (n, width)), ("y.b", (n,)), ("x", (n, width)), ("x.b", (n,)), ("conv", (n, self.conv)), ("conv.b", (n,)),
                ("ra", (self.blocks, b, b)), ("ra.b", (self.blocks, b)), ("ri", (self.blocks, b, b)),
                ("ri.b", (self.blocks, b)), ("lam", (n,)), ("o", (width, n))]

    def flops(self, T: int) -> float:
        return 12.0 * self.width


@dataclass
class MlstmSpec:
    """Matrix memory with exponential gates: per head a state of key x value channels, a normaliser of key
    channels and the running maximum of the gates' logarithms, which are bounded by ``gate_cap``."""
    heads: int
    dim: int                     # query / key head size
    vdim: int
    gate_cap: float
    kind = "mlstm"
    recurrent = True

    @staticmethod
    def from_json(m: dict) -> "MlstmSpec":
        return MlstmSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))

    def to_json(self) -> dict:
        return asdict(self)

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    def check(self):
        if not self.gate_cap > 0:
            raise ValueError("mlstm: the gates' bound is positive")

    def tensors(self, width: int):
        n, h = self.inner, self.heads
        return [("q", (h * self.dim, width)), ("k", (h * self.dim, width)), ("v", (n, width)), ("g", (n, width)),
                ("o", (width, n)), ("norm", (n,)), ("i", (h, width)), ("i.b", (h,)), ("f", (h, width)), ("f.b", (h,))]

    def flops(self, T: int) -> float:
        return 6.0 * self.heads * self.dim * self.vdim


@dataclass
class GatedLinearSpec:
    """Linear attention whose state (key x value channels per head) decays by a rate of its own for every key channel
    and token, sigmoid(z)^(1 / tau) with z from a low-rank projection of ``decay_rank`` (0: as the checkpoint has it)."""
    heads: int
    dim: int                     # query / key head size
    vdim: int
    tau: float
    decay_rank: int = 0
    kind = "gated_linear"
    recurrent = True

    @staticmethod
    def from_json(m: dict) -> "GatedLinearSpec":
        return GatedLinearSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]),
                               decay_rank=int(m.get("decay_rank") or 0))

    def to_json(self) -> dict:
        return {k: v for k, v in asdict(self).items() if v}

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    def fill(self, shape):
        self.decay_rank = self.decay_rank or shape("a1")[0]

    def check(self):
        if not self.tau > 0:
            raise ValueError("gated linear attention: the decay's root is positive")
        if self.dim > 512:
            raise ValueError("gated linear attention: heads of up to 512 key channels")

    def tensors(self, width: int):
        k, v = self.heads * self.dim, self.heads * self.vdim
        return [("q", (k, width)), ("k", (k, width)), ("v", (v, width)), ("g", (v, width)), ("o", (width, v)),
                ("norm", (self.vdim,)), ("a1", (self.decay_rank, width)), ("a2", (k, self.decay_rank)), ("a2.b", (k,))]

    def flops(self, T: int) -> float:
        return 6.0 * self.heads * self.dim * self.vdim


@dataclass
class RetentionSpec:
    """Linear attention whose state decays by a constant per head; queries and keys are rotated."""
    heads: int
    dim: int
    vdim: int
    decay: List[float]
    rot: Optional[RotarySpec] = None
    kind = "retention"
    recurrent = True

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @staticmethod
    def from_json(m: dict, interleaved: bool = False) -> "RetentionSpec":
        rot = m.get("rot")
        return RetentionSpec(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), decay=[float(x) for x in m["decay"]],
                             rot=RotarySpec.from_json(rot, interleaved=interleaved) if rot else None)

    def to_json(self) -> dict:
        m = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        return m if self.rot is None else dict(m, rot={"dims": self.rot.dims, "base": self.rot.base})

    def check(self):
        if len(self.decay) != self.heads or not all(0.0 < x <= 1.0 for x in self.decay):
            raise ValueError(f"retention: a decay in (0, 1] for each of {self.heads} heads")
        if self.rot is not None and (self.rot.dims % 2 or self.rot.dims > self.dim):
            raise ValueError(f"retention: cannot rotate {self.rot.dims} of {self.dim} dimensions")
        if self.dim > 512:
            raise ValueError("retention: heads of up to 512 key channels")

    def tensors(self, width: int):
        k, v = self.heads * self.dim, self.heads * self.vdim
        return [("q", (k, width)), ("k", (k, width)), ("v", (v, width)), ("g", (v, width)), ("o", (width, v))]

    def flops(self, T: int) -> float:
        return 6.0 * self.heads * self.dim * self.vdim


@dataclass
class ParallelSpec:
    """Two mixers reading the same input; their results are added with a factor each, either as they are or
    (``normed``) each over its root mean square and times a gain."""
    left: object
    right: object
    left_scale: float
    right_scale: float
    normed: bool = False
    kind = "parallel"

    @staticmethod
    def from_json(m: dict, left, right, normed: bool = False) -> "ParallelSpec":
        factor = (lambda n: 0.5) if normed else (lambda n: float(m[n]))
        return ParallelSpec(left(m["left"]), right(m["right"]), factor("left_scale"), factor("right_scale"), normed)

    def to_json(self) -> dict:
        m = {"left": self.left.to_json(), "right": self.right.to_json()}
        return m if self.normed else dict(m, left_scale=self.left_scale, right_scale=self.right_scale)

    def fill(self, shape):
        for side in ("left", "right"):
            m = getattr(self, side)
            if hasattr(m, "fill"):
                m.fill(lambda n, side=side: shape(side + "." + n))

    @property
    def recurrent(self) -> bool:
        return self.left.recurrent or self.right.recurrent

    def check(self):
        self.left.check()
        self.right.check()

    def tensors(self, width: int):
        out = [(side + "." + n, s) for side in ("left", "right") for n, s in getattr(self, side).tensors(width)]
        return out + [("left.out", (width,)), ("right.out", (width,))] if self.normed else out

    def flops(self, T: int) -> float:
        return self.left.flops(T) + self.right.flops(T)


@dataclass
class ClampedGluSpec:
    """min(g, limit) sigmoid(alpha g) (clamp(u) + shift) between the gate / up and down projections."""
    ff: int
    limit: float
    alpha: float = 1.702
    shift: float = 1.0
    kind = "clamped_glu"

    @staticmethod
    def from_json(f: dict) -> "ClampedGluSpec":
        return ClampedGluSpec(int(f["ff"]), float(f["limit"]))

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}

    def tensors(self, width: int):
        return [("gate", (self.ff, width)), ("up", (self.ff, width)), ("down", (width, self.ff))]


@dataclass
class PolyNormSpec:
    """a N(z) + b N(z^2) + c N(z^3) + e between the up and down projections, N dividing by the root mean
    square; projections with biases."""
    ff: int
    kind = "polynorm"

    @staticmethod
    def from_json(f: dict) -> "PolyNormSpec":
        return PolyNormSpec(int(f["ff"]))

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff}

    def tensors(self, width: int):
        return [("up", (self.ff, width)), ("up.b", (self.ff,)), ("down", (width, self.ff)), ("down.b", (width,)), ("act", (4,))]


@dataclass
class GeluGluSpec:
    """gelu(gate) up between the gate / up and down projections (gelu in its tanh form); projections with biases."""
    ff: int
    kind = "gelu_glu"

    @staticmethod
    def from_json(f: dict) -> "GeluGluSpec":
        return GeluGluSpec(int(f["ff"]))

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff}

    def tensors(self, width: int):
        return [("gate", (self.ff, width)), ("gate.b", (self.ff,)), ("up", (self.ff, width)), ("up.b", (self.ff,)),
                ("down", (width, self.ff)), ("down.b", (width,))]


@dataclass
class GeluSpec:
    """gelu (in its tanh form) between the up and down projections."""
    ff: int
    kind = "gelu"

    @staticmethod
    def from_json(f: dict) -> "GeluSpec":
        return GeluSpec(int(f["ff"]))

    def to_json(self) -> dict:
        return {"kind": "dense", "ff": self.ff}

    def tensors(self, width: int):
        return [("up", (self.ff, width)), ("down", (width, self.ff))]


@dataclass
class SiluGluSpec:
    """silu(gate) up between the gate / up and down projections: the clamped unit without its bounds."""
    ff: int
    kind = "silu_glu"
    limit, alpha, shift = math.inf, 1.0, 0.0

    @staticmethod
    def from_json(f: dict) -> "SiluGluSpec":
        return SiluGluSpec(int(f["ff"]))

    def tensors(self, width: int):
        return [("gate", (self.ff, width)), ("up", (self.ff, width)), ("down", (width, self.ff))]


@dataclass
class RoutedSpec:
    """Mixture of gated experts.  A router's scores (their softmax, or the sigmoid of each) pick ``top`` experts of
    every token, within the ``keep`` groups (of ``groups`` equal ones) whose best expert scores highest.  An expert's
    weight is its score (softmax: over the chosen scores' sum), times ``scale``; it multiplies the expert's output, or
    with ``weigh_input`` its input.  An optional shared expert runs for every token."""
    expert: object
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    shared: Optional[object] = None
    scores: str = "softmax"
    weigh_input: bool = False
    kind = "routed"
    #: added to the sum that the chosen scores are divided by
    tiny = 1e-20

    @staticmethod
    def from_json(f: dict, expert: type = ClampedGluSpec, **constants) -> "RoutedSpec":
        r, sh = f["router"], f.get("shared")
        g = r.get("groups") or {}
        return RoutedSpec(expert.from_json(f["expert"]), int(r["experts"]), int(r["top"]), int(g.get("count", 1)),
                          int(g.get("keep", 1)), float(r.get("scale", 1.0)), expert.from_json(sh) if sh else None, **constants)

    def to_json(self) -> dict:
        size = lambda e: {"ff": e.ff, "limit": e.limit} if e.kind == "clamped_glu" else {"ff": e.ff}
        router = {"experts": self.experts, "top": self.top}
        if self.scores == "softmax":
            router.update(groups={"count": self.groups, "keep": self.keep}, scale=self.scale)
        out = {"kind": "moe", "expert": size(self.expert), "router": router}
        return out if self.shared is None else dict(out, shared=size(self.shared))

    def check(self):
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep <= self.groups:
            raise ValueError(f"routed: {self.experts} experts in {self.groups} groups, {self.keep} of them kept")
        if not 1 <= self.top <= self.experts // self.groups * self.keep:
            raise ValueError(f"routed: {self.top} experts out of {self.experts // self.groups * self.keep}")
        if self.experts > 1024 or self.top > 32:
            raise ValueError("routed: up to 1024 experts, 32 of a token")

    def tensors(self, width: int):
        out = [(f"e{e}.{n}", s) for e in range(self.experts) for n, s in self.expert.tensors(width)]
        out.append(("router", (self.experts, width)))
        return out + ([] if self.shared is None else [("shared." + n, s) for n, s in self.shared.tensors(width)])


@dataclass
class HybridLayer:
    mixer: object                # one of the mixer records above
    mlp: Optional[object] = None


@dataclass(frozen=True)
class MixerForm:
    """A mixer record as a design has it: with some of its constants fixed."""
    spec: type
    constants: tuple = ()

    @property
    def kind(self) -> str:
        return self.spec.kind

    def __call__(self, m: dict):
        return self.spec.from_json(m, **dict(self.constants))


def mixer_form(spec: type, **constants) -> MixerForm:
    return MixerForm(spec, tuple(constants.items()))


@dataclass(frozen=True)
class HybridDesign:
    """What the layers of a design have in common."""
    mixers: tuple                # mixers its layers may name
    mlp: type                    # its dense feed-forward
    routed: Optional[object] = None  # its mixture of experts
    norm_offset: float = 0.0     # norms multiply by this plus the stored gain
    embed_norm: bool = False     # a norm behind the embedding
    positions: bool = False      # a factor on the embedding, and a learned vector per position added to it
    two_norms: bool = False      # the feed-forward reads a norm of its own
    depth_average: bool = False  # what a layer passes on is a weighted sum of all results so far
    tied: bool = False           # the embedding table is the output projection
    residual_mult: bool = False  # a factor on what a layer adds
    streams: bool = False        # several copies of the residual stream: every sublayer (the mixer, then the feed-forward,
                                 # each with a norm of its own) reads a weighted sum of them and is spread over their mixture
    layer_norm: bool = False     # norms subtract the mean and have a bias
    token_shift: bool = False    # a mixer's input is moved towards that of the token before, channel by channel
    loop: bool = False           # a run of layers may be passed several times, with caches and states for each pass
    logit_softcap: bool = False

    @property
    def embed_factor(self) -> bool:
        return self.positions or self.streams


_MATRIX_MEMORY = mixer_form(MlstmSpec)
HYBRID_FAMILY = {
    "Pakalix": HybridDesign((mixer_form(AttentionSpec), mixer_form(Mamba2Spec)), ClampedGluSpec, norm_offset=1.0, embed_norm=True,
                            residual_mult=True),
    "Nezalorn": HybridDesign((mixer_form(LatentAttentionSpec), mixer_form(GeneralDeltaSpec), mixer_form(RgLruSpec)), PolyNormSpec,
                             two_norms=True, depth_average=True, tied=True),
    "Zepesun": HybridDesign((mixer_form(LatentAttentionSpec, interleaved=False, q_latent=False, head_gate=True), _MATRIX_MEMORY,
                             mixer_form(ParallelSpec, left=mixer_form(AttentionSpec, qk_norm=False, bias=True, gate="element"),
                                        right=_MATRIX_MEMORY)),
                            GeluGluSpec, RoutedSpec, positions=True),
    "Povipel": HybridDesign((mixer_form(RetentionSpec),
                             mixer_form(ParallelSpec, normed=True, right=mixer_form(GatedLinearSpec),
                                        left=mixer_form(AttentionSpec, interleaved=True, qk_norm="head", gate=None, sink=True,
                                                        turn_values=True))),
                            GeluSpec, mixer_form(RoutedSpec, expert=SiluGluSpec, scores="sigmoid", weigh_input=True),
                            streams=True, layer_norm=True, token_shift=True, loop=True, logit_softcap=True),
}
#: copies of the residual stream that the kernels hold at once
MAX_STREAMS = 16


@dataclass
class HybridConfig:
    vocab: int
    width: int
    layers: List[HybridLayer]
    eps: float
    residual_mult: float = 1.0
    design: str = "Pakalix"
    #: rows of the table of positions; without one positions are not limited, and this is what a server may
    #: reserve pages for
    max_position_embeddings: int = 131072
    embed_scale: float = 1.0
    streams: int = 1
    #: (first, one past the last, times): layers that run several times in a row
    loop: Optional[tuple] = None
    logit_softcap: Optional[float] = None

    def __post_init__(self):
        if not self.layers:
            raise ValueError("a hybrid decoder needs at least one layer")
        if not 1 <= self.streams <= MAX_STREAMS:
            raise ValueError(f"{self.streams} residual streams: 1 to {MAX_STREAMS}")
        if self.loop is not None:
            a, b, times = self.loop
            if not 0 <= a <= b <= len(self.layers) or times < 1:
                raise ValueError(f"loop: layers {a} to {b} of {len(self.layers)}, {times} times")
        if self.logit_softcap is not None and not self.logit_softcap > 0:
            raise ValueError("the logits' bound is positive")
        vals = set()
        for i, l in enumerate(self.layers):
            m = l.mixer
            m.check()
            if hasattr(l.mlp, "check"):
                l.mlp.check()
            if m.kind == "attention" and m.v_mix:
                vals.add((m.kv_heads, m.vdim))
            if m.kind == "latent_attention" and m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if src is None or src.kind != m.kind or src.kv_from is not None:
                    raise ValueError(f"layer {i}: layer {m.kv_from} has no latents of its own to share")
                if (src.kv_rank, src.rot_dim, src.rot) != (m.kv_rank, m.rot_dim, m.rot):
                    raise ValueError(f"layer {i}: its latents differ in size or rotation from those of layer {m.kv_from}")
        if len(vals) > 1:
            raise ValueError(f"layers that mix values differ in their value sizes: {sorted(vals)}")

    @property
    def traits(self) -> HybridDesign:
        return HYBRID_FAMILY[self.design]

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> List[int]:
        """Which layer runs, pass by pass."""
        n = self.n_layers
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    @property
    def d_model(self) -> int:
        return self.width

    @property
    def block_size(self) -> int:
        return self.max_position_embeddings

    @property
    def recurrent(self) -> bool:
        return self.traits.token_shift or any(l.mixer.recurrent for l in self.layers)

    # ---- JSON: the design's own config file
    def to_json(self) -> dict:
        out = {"architecture": self.design, "vocab": self.vocab, "width": self.width,
               "layers": [{"type": l.mixer.kind, "mixer": l.mixer.to_json(), "mlp": None if l.mlp is None else l.mlp.to_json()}
                          for l in self.layers],
               "norm": {"eps": self.eps}}
        if self.traits.residual_mult:
            out["residual_mult"] = self.residual_mult
        if self.traits.embed_factor:
            out["embedding"] = {"scale": self.embed_scale}
        if self.traits.positions:
            out["max_positions"] = self.max_position_embeddings
        if self.traits.streams:
            out["streams"] = self.streams
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    @staticmethod
    def from_json(c: dict) -> "HybridConfig":
        design = HYBRID_FAMILY[c["architecture"]]
        mixers = {m.kind: m for m in design.mixers}
        read = lambda f: f.from_json if isinstance(f, type) else f
        mlps = {"dense": read(design.mlp), "moe": design.routed and read(design.routed)}
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] not in mixers:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            f = e.get("mlp")
            if f is not None and mlps.get(f.get("kind", "dense")) is None:
                raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
            layers.append(HybridLayer(mixers[e["type"]](e["mixer"]),
                                      None if f is None else mlps[f.get("kind", "dense")](f)))
        more = {}
        if design.embed_factor:
            more["embed_scale"] = float((c.get("embedding") or {}).get("scale", 1.0))
        if design.positions:
            more["max_position_embeddings"] = int(c["max_positions"])
        if design.streams:
            more["streams"] = int(c.get("streams") or 1)
        if design.loop and c.get("loop"):
            more["loop"] = tuple(int(c["loop"][k]) for k in ("start", "stop", "times"))
        if design.logit_softcap and c.get("logit_softcap"):
            more["logit_softcap"] = float(c["logit_softcap"])
        return HybridConfig(vocab=int(c["vocab"]), width=int(c["width"]), layers=layers, eps=float(c["norm"]["eps"]),
                            residual_mult=float(c.get("residual_mult", 1.0)), design=c["architecture"], **more)

    def fill_sizes(self, shapes) -> None:
        """Sizes that the config file leaves to the tensors; ``shapes``: tensor name -> shape."""
        for i, l in enumerate(self.layers):
            if hasattr(l.mixer, "fill"):
                l.mixer.fill(lambda n, p=f"l{i}.mix.": shapes[p + n])

    def tensors(self):
        """(name, shape) of every tensor of a checkpoint, in order."""
        d, t = self.width, self.traits
        norm = lambda n: [(n, (d,)), (n + ".b", (d,))] if t.layer_norm else [(n, (d,))]
        out = [("embed", (self.vocab, d))]
        if t.embed_norm:
            out.append(("embed.norm", (d,)))
        if t.positions:
            out.append(("pos", (self.max_position_embeddings, d)))
        for i, l in enumerate(self.layers):
            out += norm(f"l{i}.norm1")
            if (t.two_norms or t.streams) and l.mlp is not None:
                out += norm(f"l{i}.norm2")
            out += [(f"l{i}.mix.{n}", s) for n, s in l.mixer.tensors(d)]
            if l.mlp is not None:
                out += [(f"l{i}.mlp.{n}", s) for n, s in l.mlp.tensors(d)]
            if t.depth_average:
                out.append((f"l{i}.dwa", (i + 2,)))
            if t.streams:
                n = self.streams
                for q in (1,) if l.mlp is None else (1, 2):
                    out += [(f"l{i}.hc{q}.in", (n,)), (f"l{i}.hc{q}.out", (n,)), (f"l{i}.hc{q}.mix", (n, n))]
            if t.token_shift:
                out.append((f"l{i}.shift", (d,)))
        out += norm("final.norm")
        return out if t.tied else out + [("head", (self.vocab, d))]

    def param_list(self):
        out = []
        for n, s in self.tensors():
            k = 1
            for x in s:
                k *= x
            out.append((n, k))
        return out

    def param_count(self) -> int:
        return sum(n for _, n in self.param_list())


#: architecture name of a config file -> reader of its configuration
HYBRID_DESIGNS = {name: HybridConfig.from_json for name in HYBRID_FAMILY}


def config_from_json(c) -> object:
    """Rebuild the right config record from a checkpoint's ``brain.config`` JSON."""
    if isinstance(c, str):
        c = json.loads(c)
    design = c.get("architecture")
    if design is not None:
        if design not in HYBRID_DESIGNS:
            raise ValueError(f"unknown architecture {design!r}; have {sorted(HYBRID_DESIGNS)}")
        return HYBRID_DESIGNS[design](c)
    kind = c.get("model", "qwen")
    if kind == "gpt":
        return GptConfig.from_json(c)
    if kind in ("moe", "qwen_moe"):
        return MoeConfig.from_json(c)
    return QwenConfig.from_json(c)
