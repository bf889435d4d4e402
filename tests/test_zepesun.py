"""Zepesun decoders without a GPU: configuration, checkpoints, command line, and the tests' own oracle (its
mechanisms against closed forms, and mistakes planted in it that the GPU tests' inputs must make visible)."""
import json
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_util as hu  # noqa: E402
import zepesun_oracle as oracle  # noqa: E402
import zepesun_util as zu  # noqa: E402

from brain_b200.checkpoint import st  # noqa: E402
from brain_b200.models import build_from_config  # noqa: E402
from brain_b200.models.config import HybridConfig, config_from_json  # noqa: E402


def test_config_round_trip_and_registry():
    m, _, cfg = zu.mixed_model()
    again = config_from_json(json.dumps(cfg))
    assert isinstance(again, HybridConfig) and again == m.cfg and again.to_json() == cfg
    assert cfg["embedding"] == {"scale": 7.0} and cfg["max_positions"] == 640 and "residual_mult" not in cfg
    assert cfg["layers"][2]["mlp"]["kind"] == "moe" and "shared" not in cfg["layers"][2]["mlp"]
    assert build_from_config(cfg).cfg == m.cfg
    assert m.cfg.recurrent and m.cfg.param_count() == sum(t.numel() for t in m.reference_state().values())
    names = dict(m.cfg.tensors())
    assert names["pos"] == (640, 120) and "embed.norm" not in names and names["head"] == (203, 120)
    assert names["l0.mix.left.q.b"] == (240,) and names["l0.mix.left.g"] == (144, 120) and names["l0.mix.right.i"] == (3, 120)
    assert names["l2.mix.g"] == (5, 120) and "l2.mix.dq" not in names and names["l1.mlp.e11.down"] == (120, 40)
    assert "l2.mlp.shared.up" not in names and not any(n.startswith("l4.mlp") for n in names)
    # only a token's own experts count
    more, _, _ = zu.make([(zu.memory(), zu.moe(experts=24, groups=4))])
    less, _, _ = zu.make([(zu.memory(), zu.moe(experts=12, groups=4))])
    assert more.flops_per_token(64) - less.flops_per_token(64) == 2.0 * 12 * 120       # the router's rows
    from brain_b200 import arch
    assert arch.by_id("zepesun").family == "hybrid"


def test_designs_without_recurrence():
    m, _, _ = zu.make([(zu.latent(), None)])
    assert not m.cfg.recurrent


def test_defaults_of_the_config_file():
    cfg = zu.make([(zu.both(), zu.moe())])[2]
    del cfg["layers"][0]["mixer"]["left"]["mask"]
    f = cfg["layers"][0]["mlp"]
    del f["router"]["groups"], f["router"]["scale"], f["shared"]
    spec = config_from_json(cfg).layers[0]
    assert spec.mixer.left.window is None and (spec.mlp.groups, spec.mlp.keep, spec.mlp.scale, spec.mlp.shared) == (1, 1, 1.0, None)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"]["left"].update(mask={"size": -1}),
    lambda c: c["layers"][0]["mixer"]["left"].update(rot={"dims": 8, "base": 10.0}),
    lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0),
    lambda c: c["layers"][2]["mixer"]["rot"].update(dims=8),
    lambda c: c["layers"][1].update(type="mamba2"),
    lambda c: c["layers"][1]["mlp"].update(kind="routed"),
    lambda c: c["layers"][1]["mlp"]["router"].update(groups={"count": 5, "keep": 2}),
    lambda c: c["layers"][1]["mlp"]["router"].update(groups={"count": 4, "keep": 5}),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7),
])
def test_config_errors_are_reported(change):
    cfg = json.loads(json.dumps(zu.mixed_model()[2]))
    change(cfg)
    with pytest.raises(ValueError):
        config_from_json(cfg)


def test_other_designs_have_no_mixture():
    cfg = hu.make([(hu.mamba(), hu.glu())])[2]
    cfg["layers"][0]["mlp"] = zu.make([(zu.memory(), zu.moe())])[2]["layers"][0]["mlp"]
    with pytest.raises(ValueError):
        config_from_json(cfg)


def test_checkpoint_directory_and_command_line(tmp_path):
    m, _, cfg = zu.mixed_model()
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    specs = [(n, s, "BF16") for n, s in m.cfg.tensors()]
    w = st.StWriter(str(tmp_path / "model.safetensors"), specs, {})
    for n, _, _ in specs:
        w.write(n, m.tensor(n))
    w.close()
    from brain_b200.cli.main import main
    out = str(tmp_path / "one.safetensors")
    assert main(["zepesun", "import", str(tmp_path), "--out", out]) == 0
    for src in (str(tmp_path), out):
        again, _, _ = st.load_model(src)
        assert again.cfg == m.cfg
        for n, t in m.reference_state().items():
            assert torch.equal(again.tensor(n), t), n
    assert main(["zepesun"]) == 2 and main(["zepesun", "infer"]) == 2
    bad = dict(m.reference_state())
    del bad["l1.mlp.e3.up"]
    with pytest.raises(KeyError):
        build_from_config(cfg).load_reference_state(bad)


# ------------------------------------------------------------------------------------ the oracle itself
def test_oracle_mechanisms_against_closed_forms():
    rng = np.random.default_rng(1)
    s = rng.standard_normal((7, 7))
    p = oracle.softmax_weights(s, 3)
    assert np.allclose(p.sum(1), 1) and p[6, 3] == 0 and p[6, 4] > 0 and p[0, 0] == 1 and p[2, 0] > 0
    assert np.allclose(oracle.softmax_weights(s, 0), oracle.softmax_weights(s, 7))
    # rotation: complex multiplication of the two halves
    x = rng.standard_normal((5, 2, 6))
    r = oracle.rotate_halves(x, np.arange(5), 6, 50.0)
    z = (x[..., :3] + 1j * x[..., 3:]) * np.exp(1j * np.arange(5)[:, None, None] * 50.0 ** (-np.arange(3) / 3))
    assert np.allclose(r[..., :3], z.real) and np.allclose(r[..., 3:], z.imag)
    # matrix memory: with open input gates and nothing forgotten it is a sum over the past, over the sum of scores
    T, H, D, E = 6, 2, 4, 3
    q, k, v = rng.random((T, H, D)), rng.random((T, H, D)), rng.standard_normal((T, H, E))
    o, (S, n, m) = oracle.matrix_memory(q, k, v, np.full((T, H), 3.0), np.zeros((T, H)))
    for t in range(T):
        for h in range(H):
            sc = k[:t + 1, h] @ q[t, h]
            assert np.allclose(o[t, h], sc @ v[:t + 1, h] / (max(sc.sum(), np.exp(-3.0)) + 1e-6))
    assert np.allclose(m, 3.0) and np.allclose(n, k.sum(0))
    # ... and in two pieces what it is in one, whatever the gates
    i, f = oracle.gates(4 * rng.standard_normal((T, H)), 4 * rng.standard_normal((T, H)), 2.0)
    assert np.abs(i).max() < 2.0 and f.max() < 0 and f.min() > -2.2
    o, (S, n, m) = oracle.matrix_memory(q, k, v, i, f)
    a, mid = oracle.matrix_memory(q[:2], k[:2], v[:2], i[:2], f[:2])
    b, end = oracle.matrix_memory(q[2:], k[2:], v[2:], i[2:], f[2:], mid)
    assert np.allclose(np.concatenate([a, b]), o) and all(np.allclose(x, y) for x, y in zip(end, (S, n, m)))
    # the stabiliser cancels: the same from plain exponentials (where the floor does not bind)
    w = np.exp(i[:, 0][None] + np.tril(np.cumsum(f[:, 0])[:, None] - np.cumsum(f[:, 0])[None])) * np.tril(np.ones((T, T)))
    sc = w * (q[:, 0] @ k[:, 0].T)
    den = np.maximum(np.abs(sc.sum(1)), 1.0)
    assert np.allclose(o[:, 0], sc @ v[:, 0] / den[:, None], atol=1e-5)
    # routing: the best groups first, then the best of their experts
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}, "scale": 2.0}
    z = np.array([1.0, 0.9, 3.0, -9.0, 2.0, 1.5])
    got = dict(oracle.route(z, r))
    assert sorted(got) == [2, 3] and abs(sum(got.values()) - 2.0) < 1e-9 and abs(got[2] / got[3] - np.exp(12.0)) < 1e-3 * np.exp(12.0)
    assert sorted(dict(oracle.route(z, dict(r, groups={"count": 3, "keep": 2})))) == [2, 4]
    assert sorted(dict(oracle.route(z, dict(r, groups=None, top=3)))) == [2, 4, 5]
    z = torch.randn(5)
    assert np.allclose(oracle.gelu_tanh(z.double().numpy()), torch.nn.functional.gelu(z.double(), approximate="tanh").numpy())


def _memory(change):
    return lambda fn: lambda q, k, v, i, f, s=None: change(fn, q, k, v, i, f)


def _cut(fn, at, *x):
    return np.concatenate([fn(*(y[:at] for y in x))[0], fn(*(y[at:] for y in x))[0]]), None


def _no_bias(name):
    return lambda fn: lambda h, W, *a: fn(h, {n: (0 * w if n.endswith(name) else w) for n, w in W.items()}, *a)


def _no_floor(fn, q, k, v, i, f):
    o, _ = fn(q, k, v, i, f)
    out = np.zeros_like(o)
    for h in range(q.shape[1]):
        F = np.cumsum(f[:, h])
        w = np.where(np.tril(np.ones((len(F),) * 2)) > 0, np.exp(np.minimum(i[:, h][None] + F[:, None] - F[None], 50)), 0)
        sc = w * (q[:, h] @ k[:, h].T)
        out[:, h] = sc @ v[:, h] / (np.abs(sc.sum(1))[:, None] + 1e-6)
    return out, None


PLANTED = {
    "window one key short": ("softmax_weights", lambda f: lambda s, n: f(s, n - 1 if n else 0)),
    "window one key long": ("softmax_weights", lambda f: lambda s, n: f(s, n + 1 if n else 0)),
    "rotation of neighbouring pairs": ("rotate_halves", lambda f: lambda x, p, d, b: f(
        x.reshape(*x.shape[:-1], -1, 2).swapaxes(-1, -2).reshape(x.shape), p, d, b)),
    "a lost memory": ("matrix_memory", _memory(lambda fn, *x: _cut(fn, 60, *x))),
    "nothing forgotten": ("matrix_memory", _memory(lambda fn, q, k, v, i, f: fn(q, k, v, i, 0 * f))),
    "input gate left out": ("matrix_memory", _memory(lambda fn, q, k, v, i, f: fn(q, k, v, 0 * i, f))),
    "no floor under the normaliser": ("matrix_memory", _memory(_no_floor)),
    "gates without their bound": ("gates", lambda fn: lambda i, f, cap: fn(i, f, 1e6)),
    "no gate bias": ("mlstm", _no_bias("f.b")),
    "no query bias": ("attention", _no_bias("q.b")),
    "no value bias": ("attention", _no_bias("v.b")),
    "no output bias": ("attention", _no_bias("o.b")),
    "gates of attention half open": ("attention", _no_bias("left.g")),
    "head gates half open": ("latent_attention", _no_bias("mix.g")),
    "both sides with one factor": ("side_by_side", lambda fn: lambda a, b, m: fn(a, b, dict(m, left_scale=1.0, right_scale=1.0))),
    "feed-forward without biases": ("gelu_glu", _no_bias(".b")),
    "no clamp": ("clamped_glu", lambda fn: lambda h, W, p, limit: fn(h, W, p, 1e9)),
    "groups ignored": ("route", lambda fn: lambda z, r: fn(z, dict(r, groups=None))),
    "router's factor left out": ("route", lambda fn: lambda z, r: fn(z, dict(r, scale=1.0))),
    "one expert less": ("route", lambda fn: lambda z, r: fn(z, r)[:-1] if r["top"] > 1 else fn(z, r)),
    "positions one off": ("embed", lambda fn: lambda W, t, s: fn(dict(W, pos=W["pos"][1:]), t, s)),
    "embedding without its factor": ("embed", lambda fn: lambda W, t, s: fn(W, t, 1.0)),
}


@pytest.mark.parametrize("name", sorted(PLANTED))
def test_planted_mistakes_show(name, monkeypatch):
    """The inputs of the GPU tests (these models, random tokens) turn each mistake into an error well above what
    those tests allow in bf16."""
    _, W, cfg = zu.mixed_model(sharp=3.0, eps=0.02 if "norm" in name else 3e-6)
    toks = hu.tokens(110, 203, 4)
    want = oracle.forward(cfg, W, toks)
    fn, wrap = PLANTED[name]
    monkeypatch.setattr(oracle, fn, wrap(getattr(oracle, fn)))
    assert hu.error(oracle.forward(cfg, W, toks), want) > 1.5 * hu.TOL["bf16"]
