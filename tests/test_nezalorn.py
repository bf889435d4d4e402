"""Nezalorn decoders without a GPU: configuration, checkpoints, command line, the packing of weights, and the
tests' own oracle (its mechanisms against closed forms, and mistakes planted in it that the GPU tests' inputs
must make visible)."""
import json
import math
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_util as hu  # noqa: E402
import nezalorn_oracle as oracle  # noqa: E402
import nezalorn_util as nu  # noqa: E402

from brain_b200.checkpoint import st  # noqa: E402
from brain_b200.models import build_from_config  # noqa: E402
from brain_b200.models.config import HybridConfig, RotarySpec, config_from_json  # noqa: E402


def test_config_round_trip_and_registry():
    m, _, cfg = nu.mixed_model()
    again = config_from_json(json.dumps(cfg))
    assert isinstance(again, HybridConfig) and again == m.cfg and again.to_json() == cfg
    assert "residual_mult" not in cfg and "mask" in cfg["layers"][1]["mixer"] and cfg["layers"][3]["mixer"]["kv_from"] == 1
    assert build_from_config(cfg).cfg == m.cfg
    assert m.cfg.recurrent and m.cfg.param_count() == sum(t.numel() for t in m.reference_state().values())
    names = dict(m.cfg.tensors())
    assert "head" not in names and "embed.norm" not in names and names["l3.dwa"] == (5,)
    assert "l3.mix.dkv" not in names and "l2.norm2" not in names and names["l0.mlp.act"] == (4,)
    assert m.flops_per_token(64) < m.flops_per_token(4096) == m.flops_per_token(8192)
    from brain_b200 import arch
    assert arch.by_id("nezalorn").family == "hybrid"


def test_defaults_of_the_config_file():
    cfg = nu.make([(nu.latent(), None)])[2]
    mix = cfg["layers"][0]["mixer"]
    for k in ("mask", "kv_from"):
        mix[k] = None
    mix["rot"]["scaling"] = None
    del cfg["layers"][0]["mlp"]
    spec = config_from_json(cfg).layers[0]
    assert spec.mixer.window is None and spec.mixer.rot.scaling is None and spec.mlp is None


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8),
    lambda c: c["layers"][1]["mixer"].update(mask={"size": -2}),
    lambda c: c["layers"][3]["mixer"].update(kv_from=3),
    lambda c: c["layers"][3]["mixer"].update(kv_from=0),
    lambda c: c["layers"][3]["mixer"].update(kv_rank=40),
    lambda c: c["layers"][3]["mixer"]["rot"].update(base=10.0),
    lambda c: c["layers"][6]["mixer"].update(kv_from=3),
    lambda c: c["layers"][0]["mixer"].update(blocks=7),
    lambda c: c["layers"][0]["mixer"].update(conv=0),
    lambda c: c["layers"][0].update(type="mamba2"),
    lambda c: c["layers"][0]["mlp"].update(kind="routed"),
])
def test_config_errors_are_reported(change):
    cfg = json.loads(json.dumps(nu.mixed_model()[2]))
    change(cfg)
    with pytest.raises(ValueError):
        config_from_json(cfg)


def test_checkpoint_directory_gives_the_sizes_the_config_leaves_out(tmp_path):
    m, _, cfg = nu.mixed_model()
    bare = json.loads(json.dumps(cfg))
    for l in bare["layers"]:
        l["mixer"].pop("decay_rank", None)
        l["mixer"].pop("q_rank", None)
    (tmp_path / "config.json").write_text(json.dumps(bare))
    specs = [(n, s, "BF16") for n, s in m.cfg.tensors()]
    w = st.StWriter(str(tmp_path / "model.safetensors"), specs, {})
    for n, _, _ in specs:
        w.write(n, m.tensor(n))
    w.close()
    from brain_b200.cli.main import main
    out = str(tmp_path / "one.safetensors")
    assert main(["nezalorn", "import", str(tmp_path), "--out", out]) == 0
    for src in (str(tmp_path), out):
        again, _, _ = st.load_model(src)
        assert again.cfg == m.cfg
        for n, t in m.reference_state().items():
            assert torch.equal(again.tensor(n), t), n
    assert main(["nezalorn"]) == 2 and main(["nezalorn", "infer"]) == 2
    bad = dict(m.reference_state())
    del bad["l1.dwa"]
    with pytest.raises(KeyError):
        build_from_config(cfg).load_reference_state(bad)


def test_rotary_frequencies_against_the_oracle():
    for dims in (2, 16, 64):
        for y in (None, nu.YARN):
            f, mag = RotarySpec(dims, 3000.0, y, True).frequencies()
            g, mag2 = oracle.frequencies(dims, 3000.0, None if y is None else vars(y))
            assert np.allclose(f, g, rtol=1e-12) and abs(mag - mag2) < 1e-12
    # fast pairs keep their frequency, slow ones are divided by the factor
    f, mag = oracle.frequencies(64, 3000.0, vars(nu.YARN))
    plain, _ = oracle.frequencies(64, 3000.0, None)
    assert f[0] == plain[0] and abs(f[-1] * 5.0 / plain[-1] - 1) < 1e-9 and abs(mag - (0.1 * math.log(5.0) + 1)) < 1e-12


def test_padded_groups():
    from brain_b200.serve import hybrid_native as hn
    w = torch.arange(2 * 3 * 5, dtype=torch.float32).view(2, 3, 5)
    p = hn.padded_groups(w, 8, 8)
    assert p.shape == (2, 8, 8) and torch.equal(p[:, :3, :5], w) and p.sum() == w.sum()
    assert torch.equal(hn.padded_groups(w, 3, 5), w)


# ------------------------------------------------------------------------------------ the oracle itself
def test_oracle_mechanisms_against_closed_forms():
    rng = np.random.default_rng(1)
    # window: at a row, only the latest keys carry weight, and those as in an ordinary softmax
    s = rng.standard_normal((7, 7))
    p = oracle.window_softmax(s, 3)
    assert np.allclose(p.sum(1), 1) and p[6, 3] == 0 and p[6, 4] > 0 and p[0, 0] == 1 and p[2, 0] > 0
    e = np.exp(s[6, 4:7])
    assert np.allclose(p[6, 4:7], e / e.sum())
    assert np.allclose(oracle.window_softmax(s, 0), oracle.window_softmax(s, 7))
    # rotation: complex multiplication of neighbouring pairs
    x = rng.standard_normal((5, 2, 6))
    r = oracle.rotate_pairs(x, np.arange(5), {"dims": 6, "base": 50.0})
    z = (x[..., 0::2] + 1j * x[..., 1::2]) * np.exp(1j * np.arange(5)[:, None, None] * 50.0 ** (-np.arange(3) / 3))
    assert np.allclose(r[..., 0::2], z.real) and np.allclose(r[..., 1::2], z.imag)
    # delta rule: without decay and with full removal a repeated unit key is overwritten, not added to
    k = np.zeros((2, 1, 4)); k[:, 0, 1] = 1.0
    v = rng.standard_normal((2, 1, 4))
    one = np.ones((2, 1, 4))
    o, S = oracle.delta_rule(k, k, v, one, one)
    assert np.allclose(S[0, 1], v[1, 0], atol=1e-5) and np.allclose(o[1, 0], v[1, 0], atol=1e-5)
    q = rng.standard_normal((6, 2, 4))
    args = [rng.standard_normal((6, 2, 4)) for _ in range(2)] + [rng.random((6, 2, 4)) for _ in range(2)]
    o, S = oracle.delta_rule(q, *args)
    o1, S1 = oracle.delta_rule(q[:2], *(x[:2] for x in args))
    o2, S2 = oracle.delta_rule(q[2:], *(x[2:] for x in args), state0=S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)
    # linear recurrence: constant gates give a geometric sum
    lam = np.array([-1.0]); r = np.full((9, 1), 0.5); u = np.ones((9, 1))
    a = math.exp(-4.0 * math.log1p(math.exp(-1.0)))
    s, last = oracle.linear_recurrence(r, np.ones((9, 1)), u, lam)
    assert np.allclose(last, math.sqrt(1 - a * a) * (1 - a ** 9) / (1 - a)) and np.allclose(s[-1], last)
    u, w, b = rng.standard_normal((9, 3)), rng.standard_normal((3, 4)), rng.standard_normal(3)
    ref = torch.nn.functional.conv1d(torch.tensor(u.T)[None], torch.tensor(w)[:, None], torch.tensor(b), padding=3,
                                     groups=3)[0, :, :9].T.numpy()
    assert np.allclose(oracle.causal_conv(u, w, b), ref)
    g = oracle.block_gates(u[:, :2], np.array([[[2.0]], [[-1.0]]]), np.zeros((2, 1)))
    assert np.allclose(g, oracle.sigmoid(u[:, :2] * [2.0, -1.0]))
    z = torch.randn(5)
    assert np.allclose(oracle.gelu_tanh(z.double().numpy()), torch.nn.functional.gelu(z.double(), approximate="tanh").numpy())
    z = rng.standard_normal((2, 8))
    p = oracle.poly_norm(z, [1.0, 0.0, 0.0, 0.25], 0.0) - 0.25
    assert np.allclose((p ** 2).mean(1), 1) and np.allclose(oracle.poly_norm(z, [0, 0, 1, 0], 0.0), z ** 3 / np.sqrt((z ** 6).mean(1))[:, None])
    assert np.allclose(oracle.depth_average([z, 2 * z, 3 * z], [1.0, 0.5, -1.0]), -z)


def _shift(n):
    return lambda f: lambda s, size: f(s, size + n if size else size)


PLANTED = {
    "window one key short": ("window_softmax", _shift(-1)),
    "window one key long": ("window_softmax", _shift(1)),
    "rotation of half-split pairs": ("rotate_pairs", lambda f: lambda x, p, r: f(
        x.reshape(*x.shape[:-1], 2, -1).swapaxes(-1, -2).reshape(x.shape), p, r)),
    "no yarn": ("frequencies", lambda f: lambda d, b, s: f(d, b, None)),
    "yarn without its factor on cos and sin": ("frequencies", lambda f: lambda d, b, s: (f(d, b, s)[0], 1.0)),
    "removal with the plain key": ("delta_rule", lambda f: lambda r, k, v, w, a, s=None: f(
        r, k, v, w, a * np.sqrt((k * k).sum(-1, keepdims=True)), s)),
    "no decay": ("delta_rule", lambda f: lambda r, k, v, w, a, s=None: f(r, k, v, np.ones_like(w), a, s)),
    "a lost delta state": ("delta_rule", lambda f: lambda r, k, v, w, a: (np.concatenate(
        [f(*(x[:60] for x in (r, k, v, w, a)))[0], f(*(x[60:] for x in (r, k, v, w, a)))[0]]), None)),
    "a lost recurrence state": ("linear_recurrence", lambda f: lambda r, i, u, lam: (np.concatenate(
        [f(r[:60], i[:60], u[:60], lam)[0], f(r[60:], i[60:], u[60:], lam)[0]]), None)),
    "inputs of the recurrence not scaled": ("linear_recurrence", lambda f: lambda r, i, u, lam: f(
        r, i / np.sqrt(1 - np.exp(-16.0 * r * oracle.softplus(lam))), u, lam)),
    "gates from the wrong block": ("block_gates", lambda f: lambda u, w, b: f(u, w[::-1], b)),
    "a lost tap": ("causal_conv", lambda f: lambda u, w, b: f(u, np.concatenate([0 * w[:, :1], w[:, 1:]], 1), b)),
    "no cubic term": ("poly_norm", lambda f: lambda z, c, e: f(z, [c[0], c[1], 0.0, c[3]], e)),
    "the last result alone": ("depth_average", lambda f: lambda x, w: x[-1]),
}


@pytest.mark.parametrize("name", sorted(PLANTED))
def test_planted_mistakes_show(name, monkeypatch):
    """The inputs of the GPU tests (this model, random tokens) turn each mistake into an error well above
    what those tests allow in bf16."""
    _, W, cfg = nu.mixed_model(sharp=3.0)
    toks = hu.tokens(110, 203, 4)
    want = oracle.forward(cfg, W, toks)
    fn, wrap = PLANTED[name]
    monkeypatch.setattr(oracle, fn, wrap(getattr(oracle, fn)))
    assert hu.error(oracle.forward(cfg, W, toks), want) > 1.5 * hu.TOL["bf16"]
