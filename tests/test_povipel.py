"""Povipel decoders without a GPU: configuration, checkpoints, command line, and the tests' own oracle (its mechanisms
against closed forms, and mistakes planted in it that the GPU tests' inputs must make visible)."""
import json
import os
import sys

import numpy as np
import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_util as hu  # noqa: E402
import povipel_oracle as oracle  # noqa: E402
import povipel_util as pu  # noqa: E402

from brain_b200.checkpoint import st  # noqa: E402
from brain_b200.models import build_from_config  # noqa: E402
from brain_b200.models.config import HybridConfig, config_from_json  # noqa: E402


def test_config_round_trip_and_registry():
    m, _, cfg = pu.mixed_model()
    again = config_from_json(json.dumps(cfg))
    assert isinstance(again, HybridConfig) and again == m.cfg and again.to_json() == cfg
    assert cfg["embedding"] == {"scale": 2.0} and cfg["streams"] == 3 and cfg["logit_softcap"] == 9.0
    assert cfg["loop"] == {"start": 2, "stop": 4, "times": 2} and m.cfg.runs == [0, 1, 2, 3, 2, 3, 4]
    assert cfg["layers"][0]["mixer"]["left"]["mask"] == {"size": 21, "pool": 6}
    assert cfg["layers"][1]["mlp"] == {"kind": "moe", "expert": {"ff": 40}, "router": {"experts": 10, "top": 2}}
    assert build_from_config(cfg).cfg == m.cfg
    assert m.cfg.recurrent and m.cfg.param_count() == sum(t.numel() for t in m.reference_state().values())
    names = dict(m.cfg.tensors())
    assert names["l0.mix.left.q.norm"] == (40,) and names["l0.mix.left.sink"] == (6,) and "l0.mix.left.g" not in names
    assert names["l0.mix.right.a1"] == (11, 120) and names["l0.mix.right.a2"] == (72, 11) and names["l0.mix.right.norm"] == (40,)
    assert names["l0.mix.left.out"] == (120,) and names["l0.mlp.up"] == (88, 120) and "l0.mlp.gate" not in names
    assert names["l1.hc2.mix"] == (3, 3) and names["l1.shift"] == (120,) and names["l1.norm2.b"] == (120,)
    assert "l3.hc2.in" not in names and "l3.norm2" not in names and names["final.norm.b"] == (120,)
    # a layer's products count once per pass
    once = pu.mixed_model(loop=None)[0]
    assert m.flops_per_token(64) > 1.2 * once.flops_per_token(64)
    from brain_b200 import arch
    assert arch.by_id("povipel").family == "hybrid"


def test_other_designs_have_none_of_it():
    m, _, cfg = hu.make([(hu.mamba(), hu.glu())])
    assert m.cfg.runs == [0] and m.cfg.streams == 1 and not {"streams", "loop", "logit_softcap", "embedding"} & set(cfg)
    assert "l0.shift" not in dict(m.cfg.tensors())


def test_defaults_of_the_config_file():
    cfg = pu.mixed_model()[2]
    for k in ("loop", "streams", "logit_softcap", "embedding"):
        del cfg[k]
    del cfg["layers"][0]["mixer"]["left"]["mask"]
    del cfg["layers"][0]["mixer"]["right"]["decay_rank"]
    c = config_from_json(cfg)
    assert (c.loop, c.streams, c.logit_softcap, c.embed_scale) == (None, 1, None, 1.0)
    left, right = c.layers[0].mixer.left, c.layers[0].mixer.right
    assert left.window is None and left.pool is None and right.decay_rank == 0
    c.fill_sizes({f"l{i}.mix.right.a1": (13, 120) for i in (0, 2, 4)})
    assert right.decay_rank == 13 and c.layers[2].mixer.right.decay_rank == 8


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=-1),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(pool=-2),
    lambda c: c["layers"][0]["mixer"]["left"].update(vdim=23),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=42),
    lambda c: c["layers"][0]["mixer"]["right"].update(tau=0.0),
    lambda c: c["layers"][0]["mixer"]["right"].update(dim=520),
    lambda c: c["layers"][1]["mixer"]["decay"].append(0.5),
    lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 1.5, 0.5]),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][1].update(type="mlstm"),
    lambda c: c["layers"][1]["mlp"].update(kind="routed"),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=11),
    lambda c: c.update(streams=17),
    lambda c: c["loop"].update(stop=6),
    lambda c: c["loop"].update(times=0),
    lambda c: c.update(logit_softcap=-1.0),
])
def test_config_errors_are_reported(change):
    cfg = json.loads(json.dumps(pu.mixed_model()[2]))
    change(cfg)
    with pytest.raises(ValueError):
        config_from_json(cfg)


def test_checkpoint_directory_and_command_line(tmp_path):
    m, _, cfg = pu.mixed_model()
    for layer in cfg["layers"]:
        layer["mixer"].get("right", {}).pop("decay_rank", None)        # the tensors give it
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    specs = [(n, s, "BF16") for n, s in m.cfg.tensors()]
    w = st.StWriter(str(tmp_path / "model.safetensors"), specs, {})
    for n, _, _ in specs:
        w.write(n, m.tensor(n))
    w.close()
    from brain_b200.cli.main import main
    out = str(tmp_path / "one.safetensors")
    assert main(["povipel", "import", str(tmp_path), "--out", out]) == 0
    for src in (str(tmp_path), out):
        again, _, _ = st.load_model(src)
        assert again.cfg == m.cfg
        for n, t in m.reference_state().items():
            assert torch.equal(again.tensor(n), t), n
    assert main(["povipel"]) == 2 and main(["povipel", "infer"]) == 2
    bad = dict(m.reference_state())
    del bad["l1.hc1.mix"]
    with pytest.raises(KeyError):
        build_from_config(pu.mixed_model()[2]).load_reference_state(bad)


def test_first_compilation_has_every_file_of_the_step():
    """Programs that compile on first use build a list of files: every kernel that the hybrid step calls is in one."""
    import re
    from brain_b200 import _build
    step = (_build.CSRC / "serve/hybrid_forward.cu").read_text()
    called = set(re.findall(r"^int (bb_\w+)\(", step, re.M))
    have = {f for t in _build.HYBRID_TUS for f in re.findall(r"BB_API int (bb_\w+)\(", (_build.CSRC / t).read_text())}
    assert called and called <= have


# ------------------------------------------------------------------------------------ the oracle itself
def test_oracle_mechanisms_against_closed_forms():
    rng = np.random.default_rng(1)
    # what a position sees
    assert oracle.seen(0, 3, 2) == ([0], []) and oracle.seen(3, 3, 2) == ([1, 2, 3], [])
    assert oracle.seen(4, 3, 2) == ([2, 3, 4], [0]) and oracle.seen(5, 3, 2) == ([3, 4, 5], [0])
    # equal scores: the mean over everything seen, the sink counted once
    T, P, n = 11, 3, 4
    v = rng.standard_normal((T, 2))
    o = oracle.pooled_window(np.zeros((T, 5)), rng.standard_normal((T, 5)), v, 0.7, n, P, float(np.log(2.0)))
    want = (v[7:11].sum(0) + v[0:3].mean(0) + v[3:6].mean(0)) / (4 + 2 + 2)
    assert np.allclose(o[10], want)
    # rotation: complex multiplication of the pairs; values turned to a position and back again are what they were
    x = rng.standard_normal((5, 2, 6))
    turn = np.exp(1j * np.arange(5)[:, None, None] * 50.0 ** (-np.arange(3) / 3))
    r = oracle.rotate(x, np.arange(5), 6, 50.0, True)
    z = (x[..., ::2] + 1j * x[..., 1::2]) * turn
    assert np.allclose(r[..., ::2], z.real) and np.allclose(r[..., 1::2], z.imag)
    assert np.allclose(oracle.rotate(r, np.arange(5), 6, 50.0, True, back=True), x)
    r = oracle.rotate(x, np.arange(5), 4, 50.0, False)
    z = (x[..., :2] + 1j * x[..., 2:4]) * np.exp(1j * np.arange(5)[:, None, None] * 50.0 ** (-np.arange(2) / 2))
    assert np.allclose(r[..., :2], z.real) and np.allclose(r[..., 2:4], z.imag) and np.allclose(r[..., 4:], x[..., 4:])
    # memory: in two pieces what it is in one; with constant decays a weighted sum over the past
    T, H, D, E = 6, 2, 4, 3
    q, k, v = (rng.standard_normal((T, H, s)) for s in (D, D, E))
    a = rng.uniform(0.3, 1.0, (T, H, D))
    o, S = oracle.decayed_memory(q, k, v, a)
    o1, mid = oracle.decayed_memory(q[:2], k[:2], v[:2], a[:2])
    o2, end = oracle.decayed_memory(q[2:], k[2:], v[2:], a[2:], mid)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(end, S)
    o, _ = oracle.decayed_memory(q, k, v, np.full((T, H, D), 0.7))
    for t in range(T):
        w = 0.7 ** (t - np.arange(t + 1)) * (k[:t + 1, 1] @ q[t, 1])
        assert np.allclose(o[t, 1], w @ v[:t + 1, 1])
    # connections: with the identity and equal parts, every stream is a plain residual stream
    X, y = np.repeat(rng.standard_normal((1, 4, 3)), 2, axis=0), rng.standard_normal((4, 3))
    assert np.allclose(oracle.streams_in(X, np.full(2, 0.5)), X[0])
    assert np.allclose(oracle.streams_out(X, y, np.eye(2), np.ones(2)), X + y)
    moved = oracle.streams_out(X, 0 * y, np.array([[0.0, 2.0], [0.0, 0.0]]), np.ones(2))
    assert np.allclose(moved[0], 0) and np.allclose(moved[1], 2 * X[0])
    h = rng.standard_normal((4, 3))
    s = oracle.token_shift(h, np.array([0.0, 1.0, 0.5]))
    assert np.allclose(s[:, 0], h[:, 0]) and np.allclose(s[1:, 1], h[:-1, 1]) and s[0, 1] == 0 and np.allclose(s[2, 2], h[1:3, 2].mean())
    u = oracle.layer_norm(h, np.ones(3), np.zeros(3), 0.0)
    assert np.allclose(u.mean(1), 0) and np.allclose(u.var(1), 1)
    got = oracle.route(np.array([1.0, -2.0, 3.0, 0.0]), 2)
    assert [e for e, _ in got] == [2, 0] and np.allclose([w for _, w in got], 1 / (1 + np.exp([-3.0, -1.0])))
    z = torch.randn(5).double()
    assert np.allclose(oracle.gelu_tanh(z.numpy()), torch.nn.functional.gelu(z, approximate="tanh").numpy())
    assert oracle.runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 3}}) == [0, 1, 2, 1, 2, 1, 2, 3]


def _window(**change):
    return lambda f: lambda q, k, v, scale, size, pool, sink: f(q, k, v, scale, change.get("size", lambda s: s)(size),
                                                                change.get("pool", lambda p: p)(pool),
                                                                change.get("sink", lambda s: s)(sink))


def _seen(change):
    return lambda f: lambda i, size, pool: change(i, size, pool, *f(i, size, pool))


def _cut(fn, at, q, k, v, a):
    return np.concatenate([fn(q[:at], k[:at], v[:at], a[:at])[0], fn(q[at:], k[at:], v[at:], a[at:])[0]]), None


def _weights(name, value):
    return lambda fn: lambda h, W, *a: fn(h, {n: (value(w) if n.endswith(name) else w) for n, w in W.items()}, *a)


def _recursive(h, s):
    out, before = [], np.zeros(h.shape[1])
    for x in h:
        before = x + (before - x) * s
        out.append(before)
    return out


def _weigh_output(h, W, p, f):
    out = np.zeros_like(h)
    z = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        for e, w in oracle.route(z[t], f["router"]["top"]):
            out[t] += w * oracle.expert(h[t:t + 1], W, p + f"e{e}.")[0]
    return out


PLANTED = {
    "window one key short": ("pooled_window", _window(size=lambda s: s - 1)),
    "window one key long": ("pooled_window", _window(size=lambda s: s + 1)),
    "no pooled blocks": ("seen", _seen(lambda i, s, p, t, b: (t, []))),
    "a block seen a token early": ("seen", _seen(lambda i, s, p, t, b: (t, [x for x in range(i // p + 1) if x * p + p - 1 <= i - s + 1]))),
    "a block seen a token late": ("seen", _seen(lambda i, s, p, t, b: (t, [x for x in b if x * p + p - 1 <= i - s - 1]))),
    "the first block lost": ("seen", _seen(lambda i, s, p, t, b: (t, b[1:]))),
    "no sink": ("pooled_window", _window(sink=lambda s: -1e9)),
    "sink counted twice": ("pooled_window", _window(sink=lambda s: s + np.log(2.0))),
    "rotation of halves in attention": ("rotate", lambda f: lambda x, p, d, b, inter, back=False: f(x, p, d, b, False, back)),
    "rotation of neighbours in retention": ("rotate", lambda f: lambda x, p, d, b, inter, back=False: f(x, p, d, b, True, back)),
    "outputs not turned back": ("rotate", lambda f: lambda x, p, d, b, inter, back=False: x if back else f(x, p, d, b, inter)),
    "no query gain": ("attention", _weights("q.norm", lambda w: 0 * w + 1)),
    "no key gain": ("attention", _weights("k.norm", lambda w: 0 * w + 1)),
    "a lost memory": ("decayed_memory", lambda fn: lambda *x: _cut(fn, 60, *x)),
    "nothing forgotten": ("decayed_memory", lambda fn: lambda q, k, v, a: fn(q, k, v, 0 * a + 1)),
    "decays of the first channel for all": ("decayed_memory", lambda fn: lambda q, k, v, a: fn(q, k, v, 0 * a + a[:, :, :1])),
    "decays without their root": ("gated_linear", lambda fn: lambda h, W, p, m, eps: fn(h, W, p, dict(m, tau=1.0), eps)),
    "no decay bias": ("gated_linear", _weights("a2.b", lambda w: 0 * w)),
    "no head gain": ("gated_linear", _weights("right.norm", lambda w: 0 * w + 1)),
    "sides without norms": ("side_by_side", lambda fn: lambda a, b, W, p, eps: 0.5 * (a * W[p + "left.out"] + b * W[p + "right.out"])),
    "sides added up": ("side_by_side", lambda fn: lambda *x: 2 * fn(*x)),
    "no token shift": ("token_shift", lambda fn: lambda h, s: h),
    "shift of shifted inputs": ("token_shift", lambda fn: lambda h, s: np.stack(_recursive(h, s))),
    "a lost input": ("token_shift", lambda fn: lambda h, s: np.concatenate([fn(h[:60], s), fn(h[60:], s)])),
    "mixture the other way": ("streams_out", lambda fn: lambda X, y, m, w: fn(X, y, m.T, w)),
    "no mixture": ("streams_out", lambda fn: lambda X, y, m, w: fn(X, y, np.eye(len(m)), w)),
    "first stream read": ("streams_in", lambda fn: lambda X, w: X[0]),
    "norm without bias": ("layer_norm", lambda fn: lambda x, w, b, eps: fn(x, w, 0 * b, eps)),
    "norm without mean": ("layer_norm", lambda fn: lambda x, w, b, eps: oracle.rms(x, eps) * w + b),
    "weights on the output": ("moe", lambda fn: _weigh_output),
    "weights renormalised": ("route", lambda fn: lambda z, top: [(e, w / sum(x for _, x in fn(z, top))) for e, w in fn(z, top)]),
    "one expert less": ("route", lambda fn: lambda z, top: fn(z, max(top - 1, 1))),
    "one pass too few": ("runs", lambda fn: lambda c: fn(dict(c, loop=dict(c["loop"], times=1)))),
    "gelu of the other kind": ("gelu_tanh", lambda fn: lambda z: z * oracle.sigmoid(1.702 * z) * 1.02),
}


@pytest.mark.parametrize("name", sorted(PLANTED))
def test_planted_mistakes_show(name, monkeypatch):
    """The inputs of the GPU tests (these models, random tokens) turn each mistake into an error well above what those
    tests allow in fp32, and all but the finest of them into one that they do not take for rounding in bf16."""
    _, W, cfg = pu.mixed_model(sharp=2.0)
    toks = hu.tokens(110, 203, 4)
    want = oracle.forward(cfg, W, toks)
    fn, wrap = PLANTED[name]
    monkeypatch.setattr(oracle, fn, wrap(getattr(oracle, fn)))
    fine = name in ("gelu of the other kind", "a block seen a token early", "a block seen a token late")
    got = oracle.forward(cfg, W, toks)
    assert hu.error(got, want) > 50 * hu.TOL["fp32"] and (fine or not pu.close(got, want, "bf16"))


def test_the_bound_of_the_logits_shows():
    _, W, cfg = pu.mixed_model(spread=6.0)
    toks = hu.tokens(40, 203, 4)
    want = oracle.forward(cfg, W, toks)
    assert np.abs(want).max() > 8.0
    assert hu.error(oracle.forward(dict(cfg, logit_softcap=1e6), W, toks), want) > 0.1


@pytest.mark.parametrize("size,pool", pu.BORDERS)
@pytest.mark.parametrize("name", ["window one key short", "window one key long", "a block seen a token early",
                                  "a block seen a token late", "the first block lost"])
def test_mistakes_at_borders_show(name, size, pool, monkeypatch):
    """... and the loud tokens turn the finest of them into an error far above rounding."""
    if size == 1 and name == "window one key short":
        return                                       # (nothing would be left)
    _, W, cfg, toks = pu.borders_model(size, pool)
    want = oracle.forward(cfg, W, toks)
    fn, wrap = PLANTED[name]
    monkeypatch.setattr(oracle, fn, wrap(getattr(oracle, fn)))
    assert hu.error(oracle.forward(cfg, W, toks), want) > 2 * hu.TOL["bf16"]
