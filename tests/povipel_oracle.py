"""Plain restatement of the Povipel decoder in numpy, one function per mechanism, token by token and head by head.
Slow on purpose: no cache, no chunks, no batches.  It is what the engine is compared with and shares no code with it."""
import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def sigmoid(x):
    return np.exp(-np.logaddexp(0.0, -x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def token_shift(h, shift):
    """Every row moved towards the row before it (zeros before the first)."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * shift


def rotate(x, pos, dims, base, interleaved, back=False):
    """Rotation of the first ``dims`` dimensions of x [T, ..., size]: pairs (2i, 2i + 1), or (i, i + dims / 2)."""
    out = x.copy()
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        ang = pos * base ** (-2.0 * i / dims) * (-1.0 if back else 1.0)
        c, s = (f(ang).reshape((-1,) + (1,) * (x.ndim - 2)) for f in (np.cos, np.sin))
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# ------------------------------------------------------------------------------------ mixers
def seen(i, size, pool):
    """(tokens, pooled blocks) that position i attends to."""
    toks = list(range(max(0, i - size + 1) if size else 0, i + 1))
    return toks, [b for b in range(i // pool + 1) if b * pool + pool - 1 <= i - size] if pool else []


def pooled_window(q, k, v, scale, size, pool, sink):
    """One head: q, k [T, D], v [T, E]; a window of tokens, means of the blocks behind it, a sink in the denominator."""
    T, n = q.shape[0], q.shape[0] // pool if pool else 0
    kp, vp = (x[:n * (pool or 1)].reshape(n, pool or 1, x.shape[1]).mean(axis=1) for x in (k, v))
    out = np.zeros((T, v.shape[1]))
    for i in range(T):
        toks, blocks = seen(i, size, pool)
        s = np.concatenate([k[toks], kp[blocks]]) @ q[i] * scale
        top = max(s.max(), sink)
        e = np.exp(s - top)
        out[i] = e @ np.concatenate([v[toks], vp[blocks]]) / (e.sum() + math.exp(sink - top))
    return out


def attention(h, W, p, m, eps):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, rot, mask = np.arange(T), m["rot"], m.get("mask") or {}
    proj = lambda n, heads, size: (h @ W[p + n].T).reshape(T, heads, size)
    q = rotate(rms(proj("q", H, D), eps) * W[p + "q.norm"], pos, rot["dims"], rot["base"], True)
    k = rotate(rms(proj("k", G, D), eps) * W[p + "k.norm"], pos, rot["dims"], rot["base"], True)
    v = rotate(proj("v", G, E), pos, E, rot["base"], True)
    out = np.zeros((T, H, E))
    for i in range(H):
        g = i // (H // G)
        out[:, i] = pooled_window(q[:, i], k[:, g], v[:, g], m["scale"], mask.get("size"), mask.get("pool"), W[p + "sink"][i])
    return rotate(out, pos, E, rot["base"], True, back=True).reshape(T, H * E) @ W[p + "o"].T


def decayed_memory(q, k, v, alpha, S=None):
    """q, k, alpha [T, H, D], v [T, H, E]: S <- diag(alpha) S + k v^T, o = S^T q; outputs and the last S [H, D, E]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if S is None else S.copy()
    o = np.zeros(v.shape)
    for t in range(T):
        for h in range(H):
            S[h] = alpha[t, h][:, None] * S[h] + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def gated_linear(h, W, p, m, eps):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    proj = lambda n, size: (h @ W[p + n].T).reshape(T, H, size)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = np.exp(-np.logaddexp(0.0, -z) / m["tau"]).reshape(T, H, D)
    o, _ = decayed_memory(proj("q", D) * D ** -0.5, proj("k", D), proj("v", E), alpha)
    return ((rms(o, eps) * W[p + "norm"]).reshape(T, H * E) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def side_by_side(left, right, W, p, eps):
    return 0.5 * (rms(left, eps) * W[p + "left.out"] + rms(right, eps) * W[p + "right.out"])


def retention(h, W, p, m, eps):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    proj = lambda n, size: (h @ W[p + n].T).reshape(T, H, size)
    turn = lambda x: rotate(x, np.arange(T), m["rot"]["dims"], m["rot"]["base"], False)
    alpha = np.broadcast_to(np.asarray(m["decay"], dtype=np.float64)[None, :, None], (T, H, D))
    o, _ = decayed_memory(turn(proj("q", D)), turn(proj("k", D)) * D ** -0.5, proj("v", E), alpha)
    return (rms(o, eps).reshape(T, H * E) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------ feed-forward
def dense(h, W, p):
    return gelu_tanh(h @ W[p + "up"].T) @ W[p + "down"].T


def route(z, top):
    """Router logits of one token -> [(expert, weight)]."""
    s = sigmoid(z)
    return [(e, s[e]) for e in sorted(range(len(s)), key=lambda e: (-s[e], e))[:top]]


def expert(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def moe(h, W, p, f):
    out = np.zeros_like(h)
    z = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        for e, w in route(z[t], f["router"]["top"]):
            out[t] += expert(w * h[t:t + 1], W, p + f"e{e}.")[0]
    return out


# ------------------------------------------------------------------------------------ the whole
def streams_in(X, w):
    """X [streams, T, width]."""
    return np.einsum("s,std->td", w, X)


def streams_out(X, y, mix, w):
    return np.einsum("st,snd->tnd", mix, X) + w[:, None, None] * y[None]


def runs(cfg):
    """Layer of every run, in order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the sum of the streams after every layer run."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    X = np.repeat(x[None], cfg["streams"], axis=0)
    for i in runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        m, f = layer["mixer"], layer.get("mlp")
        norm = lambda n, u: layer_norm(u, W[p + n], W[p + n + ".b"], eps)
        h = token_shift(norm("norm1", streams_in(X, W[p + "hc1.in"])), W[p + "shift"])
        if layer["type"] == "parallel":
            y = side_by_side(attention(h, W, p + "mix.left.", m["left"], eps),
                             gated_linear(h, W, p + "mix.right.", m["right"], eps), W, p + "mix.", eps)
        else:
            y = retention(h, W, p + "mix.", m, eps)
        X = streams_out(X, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if f is not None:
            h = norm("norm2", streams_in(X, W[p + "hc2.in"]))
            y = moe(h, W, p + "mlp.", f) if f["kind"] == "moe" else dense(h, W, p + "mlp.")
            X = streams_out(X, y, W[p + "hc2.mix"], W[p + "hc2.out"])
        if layers_out is not None:
            layers_out.append(X.sum(axis=0))
    z = layer_norm(X.sum(axis=0), W["final.norm"], W["final.norm.b"], eps) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(z / cap) if cap else z
