"""Plain restatement of the Nezalorn decoder in numpy, one function per mechanism, token by token and head
by head.  Slow on purpose: no cache, no chunks, no batches, no absorbed products.  It is what the engine is
compared with and shares no code with it."""
import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------ latent attention
def frequencies(dims, base, scaling):
    """(angle per position of every pair, factor on cos and sin)."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if scaling is None:
        return f, 1.0
    s, orig = scaling["factor"], scaling["original"]

    def turns(t):                       # the pair that makes t turns over the original context
        return dims * math.log(orig / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turns(scaling["fast"])), 0)
    hi = min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s * ramp + fi * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(s) + 1.0


def rotate_pairs(x, pos, rot):
    """Rotation of neighbouring entries (2i, 2i + 1) of the last axis; x [T, ..., dims]."""
    f, mag = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    out = x.copy()
    for t in range(x.shape[0]):
        for i, fi in enumerate(f):
            c, s = mag * math.cos(pos[t] * fi), mag * math.sin(pos[t] * fi)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * c - v * s
            out[t, ..., 2 * i + 1] = v * c + u * s
    return out


def window_softmax(s, size):
    """Rows of weights over the ``size`` latest keys, oneself included."""
    out = np.zeros_like(s)
    for i in range(s.shape[0]):
        a = max(0, i - size + 1) if size else 0
        e = np.exp(s[i, a:i + 1] - s[i, a:i + 1].max())
        out[i, a:i + 1] = e / e.sum()
    return out


def latent_attention(h, W, p, m, eps, kept, layer):
    """``kept``: what layers with keys of their own leave behind: layer -> (latents, rotated key parts)."""
    T, H, D, R, E = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = np.arange(T)
    q = (norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).reshape(T, H, D + R)
    if m.get("kv_from") is None:
        ckr = h @ W[p + "dkv"].T
        kept[layer] = (norm(ckr[:, :m["kv_rank"]], W[p + "dkv.norm"], eps),
                       rotate_pairs(ckr[:, m["kv_rank"]:], pos, m["rot"]))
        c, kr = kept[layer]
    else:
        c, kr = kept[m["kv_from"]]
    k = (c @ W[p + "uk"].T).reshape(T, H, D)
    v = (c @ W[p + "uv"].T).reshape(T, H, E)
    qr = rotate_pairs(q[:, :, D:], pos, m["rot"])
    out = np.zeros((T, H, E))
    for i in range(H):
        s = (q[:, i, :D] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        out[:, i] = window_softmax(s, m["mask"]["size"] if m.get("mask") else 0) @ v[:, i]
    return out.reshape(T, H * E) @ W[p + "o"].T


# ------------------------------------------------------------------------------------ generalized delta rule
def delta_rule(r, k, v, w, a, state0=None):
    """r, k, v, w, a [T, H, D] -> outputs [T, H, D] and the last state [H, D(key), D(value)]."""
    T, H, D = r.shape
    S = np.zeros((H, D, D)) if state0 is None else state0.copy()
    o = np.zeros((T, H, D))
    for t in range(T):
        for h in range(H):
            u = k[t, h] / math.sqrt(np.sum(k[t, h] ** 2) + 1e-6)
            old = S[h]
            S[h] = w[t, h][:, None] * old - np.outer(a[t, h] * u, u @ old) + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ r[t, h]
    return o, S


def general_delta(h, W, p, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((h @ W[p + n].T).reshape(T, H, D) for n in "rkv")
    low = np.tanh(h @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"]
    w = np.exp(-math.exp(-0.5) * sigmoid(low)).reshape(T, H, D)
    a = sigmoid(h @ W[p + "a"].T + W[p + "a.b"]).reshape(T, H, D)
    o, _ = delta_rule(r, k, v, w, a)
    return (rms(o, eps).reshape(T, H * D) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------ gated linear recurrence
def causal_conv(u, w, b):
    """out[t, c] = b[c] + sum_k w[c, k] u[t - (taps - 1) + k, c], zeros before the first token."""
    taps = w.shape[1]
    out = np.tile(b[None, :].astype(u.dtype), (u.shape[0], 1))
    for t in range(u.shape[0]):
        for k in range(taps):
            j = t - (taps - 1) + k
            if j >= 0:
                out[t] += w[:, k] * u[j]
    return out


def block_gates(u, w, b):
    """sigmoid of a block-diagonal map; w [blocks, n, n], b [blocks, n]."""
    n = w.shape[1]
    return np.concatenate([sigmoid(u[:, i * n:(i + 1) * n] @ w[i].T + b[i]) for i in range(w.shape[0])], axis=1)


def linear_recurrence(r, i, u, lam, state0=None):
    S = np.zeros(u.shape[1]) if state0 is None else state0.copy()
    out = np.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        a = np.exp(log_a)
        S = a * S + np.sqrt(1.0 - a * a) * i[t] * u[t]
        out[t] = S
    return out, S


def rglru(h, W, p, m):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r = block_gates(u, W[p + "ra"], W[p + "ra.b"])
    i = block_gates(u, W[p + "ri"], W[p + "ri.b"])
    s, _ = linear_recurrence(r, i, u, W[p + "lam"])
    return (s * y) @ W[p + "o"].T


# ------------------------------------------------------------------------------------ the rest
def poly_norm(z, c, eps):
    return c[0] * rms(z, eps) + c[1] * rms(z ** 2, eps) + c[2] * rms(z ** 3, eps) + c[3]


def feed_forward(h, W, p, eps):
    z = h @ W[p + "up"].T + W[p + "up.b"]
    return poly_norm(z, W[p + "act"], eps) @ W[p + "down"].T + W[p + "down.b"]


def depth_average(results, w):
    return sum(float(w[j]) * x for j, x in enumerate(results))


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][np.asarray(tokens)]
    results, kept = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm(x, W[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, W, p + "mix.", m, eps, kept, i)
        elif layer["type"] == "general_delta":
            y = general_delta(h, W, p + "mix.", m, eps)
        else:
            y = rglru(h, W, p + "mix.", m)
        if layer.get("mlp"):
            y = y + feed_forward(norm(x, W[p + "norm2"], eps), W, p + "mlp.", eps)
        results.append(x + y)
        x = depth_average(results, W[p + "dwa"])
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm(x, W["final.norm"], eps) @ W["embed"].T
