"""Plain restatement of the Pakalix decoder in numpy, one function per mechanism, token by token and
head by head.  Slow on purpose: loops over tokens and heads, no cache, no chunks, no batches.  It is what
the engine is compared with and shares no code with it.

``plant`` makes a known mistake in one mechanism (a dict of switches, see the uses): the tests of the
tests use it to show that their inputs make such a mistake visible."""
import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_plus_one(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def silu(x):
    return x / (1.0 + np.exp(-x))


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


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


def state_space(x, B, C, dt, A_log, D, state0=None):
    """x [T, H, P], B / C [T, G, N], dt [T, H] after softplus; returns y [T, H, P] and the last state
    [H, N, P].  S <- exp(-exp(A_log) dt) S + dt B x^T ;  y = S^T C + D x."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P)) if state0 is None else state0.copy()
    y = np.zeros((T, H, P))
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    """silu(z) first, then a root-mean-square norm of each of ``groups`` equal parts, then the weight."""
    v = y * silu(z)
    T, n = v.shape
    return rms(v.reshape(T, groups, n // groups), eps).reshape(T, n) * w


def mamba2(h, W, p, m, eps):
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    zxbcdt = h @ W[p + "in"].T
    z, xbc, dt = np.split(zxbcdt, [inner, inner + inner + 2 * G * N], axis=1)
    xbc = silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    T = h.shape[0]
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    y, _ = state_space(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"])
    y = gated_group_norm(y.reshape(T, inner), z, W[p + "norm"], m["norm_groups"], eps)
    return y @ W[p + "o"].T


def rotate(x, pos, dims, base):
    """Half-split rotation of the first ``dims`` entries of every head; x [T, heads, D]."""
    out = x.copy()
    half = dims // 2
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def attend(q, k, v, scale, softcap):
    """Causal softmax attention; q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap is not None:
            s = softcap * np.tanh(s / softcap)
        s = np.where(np.tril(np.ones((T, T), dtype=bool)), s, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def attention(h, W, p, m, eps, v_first):
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = norm_plain(h @ W[p + "q"].T, W[p + "q.norm"], eps).reshape(T, H, D)
    k = norm_plain(h @ W[p + "k"].T, W[p + "k.norm"], eps).reshape(T, G, D)
    v = (h @ W[p + "v"].T).reshape(T, G, E)
    if m.get("rot"):
        pos = np.arange(T, dtype=np.float64)
        q = rotate(q, pos, m["rot"]["dims"], m["rot"]["base"])
        k = rotate(k, pos, m["rot"]["dims"], m["rot"]["base"])
    if m.get("v_mix"):
        if v_first is None:
            v_first = v
        else:
            lam = float(np.asarray(W[p + "vmix"]).reshape(()))
            v = (1.0 - lam) * v + lam * v_first
    o = attend(q, k, v, m["scale"], m.get("softcap"))
    o = o * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * E) @ W[p + "o"].T, v_first


def clamped_glu(h, W, p, limit):
    g = np.minimum(h @ W[p + "gate"].T, limit)
    u = np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = norm_plus_one(W["embed"][np.asarray(tokens)], W["embed.norm"], eps)
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = norm_plus_one(x, W[p + "norm1"], eps)
        if layer["type"] == "mamba2":
            y = mamba2(h, W, p + "mix.", layer["mixer"], eps)
        else:
            y, v_first = attention(h, W, p + "mix.", layer["mixer"], eps, v_first)
        if layer.get("mlp"):
            y = y + clamped_glu(h, W, p + "mlp.", layer["mlp"]["limit"])
        x = x + cfg["residual_mult"] * y
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm_plus_one(x, W["final.norm"], eps) @ W["head"].T
