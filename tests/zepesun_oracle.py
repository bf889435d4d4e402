"""Plain restatement of the Zepesun decoder in numpy, one function per mechanism, token by token and head by
head.  Slow on purpose: no cache, no chunks, no batches, no absorbed products.  It is what the engine is compared
with and shares no code with it."""
import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def log_sigmoid(x):
    return -np.logaddexp(0.0, -x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def embed(W, tokens, scale):
    T = len(tokens)
    return W["embed"][np.asarray(tokens)] * scale + W["pos"][:T]


# ------------------------------------------------------------------------------------ attention
def softmax_weights(s, window):
    """Rows of weights over the ``window`` latest keys, oneself included (0: every earlier one)."""
    out = np.zeros_like(s)
    for i in range(s.shape[0]):
        a = max(0, i - window + 1) if window else 0
        e = np.exp(s[i, a:i + 1] - s[i, a:i + 1].max())
        out[i, a:i + 1] = e / e.sum()
    return out


def rotate_halves(x, pos, dims, base):
    """Rotation of the pairs (i, i + dims / 2) of the last axis, which is dims long."""
    out = x.copy()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = pos[t] * base ** (-2.0 * i / dims)
            u, v = x[t, ..., i], x[t, ..., i + dims // 2]
            out[t, ..., i] = u * math.cos(a) - v * math.sin(a)
            out[t, ..., i + dims // 2] = v * math.cos(a) + u * math.sin(a)
    return out


def attention(h, W, p, m):
    """Windowed softmax attention with biases and a gate on every output element."""
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = lambda n, heads, size: (h @ W[p + n].T + W[p + n + ".b"]).reshape(T, heads, size)
    q, k, v = proj("q", H, D), proj("k", G, D), proj("v", G, E)
    out = np.zeros((T, H, E))
    for i in range(H):
        g = i // (H // G)
        out[:, i] = softmax_weights(q[:, i] @ k[:, g].T * m["scale"], m["mask"]["size"] if m.get("mask") else 0) @ v[:, g]
    return (out.reshape(T, H * E) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T + W[p + "o.b"]


def latent_attention(h, W, p, m, eps):
    T, H, D, R, E = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos, base = np.arange(T), m["rot"]["base"]
    q = (h @ W[p + "q"].T).reshape(T, H, D + R)
    ckr = h @ W[p + "dkv"].T
    c = norm(ckr[:, :m["kv_rank"]], W[p + "dkv.norm"], eps)
    kr = rotate_halves(ckr[:, m["kv_rank"]:], pos, R, base)
    k, v = (c @ W[p + "uk"].T).reshape(T, H, D), (c @ W[p + "uv"].T).reshape(T, H, E)
    qr = rotate_halves(q[:, :, D:], pos, R, base)
    out = np.zeros((T, H, E))
    for i in range(H):
        out[:, i] = softmax_weights((q[:, i, :D] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"], 0) @ v[:, i]
    out *= sigmoid(h @ W[p + "g"].T)[:, :, None]
    return out.reshape(T, H * E) @ W[p + "o"].T


# ------------------------------------------------------------------------------------ matrix memory
def gates(raw_i, raw_f, cap):
    """(log input gate, log forget gate)."""
    return cap * np.tanh(raw_i / cap), log_sigmoid(cap * np.tanh(raw_f / cap))


def matrix_memory(q, k, v, i, f, state0=None):
    """q, k [T, H, D], v [T, H, E], log gates i, f [T, H] -> outputs [T, H, E] and the last (S, n, m)."""
    T, H, D = q.shape
    S, n, m = (np.zeros((H, D, v.shape[2])), np.zeros((H, D)), np.zeros(H)) if state0 is None else (x.copy() for x in state0)
    o = np.zeros(v.shape)
    for t in range(T):
        for h in range(H):
            new = max(f[t, h] + m[h], i[t, h])
            keep, add = math.exp(f[t, h] + m[h] - new), math.exp(i[t, h] - new)
            S[h] = keep * S[h] + add * np.outer(k[t, h], v[t, h])
            n[h] = keep * n[h] + add * k[t, h]
            m[h] = new
            o[t, h] = S[h].T @ q[t, h] / (max(abs(n[h] @ q[t, h]), math.exp(-new)) + 1e-6)
    return o, (S, n, m)


def mlstm(h, W, p, m, eps):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).reshape(T, H, D) * D ** -0.5
    k, v = (h @ W[p + "k"].T).reshape(T, H, D), (h @ W[p + "v"].T).reshape(T, H, E)
    i, f = gates(h @ W[p + "i"].T + W[p + "i.b"], h @ W[p + "f"].T + W[p + "f.b"], m["gate_cap"])
    o, _ = matrix_memory(q, k, v, i, f)
    return (rms(o, eps).reshape(T, H * E) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def side_by_side(left, right, m):
    return m["left_scale"] * left + m["right_scale"] * right


# ------------------------------------------------------------------------------------ feed-forward
def clamped_glu(h, W, p, limit):
    g = np.minimum(h @ W[p + "gate"].T, limit)
    u = np.clip(h @ W[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def gelu_glu(h, W, p):
    z = gelu_tanh(h @ W[p + "gate"].T + W[p + "gate.b"]) * (h @ W[p + "up"].T + W[p + "up.b"])
    return z @ W[p + "down"].T + W[p + "down.b"]


def route(z, r):
    """Router logits of one token -> [(expert, weight)]."""
    s = np.exp(z - z.max())
    s /= s.sum()
    E, groups = r["experts"], r.get("groups") or {"count": 1, "keep": 1}
    size = E // groups["count"]
    best = [(-s[g * size:(g + 1) * size].max(), g) for g in range(groups["count"])]
    keep = [g for _, g in sorted(best)[:groups["keep"]]]
    allowed = sorted((-s[e], e) for e in range(E) if e // size in keep)
    chosen = [e for _, e in allowed[:r["top"]]]
    total = sum(s[e] for e in chosen) + 1e-20
    return [(e, s[e] / total * r["scale"]) for e in chosen]


def moe(h, W, p, f):
    out = np.zeros_like(h)
    z = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        for e, w in route(z[t], f["router"]):
            out[t] += w * clamped_glu(h[t:t + 1], W, p + f"e{e}.", f["expert"]["limit"])[0]
    if f.get("shared"):
        out += clamped_glu(h, W, p + "shared.", f["shared"]["limit"])
    return out


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = embed(W, tokens, cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = norm(x, W[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, W, p + "mix.", m, eps)
        elif layer["type"] == "mlstm":
            y = mlstm(h, W, p + "mix.", m, eps)
        else:
            y = side_by_side(attention(h, W, p + "mix.left.", m["left"]), mlstm(h, W, p + "mix.right.", m["right"], eps), m)
        if f is not None:
            y = y + (moe(h, W, p + "mlp.", f) if f["kind"] == "moe" else gelu_glu(h, W, p + "mlp."))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm(x, W["final.norm"], eps) @ W["head"].T
