"""Plain numpy restatement of the Zogevik decoder, one function per mechanism, in double precision.

Test infrastructure only: nothing here is used by, or shares code with, the library. Everything is
written for clarity - loops over tokens, heads and experts, no cache, no absorbed products, no fusion -
and every sequence is computed from its first token.
"""
import math

import numpy as np


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis, times the weight."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def linear(w, x):
    """Rows of x times W^T; w is [out][in]."""
    return x @ w.T


def angles(positions, dims, base):
    """[positions][dims / 2]: position times base^(-2i/dims)."""
    return np.outer(np.asarray(positions, dtype=np.float64), base ** (-2.0 * np.arange(dims // 2) / dims))


def rotate_neighbours(x, ang):
    """Elements 2i and 2i+1 of the last axis turn by ang[i]; ang broadcasts over the axes between."""
    y = x.copy()
    c, s = np.cos(ang), np.sin(ang)
    u, v = x[..., 0::2], x[..., 1::2]
    y[..., 0::2] = u * c - v * s
    y[..., 1::2] = v * c + u * s
    return y


def rotate_halves(x, ang):
    """Elements i and i + n of the first 2n turn by ang[i], n = ang's last axis; the others pass."""
    n = ang.shape[-1]
    y = x.copy()
    c, s = np.cos(ang), np.sin(ang)
    u, v = x[..., :n], x[..., n:2 * n]
    y[..., :n] = u * c - v * s
    y[..., n:2 * n] = v * c + u * s
    return y


def visible(i, window):
    """The last `window` positions up to i, i included (None: all of them)."""
    return np.arange(0 if window is None else max(0, i - window + 1), i + 1)


def softmax(scores):
    e = np.exp(scores - scores.max())
    return e / e.sum()


def softmax_plus_one(scores):
    """exp(s_j) / (1 + sum exp(s_j))."""
    top = max(0.0, float(scores.max()))
    e = np.exp(scores - top)
    return e / (math.exp(-top) + e.sum())


def attend(q, k, v, scale, window, weights):
    """q [T][H][a], k [T][G][a], v [T][G][b] -> [T][H * b]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        j = visible(i, window)
        for h in range(H):
            out[i, h] = weights((k[j, h // per] @ q[i, h]) * scale) @ v[j, h // per]
    return out.reshape(T, -1)


def window_of(cfg):
    return cfg["mask"]["size"] if cfg.get("mask") else None


def latent_attention(h, w, cfg, eps):
    """Keys and values out of one normed latent row per position, plus one rotated key part all heads share."""
    T = h.shape[0]
    H, dim, rot, vdim, rank = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    ang = angles(range(T), rot, cfg["rot"]["base"])
    q = linear(w["q"], h).reshape(T, H, dim + rot)
    down = linear(w["dkv"], h)
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    shared = rotate_neighbours(down[:, rank:], ang)
    q = np.concatenate([q[..., :dim], rotate_neighbours(q[..., dim:], ang[:, None])], axis=-1)
    k = linear(w["uk"], c).reshape(T, H, dim)
    k = np.concatenate([k, np.repeat(shared[:, None], H, axis=1)], axis=-1)
    v = linear(w["uv"], c).reshape(T, H, vdim)
    return linear(w["o"], attend(q, k, v, cfg["scale"], window_of(cfg), softmax))


def keys_and_values(h, w, cfg, eps):
    """Normed over the whole projection and rotated keys, and values, as a cache holds them."""
    T = h.shape[0]
    G, dim, vdim, r = cfg["kv_heads"], cfg["dim"], cfg["vdim"], cfg["rot"]
    k = rms_norm(linear(w["k"], h), w["k.norm"], eps).reshape(T, G, dim)
    return rotate_halves(k, angles(range(T), r["dims"], r["base"])[:, None]), linear(w["v"], h).reshape(T, G, vdim)


def attention(h, w, cfg, eps, kv):
    """Grouped-query attention on given keys and values."""
    T = h.shape[0]
    r = cfg["rot"]
    q = rms_norm(linear(w["q"], h), w["q.norm"], eps).reshape(T, cfg["heads"], cfg["dim"])
    q = rotate_halves(q, angles(range(T), r["dims"], r["base"])[:, None])
    return linear(w["o"], attend(q, kv[0], kv[1], cfg["scale"], window_of(cfg), softmax_plus_one))


def gelu_erf(z):
    return 0.5 * z * (1.0 + np.vectorize(math.erf)(z / math.sqrt(2.0)))


def route(z, router):
    """(chosen experts, their weights) of one token from its router logits."""
    E, top = router["experts"], router["top"]
    s = softmax(z)
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = E // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -s[g * size:(g + 1) * size].max())[:groups["keep"]]
    may = [e for g in best for e in range(g * size, (g + 1) * size)]
    chosen = sorted(may, key=lambda e: -s[e])[:top]
    return chosen, s[chosen]


def expert(x, up, down):
    return linear(down, gelu_erf(linear(up, x)))


def experts(h, w, cfg):
    """Weighted sum of the chosen experts' outputs, token by token."""
    z = linear(w["router"], h)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(*route(z[t], cfg["router"])):
            out[t] += s * expert(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    return out


def forward(config, tensors, ids, layers_out=None):
    """Logits [n][vocab] of one sequence. tensors: name -> array; layers_out: list that receives the
    residual stream after every layer."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in tensors.items()}
    eps = config["norm"]["eps"]
    x = rms_norm(W["embed"][np.asarray(ids)], W["embed.norm"], eps)
    stored = {}
    for i, layer in enumerate(config["layers"]):
        def part(kind):
            p = f"l{i}.{kind}."
            return {n[len(p):]: a for n, a in W.items() if n.startswith(p)}
        cfg, w = layer["mixer"], part("mix")
        if layer["type"] == "latent_attention":
            y = latent_attention(x, w, cfg, eps)
        else:
            if cfg.get("kv_from") is None:
                stored[i] = keys_and_values(x, w, cfg, eps)
            y = attention(x, w, cfg, eps, stored[i if cfg.get("kv_from") is None else cfg["kv_from"]])
        x = x + rms_norm(y, W[f"l{i}.norm1"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(experts(x, part("mlp"), layer["mlp"]), W[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return linear(W["head"], rms_norm(x, W["final.norm"], eps))
