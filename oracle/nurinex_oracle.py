"""Plain numpy restatement of the Nurinex decoder, one function per mechanism, in double precision.

Test infrastructure only: nothing here is used by, or shares code with, the library. Everything is
written for clarity - loops over tokens and heads, no cache, no fusion - and every sequence is
computed from its first token.
"""
import math

import numpy as np


def rms_norm(x, weight=None, eps=1e-6):
    """x / sqrt(mean(x^2) + eps) over the last axis, times an optional weight."""
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def linear(w, x):
    """Rows of x times W^T; w is [out][in]."""
    return x @ w.T


def silu(z):
    return z / (1.0 + np.exp(-z))


def xielu(z, p, q):
    """softplus(p) z^2 + z/2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z/2 below."""
    sp, sq = math.log1p(math.exp(p)), math.log1p(math.exp(q))
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, sp * z * z + 0.5 * z, (0.5 + sq) * (np.expm1(neg) - neg) + 0.5 * z)


def query_temperature(pos, coef, every):
    """Growth of the query with its position: 1 + coef ln(floor((pos + 1) / every) + 1)."""
    return 1.0 + coef * math.log(math.floor((pos + 1) / every) + 1)


def distance_bucket(n, rows, far):
    """Row of the bias table for distance n: the first half of the rows one by one, the others in equal
    steps of ln(n), reaching the last at distance `far`. Evaluated with exact integers:
    floor(ln(n/h) / ln(far/h) m) >= k  <=>  (n/h)^m >= (far/h)^k."""
    half = rows // 2
    if n < half:
        return n
    m = rows - half
    k = 0
    while k + 1 <= m - 1 and n ** m * half ** (k + 1) >= far ** (k + 1) * half ** m:
        k += 1
    return half + k


def softmax_with_sink(scores, sink):
    """Weights of one query row; exp(sink) joins the denominator only."""
    top = max(float(np.max(scores)), float(sink))
    e = np.exp(scores - top)
    return e / (e.sum() + math.exp(sink - top))


def talking_attention(h, w, cfg, eps):
    """Causal attention over all rows of h. w: dict of arrays q, k, v, rel, talk, sink, o."""
    T = h.shape[0]
    H, G, dim, vdim = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = linear(w["q"], h).reshape(T, H, dim).copy()
    k = linear(w["k"], h).reshape(T, G, dim)
    v = rms_norm(linear(w["v"], h).reshape(T, G, vdim), eps=eps)
    temp = cfg["q_temp"]
    for p in range(T):
        q[p] *= query_temperature(p, temp["coef"], temp["every"])
    rows = w["rel"].shape[0]
    bucket = np.array([distance_bucket(n, rows, cfg["bias_max"]) for n in range(T)])
    out = np.zeros((T, H, vdim))
    per = H // G
    for i in range(T):
        raw = np.empty((H, i + 1))
        for g in range(H):
            raw[g] = (k[:i + 1, g // per] @ q[i, g]) * cfg["scale"] + w["rel"][bucket[i - np.arange(i + 1)], g]
        mixed = w["talk"] @ raw
        for g in range(H):
            out[i, g] = softmax_with_sink(mixed[g], w["sink"][g]) @ v[:i + 1, g // per]
    return linear(w["o"], out.reshape(T, H * vdim))


def token_shift(h):
    """The row before each row, zeros before the first."""
    return np.vstack([np.zeros_like(h[:1]), h[:-1]])


def decay(mix_w, w):
    """Per-channel decay in (0, 1): exp(-exp(W2 tanh(W1 m) + w0))."""
    return np.exp(-np.exp(linear(w["w2"], np.tanh(linear(w["w1"], mix_w))) + w["w0"]))


def wkv(r, k, v, d, u, state=None):
    """The recurrence of one head over its rows: reads the state (plus the bonus of the row's own
    outer product), then decays it and adds that product. Returns (outputs, final state)."""
    S = np.zeros((k.shape[1], v.shape[1])) if state is None else state.copy()
    o = np.empty_like(v)
    for t in range(r.shape[0]):
        kv = np.outer(k[t], v[t])
        o[t] = (S + u[:, None] * kv).T @ r[t]
        S = d[t][:, None] * S + kv
    return o, S


def time_mixing(h, w, cfg, eps):
    """Token-shift mixes, decay, recurrence, head norm, gate, output projection."""
    T = h.shape[0]
    H, dim = cfg["heads"], cfg["dim"]
    prev = token_shift(h)
    mix = {s: h + (prev - h) * w["mu." + s] for s in "rkvgw"}
    r, k, v = (linear(w[s], mix[s]).reshape(T, H, dim) for s in "rkv")
    gate = silu(linear(w["g"], mix["g"]))
    d = decay(mix["w"], w).reshape(T, H, dim)
    o = np.empty((T, H, dim))
    for n in range(H):
        o[:, n], _ = wkv(r[:, n], k[:, n], v[:, n], d[:, n], w["u"].reshape(H, dim)[n])
    return linear(w["o"], rms_norm(o, eps=eps).reshape(T, H * dim) * w["norm"] * gate)


def side_by_side(h, w, cfg, eps):
    """Half the sum of the two mixers' outputs, each normed over the model width."""
    def sub(side):
        return {n[len(side) + 1:]: a for n, a in w.items() if n.startswith(side + ".")}
    left = talking_attention(h, sub("left"), cfg["left"], eps)
    right = time_mixing(h, sub("right"), cfg["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def dense(h, w):
    p, q = (float(a) for a in w["act"])
    return linear(w["down"], xielu(linear(w["up"], h), p, q))


def forward(config, tensors, ids, layers_out=None):
    """Logits [n][vocab] of one sequence. tensors: name -> array; layers_out: list that receives the
    residual stream after every layer."""
    W = {n: np.asarray(a, dtype=np.float64) for n, a in tensors.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][np.asarray(ids)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        src = i
        while config["layers"][src].get("weights_of") is not None:
            src = config["layers"][src]["weights_of"]
        pre = f"l{src}."
        h = rms_norm(x, W[pre + "norm1"], eps)
        mix = {n[len(pre) + 4:]: a for n, a in W.items() if n.startswith(pre + "mix.")}
        y = side_by_side(h, mix, layer["mixer"], eps)
        if layer.get("mlp"):
            y = y + dense(h, {n[len(pre) + 4:]: a for n, a in W.items() if n.startswith(pre + "mlp.")})
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return linear(W["head"], rms_norm(x, W["final.norm"], eps))
