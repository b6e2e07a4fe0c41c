"""Plain float64 recomputation of Donodra, one function per mechanism, on whole sequences with explicit loops.

Nothing is cached, fused or cut into chunks, and no code is shared with the library.  `forward` returns the logits at every
position and the residual stream after every layer.  Weights are a dict of numpy arrays under the names the checkpoint uses.
"""
import math

import numpy as np

from stack_oracle import rms_norm, sigmoid, silu


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def distance_bucket(n, buckets, far):
    """Half of the buckets for one distance each, the other half in equal ratios up to `far`; beyond that the last one."""
    near = buckets // 2
    if n < near:
        return n
    return min(buckets - 1, near + math.floor(math.log(n / near) / math.log(far / near) * (buckets - near)))


def chunked_biased_attention(q, k, v, scale, rel, far, chunk):
    """q [n, heads, dim], k [n, kv_heads, dim], v [n, kv_heads, vdim], rel [buckets, heads].  A query sees the keys of its own
    chunk up to itself; one more weight of exp(0) without a value shares the sum."""
    n, heads, _ = q.shape
    per = heads // k.shape[1]
    bias = np.array([rel[distance_bucket(d, rel.shape[0], far)] for d in range(n)])
    out = np.zeros((n, heads, v.shape[2]))
    for i in range(n):
        lo = i // chunk * chunk
        for h in range(heads):
            g = h // per
            s = k[lo:i + 1, g] @ q[i, h] * scale + bias[i - np.arange(lo, i + 1), h]
            m = max(s.max(), 0.0)
            p = np.exp(s - m)
            out[i, h] = (p / (np.exp(-m) + p.sum())) @ v[lo:i + 1, g]
    return out


def attention_mixer(h, w, p, spec, eps):
    n, heads, kv, dim, vdim = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = rms_norm((h @ w[p + "q"].T).reshape(n, heads, dim), 1.0, eps)
    k = rms_norm((h @ w[p + "k"].T).reshape(n, kv, dim), 1.0, eps)
    v = (h @ w[p + "v"].T).reshape(n, kv, vdim)
    o = chunked_biased_attention(q, k, v, spec["scale"], w[p + "rel"], spec["bias_max"], spec["mask"]["size"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(n, heads * vdim) @ w[p + "o"].T


def short_conv(x, w):
    """Per channel over time, then silu: column taps - 1 of w [channels, taps] belongs to the current token."""
    n, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for t in range(n):
        for j in range(taps):
            if t - (taps - 1) + j >= 0:
                y[t] += w[:, j] * x[t - (taps - 1) + j]
    return silu(y)


def delta_rule(q, k, v, decay, beta):
    """q, k [n, kv_heads, dim], v [n, heads, vdim], decay, beta [n, heads]: the state forgets, what it predicts for k is corrected
    towards v, and the query reads the corrected state."""
    n, heads, vdim = v.shape
    per = heads // k.shape[1]
    S = np.zeros((heads, k.shape[2], vdim))
    out = np.zeros_like(v)
    for t in range(n):
        for h in range(heads):
            kt, qt = k[t, h // per], q[t, h // per]
            S[h] *= decay[t, h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kt)
            S[h] += np.outer(kt, u)
            out[t, h] = S[h].T @ qt
    return out


def delta_mixer(h, w, p, spec, eps):
    n, heads, kv, dim, vdim = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = unit(short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).reshape(n, kv, dim)) / math.sqrt(dim)
    k = unit(short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).reshape(n, kv, dim))
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).reshape(n, heads, vdim)
    beta = sigmoid(h @ w[p + "b"].T)
    decay = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = rms_norm(delta_rule(q, k, v, decay, beta), w[p + "norm"], eps).reshape(n, heads * vdim)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def matrix_memory(q, k, v, i, f):
    """q, k [n, heads, dim], v [n, heads, vdim], log gates i, f [n, heads]; state and normaliser carry the factor exp(-m)."""
    n, heads, dim = q.shape
    out = np.zeros_like(v)
    for h in range(heads):
        S, z, m = np.zeros((dim, v.shape[2])), np.zeros(dim), 0.0
        for t in range(n):
            new = max(f[t, h] + m, i[t, h])
            keep, put = math.exp(f[t, h] + m - new), math.exp(i[t, h] - new)
            S = keep * S + put * np.outer(k[t, h], v[t, h])
            z = keep * z + put * k[t, h]
            m = new
            out[t, h] = S.T @ q[t, h] / (max(abs(z @ q[t, h]), math.exp(-m)) + 1e-6)
    return out


def mlstm_mixer(h, w, p, spec, eps):
    n, heads, dim, vdim, cap = h.shape[0], spec["heads"], spec["dim"], spec["vdim"], spec["gate_cap"]
    q = (h @ w[p + "q"].T).reshape(n, heads, dim) / math.sqrt(dim)
    k = (h @ w[p + "k"].T).reshape(n, heads, dim)
    v = (h @ w[p + "v"].T).reshape(n, heads, vdim)
    i = cap * np.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = -softplus(-cap * np.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o = rms_norm(matrix_memory(q, k, v, i, f), 1.0, eps).reshape(n, heads * vdim) * w[p + "norm"]
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def gated_ffn(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


MIXERS = {"attention": attention_mixer, "delta": delta_mixer, "mlstm": mlstm_mixer}


def forward(cfg, weights, tokens):
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][np.asarray(tokens)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = "l%d." % layer.get("weights_of", i)
        x = rms_norm(alpha * x + MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = rms_norm(alpha * x + gated_ffn(x, w, p + "mlp."), w[p + "norm2"], eps)
        after.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T, after
