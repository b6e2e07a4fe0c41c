"""Plain float64 recomputation of the layer-stack decoders, one function per mechanism.

Everything here works on whole sequences with explicit loops or dense matrices; nothing is cached, fused or chunked,
and no code is shared with the library.  `forward` returns the logits at every position and the residual stream after
every layer.  Weights are a dict of numpy arrays under the names the checkpoint uses.
"""
import math

import numpy as np


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + np.vectorize(math.erf)(z / math.sqrt(2.0)))


def rms_norm(x, gain, eps):
    """Rows divided by their root mean square, times a gain (a number or a vector)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def causal_conv(h, w):
    """Depthwise over time: out[t] = sum_j w[:, j] h[t - taps + 1 + j], zero before the start.  w is [width, taps]."""
    n, taps = h.shape[0], w.shape[1]
    out = np.zeros_like(h)
    for t in range(n):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def decay(h, a1, a2, bias, tau):
    """Per-channel decay in (0, 1): the tau-th root of a sigmoid of a low-rank projection."""
    z = (h @ a1.T) @ a2.T + bias
    log_sigmoid = np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))
    return np.exp(log_sigmoid / tau)


def gated_linear_attention(q, k, v, alpha):
    """q, k, alpha [n, heads, dim]; v [n, heads, vdim].  The decay scales the rows of the state (key channels)."""
    n, heads, dim = q.shape
    state = np.zeros((heads, dim, v.shape[2]))
    out = np.zeros((n, heads, v.shape[2]))
    for t in range(n):
        for h in range(heads):
            state[h] = alpha[t, h][:, None] * state[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = state[h].T @ q[t, h]
    return out


def gla_mixer(h, w, p, spec, eps):
    heads, dim, vdim = spec["heads"], spec["dim"], spec["vdim"]
    n = h.shape[0]
    q = (h @ w[p + "q"].T).reshape(n, heads, dim) / math.sqrt(dim)
    k = (h @ w[p + "k"].T).reshape(n, heads, dim)
    v = (h @ w[p + "v"].T).reshape(n, heads, vdim)
    alpha = decay(h, w[p + "a1"], w[p + "a2"], w[p + "a2.b"], spec["tau"]).reshape(n, heads, dim)
    o = rms_norm(gated_linear_attention(q, k, v, alpha), w[p + "norm"], eps)
    return (o.reshape(n, heads * vdim) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_softmax_attention(q, k, v, scale):
    """q, k [n, heads, dim]; v [n, heads, vdim]."""
    n, heads, _ = q.shape
    out = np.zeros((n, heads, v.shape[2]))
    mask = np.tril(np.ones((n, n), bool))
    for h in range(heads):
        s = np.where(mask, (q[:, h] @ k[:, h].T) * scale, -np.inf)
        s = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (s / s.sum(axis=1, keepdims=True)) @ v[:, h]
    return out


def latent_of(h, w, p, eps):
    return rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)


def latent_mixer(h, latent, w, p, spec):
    heads, dim, vdim = spec["heads"], spec["dim"], spec["vdim"]
    n = h.shape[0]
    q = (h @ w[p + "q"].T).reshape(n, heads, dim)
    k = (latent @ w[p + "uk"].T).reshape(n, heads, dim)
    v = (latent @ w[p + "uv"].T).reshape(n, heads, vdim)
    return causal_softmax_attention(q, k, v, spec["scale"]).reshape(n, heads * vdim) @ w[p + "o"].T


def dense_ffn(h, w, p):
    return gelu_erf(h @ w[p + "up"].T) @ w[p + "down"].T


def expert(x, w, p, limit):
    g = np.minimum(x @ w[p + "gate"].T, limit)
    u = np.clip(x @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(h, router, top):
    """Chosen experts and their scores (sigmoid, not renormalised) for every row."""
    s = sigmoid(h @ router.T)
    idx = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return idx, np.take_along_axis(s, idx, axis=1)


def moe_ffn(h, w, p, spec):
    idx, score = route(h, w[p + "router"], spec["router"]["top"])
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            e = "%se%d." % (p, idx[t, j])
            out[t] += expert(score[t, j] * h[t:t + 1], w, e, spec["expert"]["limit"])[0]
    return out


def forward(cfg, weights, tokens):
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = rms_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
    latents, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, spec = "l%d." % i, layer["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        h = h + causal_conv(h, w[p + "canon1"])
        if layer["type"] == "gla":
            y = gla_mixer(h, w, p + "mix.", spec, eps)
        else:
            src = spec.get("kv_from")
            if src is None:
                latents[i] = latent_of(h, w, p + "mix.", eps)
            y = latent_mixer(h, latents[i if src is None else src], w, p + "mix.", spec)
        x = x + m * y
        if layer["mlp"] is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            f = dense_ffn(h, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else moe_ffn(h, w, p + "mlp.", layer["mlp"])
            x = x + m * f
        after.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T, after
