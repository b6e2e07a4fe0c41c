"""Small random Donodra models for the tests: configurations and weights."""
import numpy as np

import stackkit as kit


def attention(heads, kv_heads, dim, vdim, chunk, far, scale, ff):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "bias_max": far, "scale": scale},
            "mlp": ff and kit.dense(ff)}


def delta(heads, kv_heads, dim, vdim, conv, ff):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": ff and kit.dense(ff)}


def mlstm(heads, dim, vdim, cap, ff):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": ff and kit.dense(ff)}


def again(layers, j):
    """One more layer with the tensors of layer j."""
    return dict(layers[j], weights_of=j)


def config(width, vocab, layers, eps=1e-5, alpha=2.0):
    return {"architecture": "Donodra", "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha, "vocab": vocab, "width": width}


def random_weights(cfg, seed, buckets=16, keep=2.0, write=0.0, edit=None):
    """Every tensor of a configuration, already rounded to bf16 so that both precisions see the same numbers.  keep: how slowly the
    recurrent layers forget (log of the odds or of the time, per token); write: bias of the input gates; edit(w) may change tensors."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, rows, cols, s=1.0):
        w[name] = rng.standard_normal((rows, cols)) * s / np.sqrt(cols)

    def near_one(name, n):
        w[name] = 1.0 + 0.2 * rng.standard_normal(n)

    w["embed"] = rng.standard_normal((V, W))
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m, f, kind = "l%d." % i, layer["mixer"], layer["mlp"], layer["type"]
        h, v = m["heads"], m["heads"] * m["vdim"]
        kv = m.get("kv_heads", h)
        near_one(p + "norm1", W)
        mat(p + "mix.q", (h if kind == "attention" else kv) * m["dim"], W)
        mat(p + "mix.k", kv * m["dim"], W)
        mat(p + "mix.v", kv * m["vdim"] if kind == "attention" else v, W, 1.5)
        mat(p + "mix.o", W, v, 1.2)
        if kind == "attention":
            w[p + "mix.rel"] = rng.standard_normal((buckets, h))
            mat(p + "mix.g", h, W)
        else:
            mat(p + "mix.g", v, W)
            near_one(p + "mix.norm", m["vdim"] if kind == "delta" else v)
        if kind == "delta":
            for n, rows in (("q", kv * m["dim"]), ("k", kv * m["dim"]), ("v", v)):
                w[p + "mix.%s.conv" % n] = rng.standard_normal((rows, m["conv"])) * 0.7
            mat(p + "mix.a", h, W)
            mat(p + "mix.b", h, W)
            w[p + "mix.A_log"] = 0.5 * rng.standard_normal(h) - keep
            w[p + "mix.dt_bias"] = 0.5 * rng.standard_normal(h)
        if kind == "mlstm":
            mat(p + "mix.i", h, W)
            mat(p + "mix.f", h, W)
            w[p + "mix.i.b"] = write + 0.3 * rng.standard_normal(h)
            w[p + "mix.f.b"] = keep + 0.3 * rng.standard_normal(h)
        if f is not None:
            near_one(p + "norm2", W)
            mat(p + "mlp.gate", f["ff"], W)
            mat(p + "mlp.up", f["ff"], W, 1.5)
            mat(p + "mlp.down", W, f["ff"], 1.5)
    near_one("final.norm", W)
    if edit:
        edit(w)
    return {k: kit.bf16_round(np.asarray(a, np.float32)) for k, a in w.items()}


def tokens_of(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


def pointing_queries(p, pairs, tokens, boost=1.0):
    """edit: keys read the first half of an embedding, queries the second, and the token at every place q of pairs {q: k} carries the
    first half of the token at k in its second: the query's score for that key is the largest there can be."""
    def edit(w):
        half = w["embed"].shape[1] // 2
        for q, k in pairs.items():
            w["embed"][tokens[q], half:] = w["embed"][tokens[k], :half]
        read = w[p + "mix.k"][:, :half].copy()
        w[p + "mix.k"][:, half:] = 0
        w[p + "mix.q"][:, :half] = 0
        w[p + "mix.q"][:, half:] = read
        w[p + "mix.v"] *= boost
    return edit


# sizes of their own for every mechanism, several that most models make equal or 1, and none that is a multiple of a tile
ATTENTION = config(56, 90, [attention(6, 2, 20, 28, 24, 11, 0.4, None)])
DELTA = config(40, 70, [delta(6, 2, 12, 20, 3, None)])
MLSTM = config(48, 70, [mlstm(3, 20, 28, 5.0, None)])
GATED = config(44, 70, [mlstm(1, 8, 8, 9.0, 100)], alpha=1.0)
SHARED = config(64, 90, [attention(4, 4, 16, 24, 16, 13, 0.5, 48), delta(4, 4, 16, 16, 4, 40), mlstm(2, 16, 24, 8.0, None)], alpha=2.6)
SHARED["layers"] += [again(SHARED["layers"], 0), again(SHARED["layers"], 1), again(SHARED["layers"], 2), again(SHARED["layers"], 0)]
ODD = config(77, 101, [delta(5, 1, 11, 13, 1, 33), attention(9, 1, 13, 11, 37, 50, 0.3, 21), mlstm(1, 37, 9, 2.5, 19), attention(3, 3, 9, 3, 1, 9.5, 1.3, None),
                       delta(3, 3, 37, 70, 16, None)], eps=3e-3, alpha=1.4)
WIDE = config(384, 517, [attention(10, 2, 80, 56, 100, 64, 0.1, 640), delta(4, 2, 96, 160, 4, 136), mlstm(3, 130, 72, 15.0, 200), attention(8, 1, 144, 136, 300, 90, 0.08, None),
                         delta(2, 1, 130, 40, 2, None)], alpha=2.5)
ALL = {"attention": ATTENTION, "delta": DELTA, "mlstm": MLSTM, "gated": GATED, "shared": SHARED, "odd": ODD, "wide": WIDE}
