"""Small random layer-stack models for the tests: configurations, weights, and files in a checkpoint's format."""
import json
import os
import struct

import numpy as np


def bf16_bits(a):
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16).reshape(np.shape(a))


def bf16_round(a):
    return (bf16_bits(a).astype(np.uint32) << 16).view(np.float32).reshape(np.shape(a))


def gla(heads, dim, vdim, tau, mlp):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def latent(heads, dim, vdim, rank, scale, mlp, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit=1.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, taps=3, eps=1e-4, mult=0.9):
    return {"architecture": "Zitupel", "canon": {"taps": taps}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab,
            "width": width}


def random_weights(cfg, seed, decay_rank=5, decay_bias=2.0, gain=1.0):
    """Every tensor of a configuration, already rounded to bf16 so that both precisions see the same numbers."""
    rng = np.random.default_rng(seed)
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    w = {}

    def mat(name, rows, cols, s=gain):
        w[name] = rng.standard_normal((rows, cols)) * s / np.sqrt(cols)

    def near_one(name, n):
        w[name] = 1.0 + 0.2 * rng.standard_normal(n)

    def one(name):
        w[name] = np.float64(1.0 + 0.2 * rng.standard_normal())

    w["embed"] = rng.standard_normal((V, W))
    one("embed.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, layer["mixer"], layer["mlp"]
        qk, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        one(p + "norm1")
        w[p + "canon1"] = rng.standard_normal((W, taps)) * 0.4
        mat(p + "mix.q", qk, W)
        mat(p + "mix.o", W, v)
        if layer["type"] == "gla":
            mat(p + "mix.k", qk, W)
            mat(p + "mix.v", v, W)
            mat(p + "mix.g", v, W)
            mat(p + "mix.a1", decay_rank, W)
            mat(p + "mix.a2", qk, decay_rank)
            w[p + "mix.a2.b"] = decay_bias + 0.5 * rng.standard_normal(qk)
            near_one(p + "mix.norm", m["vdim"])
        else:
            mat(p + "mix.uk", qk, m["kv_rank"])
            mat(p + "mix.uv", v, m["kv_rank"])
            if m.get("kv_from") is None:
                mat(p + "mix.dkv", m["kv_rank"], W)
                near_one(p + "mix.dkv.norm", m["kv_rank"])
        if f is None:
            continue
        one(p + "norm2")
        if f["kind"] == "dense":
            mat(p + "mlp.up", f["ff"], W)
            mat(p + "mlp.down", W, f["ff"])
        else:
            mat(p + "mlp.router", f["router"]["experts"], W)
            for e in range(f["router"]["experts"]):
                q = "%smlp.e%d." % (p, e)
                mat(q + "gate", f["expert"]["ff"], W, 1.5)
                mat(q + "up", f["expert"]["ff"], W, 1.5)
                mat(q + "down", W, f["expert"]["ff"], 1.5)
    one("final.norm")
    mat("head", V, W)
    return {k: bf16_round(np.asarray(v, np.float32)) for k, v in w.items()}


class Weights:
    """A dict of arrays under a checkpoint's interface."""

    def __init__(self, arrays):
        self.a = arrays

    def shape(self, name):
        return self.a[name].shape

    def raw(self, name, shape=None):
        a = np.ascontiguousarray(self.a[name], np.float32)
        assert shape is None or a.shape == tuple(shape), (name, a.shape, shape)
        return bf16_bits(a), 1

    def f32(self, name, shape=None):
        a = np.ascontiguousarray(self.a[name], np.float32)
        assert shape is None or a.shape == tuple(shape), (name, a.shape, shape)
        return a

    def scalar(self, name):
        return float(np.asarray(self.a[name]).reshape(-1)[0])


def save(folder, cfg, arrays):
    """config.json and a bf16 model.safetensors."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    table, blobs, at = {}, [], 0
    for name, a in arrays.items():
        b = bf16_bits(a).tobytes()
        table[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    head = json.dumps(table).encode()
    head += b" " * (-len(head) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))


def error(got, want):
    """Root mean square difference per row (mean taken off), relative to the spread of the expected rows."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    scale = np.sqrt(np.mean((want - want.mean(axis=-1, keepdims=True)) ** 2))
    return np.sqrt(np.mean(d * d, axis=-1)) / scale
