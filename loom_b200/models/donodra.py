"""Donodra: norms after the sum around chunked attention with a learned distance bias and a sink, gated delta rules, or matrix
memories, each followed by a gated feed-forward; layers may use the tensors of another layer with a cache or state of their own;
the head is the embedding table.

`parse` turns config.json and the tensor shapes into layer descriptions (no GPU needed); `build_decoder` uploads the
weights and sets the layers of a stack decoder.
"""
from __future__ import annotations

import dataclasses

import numpy as np

from .. import cabi
from . import LoadOptions, matrix, register


@dataclasses.dataclass
class Layer:
    spec: dict    # fields of cabi.LayerSpec
    tensors: int  # the layer whose tensors this one uses


@dataclasses.dataclass
class Design:
    width: int
    vocab: int
    norm_eps: float
    alpha: float
    layers: list


def tensors_of(entries: list, i: int) -> int:
    """The layer whose tensors layer i uses."""
    seen = set()
    while entries[i].get("weights_of") is not None:
        if i in seen:
            raise ValueError("layer %d: its tensors are those of itself" % i)
        seen.add(i)
        i = entries[i]["weights_of"]
        if not 0 <= i < len(entries):
            raise ValueError("weights of layer %d, which does not exist" % i)
    return i


def parse(config: dict, shape) -> Design:
    """shape(name) -> tuple; sizes that config.json does not name come from the tensors."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        kind, m, f, src = entry["type"], entry["mixer"], entry.get("mlp"), tensors_of(config["layers"], i)
        spec = dict(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_from=-1, ffn=cabi.FFN_NONE)
        if kind == "attention":
            spec.update(mixer=cabi.MIXER_ATTENTION, kv_heads=m["kv_heads"], scale=m["scale"], chunk=m["mask"]["size"],
                        buckets=shape("l%d.mix.rel" % src)[0], bias_max=m["bias_max"], qk_norm=1, sink=1, head_gate=1)
        elif kind == "delta":
            spec.update(mixer=cabi.MIXER_DELTA, kv_heads=m["kv_heads"], conv=m["conv"])
        elif kind == "mlstm":
            spec.update(mixer=cabi.MIXER_MLSTM, gate_cap=m["gate_cap"])
        else:
            raise ValueError("layer %d: unknown mixer %r" % (i, kind))
        if f is not None:
            if f["kind"] != "dense":
                raise ValueError("layer %d: unknown feed-forward %r" % (i, f["kind"]))
            spec.update(ffn=cabi.FFN_GATED, ff=f["ff"])
        layers.append(Layer(spec, src))
    return Design(config["width"], config["vocab"], config["norm"]["eps"], config["postln_alpha"], layers)


def input_projections(s: dict) -> list:
    """(tensor, rows) of the projections that read the mixer's input, in the order they are stacked."""
    h, v = s["heads"], s["heads"] * s["vdim"]
    if s["mixer"] == cabi.MIXER_ATTENTION:
        return [("q", h * s["dim"]), ("k", s["kv_heads"] * s["dim"]), ("v", s["kv_heads"] * s["vdim"]), ("g", h)]
    if s["mixer"] == cabi.MIXER_DELTA:
        qk = s["kv_heads"] * s["dim"]
        return [("q", qk), ("k", qk), ("v", v), ("g", v), ("b", h), ("a", h)]
    return [("q", h * s["dim"]), ("k", h * s["dim"]), ("v", v), ("g", v), ("i", h), ("f", h)]


def layer_weights(ctx, weights, dt: int, W: int, s: dict, p: str) -> dict:
    """The matrices and vectors of the layer whose tensors start with p."""
    h, v = s["heads"], s["heads"] * s["vdim"]
    w = {"in": matrix(ctx, weights, dt, [(p + "mix." + n, r) for n, r in input_projections(s)], W), "out": matrix(ctx, weights, dt, [(p + "mix.o", W)], v),
         "norm1_w": weights.f32(p + "norm1", (W,))}
    if s["mixer"] == cabi.MIXER_ATTENTION:
        w["rel"] = weights.f32(p + "mix.rel", (s["buckets"], h))
    elif s["mixer"] == cabi.MIXER_DELTA:
        qk = s["kv_heads"] * s["dim"]
        w.update(conv_qkv=np.concatenate([weights.f32(p + "mix.%s.conv" % n, (r, s["conv"])) for n, r in (("q", qk), ("k", qk), ("v", v))]),
                 a_log=weights.f32(p + "mix.A_log", (h,)), dt_bias=weights.f32(p + "mix.dt_bias", (h,)), mixer_norm=weights.f32(p + "mix.norm", (s["vdim"],)))
    else:
        w.update(gate_b_i=weights.f32(p + "mix.i.b", (h,)), gate_b_f=weights.f32(p + "mix.f.b", (h,)), mixer_norm=weights.f32(p + "mix.norm", (v,)))
    if s["ffn"] != cabi.FFN_NONE:
        w.update(norm2_w=weights.f32(p + "norm2", (W,)), gate=matrix(ctx, weights, dt, [(p + "mlp.gate", s["ff"])], W),
                 up=matrix(ctx, weights, dt, [(p + "mlp.up", s["ff"])], W), down=matrix(ctx, weights, dt, [(p + "mlp.down", W)], s["ff"]))
    return w


@register("Donodra")
def build_decoder(ctx, config: dict, weights, options: LoadOptions) -> "cabi.Decoder":
    d = parse(config, weights.shape)
    dt, W = options.dtype, d.width
    layers = d.layers if options.layers is None else d.layers[:options.layers]
    dec = cabi.Decoder.stack(ctx, len(layers), W, d.vocab, d.norm_eps, dtype=dt, max_seq_len=options.max_seq_len, residual_alpha=d.alpha)
    dec.set_batch(options.batch)
    loaded: dict = {}
    for i, layer in enumerate(layers):
        if layer.tensors not in loaded:
            loaded[layer.tensors] = layer_weights(ctx, weights, dt, W, layer.spec, "l%d." % layer.tensors)
        dec.set_layer(i, layer.spec, loaded[layer.tensors])
    dec.set_stack_embeddings(None, 1.0, matrix(ctx, weights, dt, [("embed", d.vocab)], W), weights.f32("final.norm", (W,)))
    return dec
