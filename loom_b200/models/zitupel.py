"""Zitupel: pre-norm layers of gated linear attention or latent attention without positions behind a short convolution,
dense or routed feed-forwards, RMS norms with a single gain, untied head.

`parse` turns config.json and the tensor shapes into layer descriptions (no GPU needed); `build_decoder` uploads the
weights and sets the layers of a stack decoder.
"""
from __future__ import annotations

import dataclasses

import numpy as np

from .. import cabi
from . import LoadOptions, register
from . import matrix as stacked


@dataclasses.dataclass
class Layer:
    spec: dict  # fields of cabi.LayerSpec


@dataclasses.dataclass
class Design:
    width: int
    vocab: int
    norm_eps: float
    residual_mult: float
    conv_taps: int
    layers: list


def parse(config: dict, shape) -> Design:
    """shape(name) -> tuple; sizes that config.json does not name come from the tensors."""
    layers = []
    for i, entry in enumerate(config["layers"]):
        kind, m, f = entry["type"], entry["mixer"], entry.get("mlp")
        p = "l%d.mix." % i
        spec = dict(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_from=-1, tau=1.0, scale=1.0, ffn=cabi.FFN_NONE, ff=0, experts=0, top=0, limit=0.0)
        if kind == "gla":
            spec.update(mixer=cabi.MIXER_GLA, rank=shape(p + "a1")[0], tau=m["tau"])
        elif kind == "latent_attention":
            src = m.get("kv_from")
            spec.update(mixer=cabi.MIXER_LATENT, rank=m["kv_rank"], scale=m["scale"], kv_from=-1 if src is None else src)
        else:
            raise ValueError("layer %d: unknown mixer %r" % (i, kind))
        if f is not None:
            if f["kind"] == "dense":
                spec.update(ffn=cabi.FFN_DENSE, ff=f["ff"])
            elif f["kind"] == "moe":
                spec.update(ffn=cabi.FFN_MOE, ff=f["expert"]["ff"], limit=f["expert"]["limit"], experts=f["router"]["experts"], top=f["router"]["top"])
            else:
                raise ValueError("layer %d: unknown feed-forward %r" % (i, f["kind"]))
        layers.append(Layer(spec))
    return Design(config["width"], config["vocab"], config["norm"]["eps"], config["residual_mult"], config["canon"]["taps"], layers)


def input_projections(spec: dict) -> list:
    """(tensor, rows) of the projections that read the mixer's input, in the order they are stacked."""
    qk, v = spec["heads"] * spec["dim"], spec["heads"] * spec["vdim"]
    if spec["mixer"] == cabi.MIXER_GLA:
        return [("q", qk), ("k", qk), ("v", v), ("g", v), ("a1", spec["rank"])]
    return [("q", qk)] + ([("dkv", spec["rank"])] if spec["kv_from"] < 0 else [])


@register("Zitupel")
def build_decoder(ctx, config: dict, weights, options: LoadOptions) -> "cabi.Decoder":
    d = parse(config, weights.shape)
    dt, W = options.dtype, d.width
    layers = d.layers if options.layers is None else d.layers[:options.layers]
    dec = cabi.Decoder.stack(ctx, len(layers), W, d.vocab, d.norm_eps, d.residual_mult, d.conv_taps, dt, options.max_seq_len)
    dec.set_batch(options.batch)

    def matrix(parts, cols):
        return stacked(ctx, weights, dt, parts, cols)

    for i, layer in enumerate(layers):
        s, p = layer.spec, "l%d." % i
        qk, v = s["heads"] * s["dim"], s["heads"] * s["vdim"]
        w = {"in": matrix([(p + "mix." + n, r) for n, r in input_projections(s)], W), "out": matrix([(p + "mix.o", W)], v),
             "conv_w": weights.f32(p + "canon1", (W, d.conv_taps)), "norm1": weights.scalar(p + "norm1")}
        if s["mixer"] == cabi.MIXER_GLA:
            w.update(mixer_norm=weights.f32(p + "mix.norm", (s["vdim"],)), decay_w=weights.f32(p + "mix.a2", (qk, s["rank"])),
                     decay_b=weights.f32(p + "mix.a2.b", (qk,)))
        else:
            w.update(up_k=matrix([(p + "mix.uk", qk)], s["rank"]), up_v=matrix([(p + "mix.uv", v)], s["rank"]))
            if s["kv_from"] < 0:
                w["mixer_norm"] = weights.f32(p + "mix.dkv.norm", (s["rank"],))
        if s["ffn"] != cabi.FFN_NONE:
            w["norm2"] = weights.scalar(p + "norm2")
        if s["ffn"] == cabi.FFN_DENSE:
            w.update(up=matrix([(p + "mlp.up", s["ff"])], W), down=matrix([(p + "mlp.down", W)], s["ff"]))
        elif s["ffn"] == cabi.FFN_MOE:
            experts = ["%smlp.e%d." % (p, e) for e in range(s["experts"])]
            w.update(router=matrix([(p + "mlp.router", s["experts"])], W), gate=matrix([[(e + "gate", s["ff"])] for e in experts], W),
                     up=matrix([[(e + "up", s["ff"])] for e in experts], W), down=matrix([[(e + "down", W)] for e in experts], s["ff"]))
        dec.set_layer(i, s, w)

    table, code = weights.raw("embed", (d.vocab, W))
    if code != dt:
        table = weights.f32("embed") if dt == cabi.DTYPE_F32 else cabi.to_bf16(table)
    if not hasattr(table, "data_ptr"):  # (already on the device otherwise)
        table = ctx.to_device(np.ascontiguousarray(table))
    dec.set_stack_embeddings(table, weights.scalar("embed.norm"), matrix([("head", d.vocab)], W), weights.scalar("final.norm"))
    return dec
