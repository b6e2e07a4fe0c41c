"""Registry of the model designs that load from a folder with config.json and model.safetensors.

A design is a function (ctx, config, checkpoint, options) -> cabi.Decoder registered under the name config.json gives as
"architecture".  It reads the configuration and the tensor names; layers, caches, the step and the loop are the library's.
"""
from __future__ import annotations

import dataclasses
import json
import os

from .. import cabi
from ..checkpoint import Checkpoint

REGISTRY: dict = {}


@dataclasses.dataclass
class LoadOptions:
    dtype: int = cabi.DTYPE_BF16  # element type of matrices and activations
    max_seq_len: int = 2048       # positions of one sequence
    batch: int = 1                # independent sequences
    layers: int | None = None     # only the first layers (inspection)


def register(name: str):
    def add(fn):
        REGISTRY[name] = fn
        return fn

    return add


def read_config(path: str) -> dict:
    with open(os.path.join(path, "config.json")) as f:
        return json.load(f)


def build(ctx, config: dict, weights, options: LoadOptions) -> "cabi.Decoder":
    name = config.get("architecture")
    if name not in REGISTRY:
        raise ValueError("architecture %r is not registered (known: %s)" % (name, ", ".join(sorted(REGISTRY))))
    return REGISTRY[name](ctx, config, weights, options)


def load(ctx, path: str, dtype: str = "bfloat16", max_seq_len: int = 2048, batch: int = 1) -> "cabi.Decoder":
    """A decoder with the weights of a model folder."""
    return build(ctx, read_config(path), Checkpoint(path), LoadOptions(cabi.DTYPES[dtype], max_seq_len, batch))


def matrix(ctx, weights, dtype: int, parts: list, cols: int) -> "cabi.Matrix":
    """A matrix out of a checkpoint: parts [(tensor, rows)] are stacked; a list of such lists gives one group each."""
    groups = parts if isinstance(parts[0], list) else [parts]
    m = cabi.Matrix(ctx, sum(r for _, r in groups[0]), cols, len(groups), dtype)
    for g, rows in enumerate(groups):
        at = 0
        for name, n in rows:
            a, code = weights.raw(name, (n, cols))
            m.put(a, code, row0=at, group=g)
            at += n
    return m


from . import donodra, zitupel  # noqa: E402,F401
