"""Donodra without a GPU: configuration reader, shared layers, checkpoint names, the oracle's mechanisms against closed forms, and
that a mistake in any mechanism would show in the logits the GPU tests compare."""
import copy
import json

import numpy as np
import pytest

import donodra_oracle as do
import donodrakit as dk
import stackkit as kit
from loom_b200 import cabi, models
from loom_b200.checkpoint import Checkpoint
from loom_b200.models import donodra


def test_parse_reads_every_size():
    cfg = dk.SHARED
    w = dk.random_weights(cfg, 1, buckets=10)
    d = donodra.parse(cfg, kit.Weights(w).shape)
    assert (d.width, d.vocab, d.norm_eps, d.alpha) == (64, 90, 1e-5, 2.6)
    s = [x.spec for x in d.layers]
    assert [x["mixer"] for x in s] == [cabi.MIXER_ATTENTION, cabi.MIXER_DELTA, cabi.MIXER_MLSTM] * 2 + [cabi.MIXER_ATTENTION]
    assert [x.tensors for x in d.layers] == [0, 1, 2, 0, 1, 2, 0]
    assert (s[0]["kv_heads"], s[0]["chunk"], s[0]["buckets"], s[0]["bias_max"], s[0]["scale"]) == (4, 16, 10, 13, 0.5)
    assert (s[1]["conv"], s[2]["gate_cap"]) == (4, 8.0)
    assert [x["ffn"] for x in s[:3]] == [cabi.FFN_GATED, cabi.FFN_GATED, cabi.FFN_NONE]
    for x in d.layers:  # the stacked input projection has the tensors' rows
        for name, rows in donodra.input_projections(x.spec):
            assert w["l%d.mix.%s" % (x.tensors, name)].shape == (rows, 64)
    for x in s:
        cabi.LayerSpec(**x)


def test_shared_layers_follow_their_source():
    entries = [{}, {"weights_of": 0}, {"weights_of": 1}, {"weights_of": 3}, {"weights_of": 9}]
    assert [donodra.tensors_of(entries, i) for i in range(3)] == [0, 0, 0]
    with pytest.raises(ValueError, match="itself"):
        donodra.tensors_of(entries, 3)
    with pytest.raises(ValueError, match="does not exist"):
        donodra.tensors_of(entries, 4)


def test_unknown_mixers_are_refused():
    bad = copy.deepcopy(dk.MLSTM)
    bad["layers"][0]["type"] = "nothing"
    with pytest.raises(ValueError, match="unknown mixer"):
        donodra.parse(bad, lambda name: (1,))
    bad = copy.deepcopy(dk.GATED)
    bad["layers"][0]["mlp"]["kind"] = "nothing"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        donodra.parse(bad, lambda name: (1,))
    assert "Donodra" in models.REGISTRY


def test_checkpoint_holds_what_the_loader_asks_for(tmp_path):
    w = dk.random_weights(dk.SHARED, 2)
    kit.save(str(tmp_path), dk.SHARED, w)
    c = Checkpoint(str(tmp_path))
    assert models.read_config(str(tmp_path)) == json.loads(json.dumps(dk.SHARED))
    d = donodra.parse(dk.SHARED, c.shape)
    for x in d.layers:
        for name, rows in donodra.input_projections(x.spec):
            assert c.raw("l%d.mix.%s" % (x.tensors, name), (rows, 64))[1] == cabi.DTYPE_BF16
    assert not any(n.startswith("l3.") for n in c.table)


# ---- the oracle itself ----


def test_distance_buckets():
    assert [do.distance_bucket(n, 8, 32) for n in (0, 1, 3)] == [0, 1, 3]
    assert [do.distance_bucket(n, 8, 64) for n in (4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    b = [do.distance_bucket(n, 32, 100) for n in range(300)]
    assert b == sorted(b) and b[-1] == 31 and set(b) == set(range(32))


def test_chunked_attention_against_dense_softmax():
    rng = np.random.default_rng(3)
    n, H, G, D, V, chunk = 11, 4, 2, 5, 3, 4
    q, k, v, rel = rng.standard_normal((n, H, D)), rng.standard_normal((n, G, D)), rng.standard_normal((n, G, V)), rng.standard_normal((6, H))
    got = do.chunked_biased_attention(q, k, v, 0.7, rel, 9, chunk)
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = (j <= i) & (i // chunk == j // chunk)
    bucket = np.array([[do.distance_bucket(max(a - b, 0), 6, 9) for b in range(n)] for a in range(n)])
    for h in range(H):
        e = np.where(seen, np.exp(q[:, h] @ k[:, h // 2].T * 0.7 + rel[bucket, h]), 0.0)
        assert np.allclose(got[:, h], e @ v[:, h // 2] / (1.0 + e.sum(axis=1, keepdims=True)))


def test_delta_rule_overwrites_and_equals_its_products():
    rng = np.random.default_rng(4)
    n, D, V = 9, 3, 4
    k = rng.standard_normal((n, 1, D))
    k /= np.linalg.norm(k, axis=-1, keepdims=True)
    k[5] = k[2]  # the same key again: with beta 1 its value is replaced
    q, v = k.copy(), rng.standard_normal((n, 1, V))
    out = do.delta_rule(q, k, v, np.ones((n, 1)), np.ones((n, 1)))
    assert np.allclose(out, v)
    g, b = rng.uniform(0.3, 1.0, (n, 1)), rng.uniform(0.1, 0.9, (n, 1))
    q = rng.standard_normal((n, 1, D))
    S = np.zeros((D, V))
    for t in range(n):  # as one matrix per token
        kt = k[t, 0][:, None]
        S = (np.eye(D) - b[t, 0] * kt @ kt.T) @ (g[t, 0] * S) + b[t, 0] * kt @ v[t, 0][None]
        assert np.allclose(do.delta_rule(q, k, v, g, b)[t, 0], S.T @ q[t, 0])


def test_matrix_memory_without_stabiliser():
    rng = np.random.default_rng(5)
    n, H, D, V = 8, 2, 3, 4
    q, k, v = rng.standard_normal((n, H, D)), rng.standard_normal((n, H, D)), rng.standard_normal((n, H, V))
    i, f = rng.standard_normal((n, H)), -np.abs(rng.standard_normal((n, H)))
    got = do.matrix_memory(q, k, v, i, f)
    for h in range(H):
        m = 0.0
        for t in range(n):
            m = max(f[t, h] + m, i[t, h])
            wt = np.array([np.exp(f[s + 1:t + 1, h].sum() + i[s, h]) * (q[t, h] @ k[s, h]) for s in range(t + 1)])
            den = max(abs(wt.sum()) * np.exp(-m), np.exp(-m)) + 1e-6
            assert np.allclose(got[t, h], np.exp(-m) * wt @ v[:t + 1, h] / den)


# ---- a mistake in any mechanism shows ----


def mutant(name):
    """(configuration, weights, tokens, change): `change` plants one mistake in copies of the configuration and the weights."""
    cfg, w = dk.SHARED, dk.random_weights(dk.SHARED, 6)
    tok = dk.tokens_of(cfg, 40)

    def mixer(i, **kw):
        def change(c, x):
            for layer in c["layers"]:
                if layer["type"] == c["layers"][i]["type"]:
                    layer["mixer"].update(kw)
        return change

    def scaled(suffix, by):
        def change(c, x):
            for n in x:
                if n.endswith(suffix):
                    x[n] = x[n] * by
        return change

    def own_state(c, x):  # the last attention layer with its own, other tensors
        c["layers"] = c["layers"][:-1]

    changes = {"chunk+1": mixer(0, mask={"size": 17}), "chunk-1": mixer(0, mask={"size": 15}), "bias_max": mixer(0, bias_max=20), "scale": mixer(0, scale=0.4),
               "no bias": scaled("mix.rel", 0.0), "cap": mixer(2, gate_cap=1.0), "head gate": scaled("l0.mix.g", 0.0), "conv": scaled("k.conv", -1.0),
               "decay": scaled("A_log", 0.5), "dt_bias": scaled("dt_bias", 0.0), "beta": scaled("mix.b", 0.0), "forget gate": scaled("f.b", 0.5),
               "input gate": scaled("mix.i", 0.0), "memory norm": scaled("l2.mix.norm", -1.0), "final norm": scaled("final.norm", np.linspace(0.5, 1.5, 64)),
               "layer dropped": own_state, "alpha": lambda c, x: c.update(postln_alpha=1.0)}
    return cfg, w, tok, changes[name]


@pytest.mark.parametrize("name", ["chunk+1", "chunk-1", "bias_max", "scale", "no bias", "cap", "head gate", "conv", "decay", "dt_bias", "beta", "forget gate", "input gate",
                                  "memory norm", "final norm", "layer dropped", "alpha"])
def test_a_planted_mistake_shows(name):
    cfg, w, tok, change = mutant(name)
    want, _ = do.forward(cfg, w, tok)
    c, x = copy.deepcopy(cfg), dict(w)
    change(c, x)
    got, _ = do.forward(c, x, tok)
    assert kit.error(got, want).max() > 0.05, "hidden by the random weights"


def test_a_missing_sink_shows():
    rng = np.random.default_rng(7)
    q, k, v, rel = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((4, 2))
    a = do.chunked_biased_attention(q, k, v, 0.5, rel, 8, 5)
    assert np.abs(a[0]).max() < np.abs(v[0]).max()  # even the first token does not get its whole value
