"""Layer stacks without a GPU: configuration and checkpoint readers, the registry, sequence slots, trace replay over a stand-in
decoder, and the oracle's mechanisms against closed forms."""
import json

import numpy as np
import pytest

import stack_oracle as so
import stackkit as kit
from loom_b200 import cabi, models, trace
from loom_b200.checkpoint import Checkpoint
from loom_b200.models import zitupel

CFG = kit.config(24, 50, [kit.gla(2, 8, 12, 4.0, kit.dense(20)), kit.latent(3, 8, 4, 16, 0.3, None), kit.gla(1, 4, 6, 2.0, kit.moe(10, 3, 2)),
                          kit.latent(2, 6, 10, 16, 0.5, kit.dense(8), kv_from=1)], taps=2)


def test_checkpoint_round_trip(tmp_path):
    w = kit.random_weights(CFG, 1)
    kit.save(str(tmp_path), CFG, w)
    c = Checkpoint(str(tmp_path))
    assert set(c.table) == set(w)
    for name in w:
        assert c.shape(name) == w[name].shape
        assert np.array_equal(c.f32(name), w[name])
        bits, code = c.raw(name)
        assert code == cabi.DTYPE_BF16 and np.array_equal(bits, kit.bf16_bits(w[name]))
    assert c.scalar("final.norm") == float(w["final.norm"])
    with pytest.raises(KeyError):
        c.raw("nothing")
    with pytest.raises(ValueError):
        c.raw("head", (3, 3))


def test_truncated_checkpoint_is_refused(tmp_path):
    (tmp_path / "model.safetensors").write_bytes(b"\x40\0\0\0\0\0\0\0{}")
    with pytest.raises(ValueError):
        Checkpoint(str(tmp_path))


def test_parse_reads_every_size():
    w = kit.random_weights(CFG, 1, decay_rank=7)
    d = zitupel.parse(CFG, kit.Weights(w).shape)
    assert (d.width, d.vocab, d.conv_taps, d.norm_eps, d.residual_mult) == (24, 50, 2, 1e-4, 0.9)
    s = [layer.spec for layer in d.layers]
    assert [x["mixer"] for x in s] == [cabi.MIXER_GLA, cabi.MIXER_LATENT, cabi.MIXER_GLA, cabi.MIXER_LATENT]
    assert [x["rank"] for x in s] == [7, 16, 7, 16]
    assert [x["kv_from"] for x in s] == [-1, -1, -1, 1]
    assert [x["ffn"] for x in s] == [cabi.FFN_DENSE, cabi.FFN_NONE, cabi.FFN_MOE, cabi.FFN_DENSE]
    assert (s[2]["experts"], s[2]["top"], s[2]["ff"], s[2]["limit"]) == (3, 2, 10, 1.0)
    for i, x in enumerate(s):  # the stacked input projection has the tensors' rows
        for name, rows in zitupel.input_projections(x):
            assert w["l%d.mix.%s" % (i, name)].shape[0] == rows


def test_unknown_designs_and_mixers_are_refused():
    with pytest.raises(ValueError, match="not registered"):
        models.build(None, {"architecture": "nothing"}, None, models.LoadOptions())
    bad = json.loads(json.dumps(CFG))
    bad["layers"][0]["type"] = "nothing"
    with pytest.raises(ValueError, match="unknown mixer"):
        zitupel.parse(bad, kit.Weights(kit.random_weights(CFG, 1)).shape)


def test_bf16_conversion_matches():
    a = np.random.default_rng(0).standard_normal(1000).astype(np.float32)
    assert np.array_equal(cabi.to_bf16(a), kit.bf16_bits(a))


class CountingDecoder:
    """Logits that spell out the sequence so far: row = (tokens seen, sum of tokens, last token)."""

    def __init__(self, batch):
        self.batch, self.seen, self.lane, self.resets = batch, {}, 0, 0

    def select(self, lane):
        self.lane = lane

    def reset(self):
        self.seen[self.lane] = []
        self.resets += 1

    def extend(self, tokens, want=()):
        s = self.seen[self.lane]
        rows = []
        for t in tokens:
            s.append(t)
            rows.append([len(s), sum(s), t])
        return np.array([rows[w] for w in want], np.float32).reshape(len(want), 3)


def test_trace_replay_keeps_requests_apart(tmp_path):
    dec, said = CountingDecoder(2), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [1], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [9], "want": [0]}, {"id": "b", "tokens": [2, 3], "want": [1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": [4, 4], "want": [1, 0]}], "end": ["b", "c"]}]
    trace.run(dec, [json.dumps(s) for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2", "done 3"]

    def rows(n):
        return np.fromfile(tmp_path / ("%d.f32" % n), "<f4").reshape(-1, 3).tolist()

    assert rows(0) == [[1, 5, 5], [3, 18, 7]]
    assert not (tmp_path / "1.f32").exists()
    assert rows(2) == [[4, 27, 9], [3, 6, 3]]
    assert rows(3) == [[2, 8, 4], [1, 4, 4]]  # the slot of "a", started anew
    assert dec.resets == 3


def test_more_requests_than_sequences_are_refused(tmp_path):
    steps = [{"step": i, "entries": [{"id": str(i), "tokens": [1], "want": []}], "end": []} for i in range(3)]
    with pytest.raises(RuntimeError):
        trace.run(CountingDecoder(2), [json.dumps(s) for s in steps], str(tmp_path), lambda _: None)


# ---- the oracle itself ----


def test_gla_recurrence_equals_its_closed_form():
    rng = np.random.default_rng(2)
    n, h, d, v = 9, 2, 3, 4
    q, k, a = rng.standard_normal((n, h, d)), rng.standard_normal((n, h, d)), rng.uniform(0.3, 1.0, (n, h, d))
    val = rng.standard_normal((n, h, v))
    got = so.gated_linear_attention(q, k, val, a)
    want = np.zeros_like(got)
    for t in range(n):
        for s in range(t + 1):
            for hh in range(h):
                w = np.sum(q[t, hh] * np.prod(a[s + 1:t + 1, hh], axis=0) * k[s, hh])
                want[t, hh] += w * val[s, hh]
    assert np.allclose(got, want)


def test_latents_absorb_into_queries():
    rng = np.random.default_rng(3)
    n, h, d, v, r = 7, 2, 5, 3, 6
    q, c = rng.standard_normal((n, h, d)), rng.standard_normal((n, r))
    uk, uv = rng.standard_normal((h, d, r)), rng.standard_normal((h, v, r))
    got = so.causal_softmax_attention(q, np.einsum("hdr,nr->nhd", uk, c), np.einsum("hvr,nr->nhv", uv, c), 0.7)
    ql = np.einsum("hdr,nhd->nhr", uk, q)
    ol = so.causal_softmax_attention(ql, np.repeat(c[:, None], h, 1), np.repeat(c[:, None], h, 1), 0.7)
    assert np.allclose(got, np.einsum("hvr,nhr->nhv", uv, ol))


def test_convolution_and_routing_by_hand():
    h = np.arange(1.0, 7.0).reshape(3, 2)
    w = np.array([[1.0, 10.0], [2.0, 20.0]])
    assert np.allclose(so.causal_conv(h, w), [[10, 40], [31, 84], [53, 128]])
    idx, score = so.route(np.array([[1.0, 0.0]]), np.array([[0.0, 1.0], [3.0, 0.0], [-1.0, 0.0], [2.0, 0.0]]), 2)
    assert idx.tolist() == [[1, 3]] and np.allclose(score, so.sigmoid(np.array([[3.0, 2.0]])))
