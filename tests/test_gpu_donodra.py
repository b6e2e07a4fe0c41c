"""Donodra on the GPU against its plain oracle (`donodra_oracle.py`): every mechanism alone and together, in float32 and in bf16, as
whole prompts, portions, single tokens, several sequences, reused slots, and through the generation entry points.

float32 is held to 2e-5 of the logits' spread (what float32 sums of this length cost), bf16 to two per cent (two roundings of 2^-9
per product through a handful of layers).
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import donodra_oracle as do
import donodrakit as dk
import loom_b200
import stackkit as kit
from loom_b200 import cabi, models

pytestmark = pytest.mark.gpu
F32, BF16 = cabi.DTYPE_F32, cabi.DTYPE_BF16
TOL = {F32: 2e-5, BF16: 0.02}
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
both = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def close(dtype, got, want):
    """Rounding costs little at almost every position (a normed head output near zero magnifies it at a few)."""
    e = kit.error(got, want)
    return np.quantile(e, 0.9) < TOL[dtype] and e.max() < 5 * TOL[dtype]


@pytest.fixture(scope="module")
def ctx():
    c = loom_b200.Context(0)
    yield c
    c.close()


class Model:
    def __init__(self, ctx, cfg, seed, dtype, max_seq=512, batch=1, layers=None, **kw):
        self.cfg, self.w = cfg, dk.random_weights(cfg, seed, **kw)
        self.dec = models.build(ctx, cfg, kit.Weights(self.w), models.LoadOptions(dtype, max_seq, batch, layers))

    def oracle(self, tokens):
        return do.forward(self.cfg, self.w, tokens)

    def whole(self, tokens):
        self.dec.reset()
        return self.dec.extend(tokens, range(len(tokens)))

    def cut(self, tokens, sizes):
        """The logits of every position, the prompt cut into portions of these sizes (the last one repeats)."""
        self.dec.reset()
        out, at, i = [], 0, 0
        while at < len(tokens):
            n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
            out.append(self.dec.extend(tokens[at:at + n], range(n)))
            at, i = at + n, i + 1
        return np.concatenate(out)

    def close(self):
        self.dec.close()


@both
@pytest.mark.parametrize("name", sorted(dk.ALL))
def test_prompt_portions_and_decoding_match_the_oracle(ctx, name, dtype):
    cfg = dk.ALL[name]
    m = Model(ctx, cfg, 3, dtype)
    tok = dk.tokens_of(cfg, 61)
    want, after = m.oracle(tok)
    assert close(dtype, m.whole(tok), want)
    assert close(dtype, m.dec.last_residual(64), after[-1])
    for sizes in ([1], [2], [3, 17, 2, 1], [40, 1], [9, 10]):
        assert close(dtype, m.cut(tok, sizes), want), sizes
    m.close()


@both
def test_residual_stream_layer_by_layer(ctx, dtype):
    cfg = dk.SHARED
    tok = dk.tokens_of(cfg, 45, 1)
    for n in range(1, len(cfg["layers"]) + 1):
        m = Model(ctx, cfg, 4, dtype, layers=n)
        after = m.oracle(tok)[1]
        rows = []
        m.dec.reset()
        for lo, hi in ((0, 30), (30, 31), (31, 33), (33, 34), (34, 45)):
            m.dec.extend(tok[lo:hi])
            rows.append(m.dec.last_residual(64))
        assert close(dtype, np.concatenate(rows), after[n - 1]), n
        m.close()


@both
def test_long_sequences_cross_every_block_border(ctx, dtype):
    cfg = dk.WIDE
    m = Model(ctx, cfg, 5, dtype, max_seq=640)
    tok = dk.tokens_of(cfg, 460, 1)
    want, _ = m.oracle(tok)
    assert close(dtype, m.whole(tok), want)
    assert close(dtype, m.cut(tok, [127, 1, 1, 128, 2, 126, 64, 9, 1]), want)
    assert close(dtype, m.cut(tok, [255, 2, 3]), want)
    m.close()


def test_tensor_core_products_match_the_plain_ones(ctx):
    m = Model(ctx, dk.WIDE, 6, BF16)
    tok = dk.tokens_of(dk.WIDE, 300, 2)
    a = m.whole(tok)
    ctx.set_option("dense_tc", 0)
    b = m.whole(tok)
    ctx.set_option("dense_tc", 1)
    assert kit.error(a, b.astype(np.float64)).max() < 0.05
    m.close()


@both
def test_caches_that_are_shorter_than_the_sequence(ctx, dtype):
    """A prompt of several passes, and portions and single tokens behind it: the rings of keys and values go round, states cross
    from pass to pass."""
    cfg = dk.config(16, 30, [dk.attention(2, 1, 8, 8, 50, 20, 0.8, None), dk.delta(1, 1, 8, 8, 3, None), dk.mlstm(1, 8, 8, 6.0, None)])
    m = Model(ctx, cfg, 7, dtype, max_seq=5000)
    tok = dk.tokens_of(cfg, 4700, 3)
    want, _ = m.oracle(tok)
    m.dec.reset()
    places = list(range(5)) + list(range(2040, 2060)) + list(range(2170, 2182)) + list(range(4090, 4100)) + [4199]
    got = [m.dec.extend(tok[:4200], places)]
    at = 4200
    for n in [130, 1, 1, 2, 64, 3, 150] + [1] * 30 + [119]:
        got.append(m.dec.extend(tok[at:at + n], range(n)))
        places += range(at, at + n)
        at += n
    assert at == 4700
    assert close(dtype, np.concatenate(got), want[places])
    m.close()


@both
def test_one_key_of_the_chunk_stands_out(ctx, dtype):
    """Scores so peaked that nearly all of the weight is on one key, near or far, first of the chunk, at a tile's border; a key just
    outside of the chunk must not be seen: a key that is missed, doubled or off by one shows at once."""
    cfg = dk.config(64, 400, [dk.attention(2, 2, 32, 24, 130, 40, 0.5, None)])
    n = 400
    tok = np.random.default_rng(1).permutation(n).astype(np.int32)  # no token twice
    inside = {129: 0, 128: 1, 64: 63, 192: 191, 193: 130, 259: 131, 256: 255, 258: 130, 320: 319, 389: 260, 388: 323, 127: 65}
    outside = {130: 129, 132: 0, 260: 259, 261: 134, 390: 389, 391: 261}  # (the key is in the chunk before)
    m = Model(ctx, cfg, 8, dtype, edit=dk.pointing_queries("l0.", {**inside, **outside}, tok, 2.0))
    want, _ = m.oracle(tok)
    # the test is sharp: with one position more or less in a chunk the expected logits move far beyond the tolerance
    for size in (129, 131):
        off = json.loads(json.dumps(cfg))
        off["layers"][0]["mixer"]["mask"]["size"] = size
        e = kit.error(do.forward(off, m.w, tok)[0], want)
        assert e[[129] if size == 129 else [130, 260, 390]].min() > 5 * TOL[BF16]
    for got in (m.whole(tok), m.cut(tok, [100, 28, 1]), m.cut(tok, [129, 2, 61, 1]), m.cut(tok, [131, 2, 127, 9])):
        assert close(dtype, got, want)
    m.close()


@both
@pytest.mark.parametrize("chunk", [1, 2, 63, 64, 65, 127, 128, 129, 600])
def test_chunk_sizes_around_the_tiles(ctx, chunk, dtype):
    cfg = dk.config(32, 60, [dk.attention(3, 3, 16, 16, chunk, 30, 1.0, None)])
    m = Model(ctx, cfg, 9, dtype, max_seq=320)
    tok = dk.tokens_of(cfg, 300, 4)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [63, 1, 2, 130]), m.cut(tok, [200, 2, 1])):
        assert close(dtype, got, want)
    m.close()


@both
@pytest.mark.parametrize("buckets,far", [(2, 1.5), (4, 7), (8, 300), (32, 64), (48, 4000)])
def test_distance_biases(ctx, buckets, far, dtype):
    """Small scores, large biases: the attention is nearly the bias alone."""
    cfg = dk.config(32, 60, [dk.attention(4, 2, 16, 16, 280, far, 0.02, None)])

    def edit(w):
        w["l0.mix.rel"] *= 2.0

    m = Model(ctx, cfg, 10, dtype, buckets=buckets, edit=edit)
    tok = dk.tokens_of(cfg, 300, 5)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [150, 7, 1, 2, 133, 1])):
        assert close(dtype, got, want)
    m.close()


def test_the_sink_takes_its_share(ctx):
    """Scores far below the sink's 0, then far above: outputs near nothing, and as if there were no sink."""
    for shift in (-6.0, 6.0):
        cfg = dk.config(32, 60, [dk.attention(2, 1, 16, 16, 100, 30, 0.05, None)], alpha=0.05)

        def edit(w):
            w["l0.mix.rel"][:] = shift

        for dtype in (F32, BF16):
            m = Model(ctx, cfg, 11, dtype, edit=edit)
            tok = dk.tokens_of(cfg, 150, 6)
            want, _ = m.oracle(tok)
            for got in (m.whole(tok), m.cut(tok, [120, 1])):
                assert close(dtype, got, want)
            m.close()


@both
@pytest.mark.parametrize("keep,write", [(8.0, 0.0), (-3.0, 0.0), (2.0, 6.0), (3.0, -9.0)], ids=["slow", "fast", "strong", "weak"])
def test_memories_from_none_to_almost_all(ctx, keep, write, dtype):
    """States that keep their first tokens for hundreds of positions, and that forget at once, over the chunks of a prompt; input gates
    that move the running maximum up, and down below 0."""
    cfg = dk.config(48, 64, [dk.delta(4, 2, 40, 36, 2, None), dk.mlstm(2, 40, 36, 12.0, None), dk.mlstm(1, 70, 20, 30.0, None)])
    m = Model(ctx, cfg, 12, dtype, keep=keep, write=write)
    tok = dk.tokens_of(cfg, 330, 7)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [63, 1, 2, 130]), m.cut(tok, [300, 1])):
        assert close(dtype, got, want)
    m.close()


@both
def test_strong_and_weak_decays_in_one_chunk(ctx, dtype):
    """Tokens that wipe the state between tokens that keep it: what survives must not feel the size of the wiping."""
    cfg = dk.config(32, 40, [dk.delta(2, 2, 16, 16, 1, None), dk.mlstm(2, 16, 16, 40.0, None)])

    def edit(w):
        w["l0.mix.a"] *= 6.0
        w["l0.mix.A_log"][:] = 2.5
        w["l0.mix.dt_bias"][:] = -6.0
        w["l1.mix.f"] *= 12.0
        w["l1.mix.i"] *= 8.0

    m = Model(ctx, cfg, 13, dtype, edit=edit)
    tok = dk.tokens_of(cfg, 200, 8)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [65, 2, 1])):
        e = kit.error(got, want)  # (the gates are steep: bf16 inputs move them)
        assert close(dtype, got, want) if dtype == F32 else np.median(e) < 0.1
    m.close()


def test_repeated_keys_are_corrected(ctx):
    """Two tokens in turn with write strength near one: every write has to take out what the one before left at the same key."""
    cfg = dk.config(24, 12, [dk.delta(2, 1, 8, 8, 1, None)], alpha=0.5)

    def edit(w):
        w["l0.mix.b"] *= 4.0

    m = Model(ctx, cfg, 14, F32, keep=6.0, edit=edit)
    tok = np.array([1, 2, 1, 1, 2, 2, 5] * 40, np.int32)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [64, 65, 1, 3]), m.cut(tok, [1])):
        assert close(F32, got, want)
    m.close()


@pytest.mark.parametrize("dim", [1, 3, 200, 300, 420])
def test_key_channels_of_every_chunk_length(ctx, dim):
    cfg = dk.config(32, 40, [dk.delta(2, 1, dim, 24, 3, None), dk.mlstm(1, dim, 20, 8.0, None)])
    m = Model(ctx, cfg, 15, F32, max_seq=160)
    tok = dk.tokens_of(cfg, 150, 9)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [70, 1, 2])):
        assert close(F32, got, want)
    m.close()


@both
def test_first_tokens_see_zeros_before_the_start(ctx, dtype):
    cfg = dk.config(40, 60, [dk.delta(2, 2, 8, 8, 7, None), dk.attention(2, 1, 8, 8, 3, 20, 0.5, None), dk.mlstm(1, 8, 8, 5.0, None)])
    m = Model(ctx, cfg, 16, dtype)
    for n in (1, 2, 3, 6, 7, 8):
        tok = dk.tokens_of(cfg, n, 20 + n)
        want, _ = m.oracle(tok)
        for got in (m.whole(tok), m.cut(tok, [1]), m.cut(tok, [2, 1])):
            assert close(dtype, got, want)
    m.close()


@both
def test_unequal_sequences_together_and_alone(ctx, dtype):
    """Eleven sequences (more than one pass) with prompts of unequal length, stepped together, against the oracle; then slots are given
    to new sequences while the others go on."""
    cfg = dk.SHARED
    B = 11
    m = Model(ctx, cfg, 17, dtype, max_seq=160, batch=B)
    lens = [1, 2, 3, 9, 33, 64, 65, 90, 17, 5, 128]
    seqs = [list(dk.tokens_of(cfg, n, 30 + i)) for i, n in enumerate(lens)]
    for i, s in enumerate(seqs):
        m.dec.select(i)
        m.dec.reset()
        assert kit.error(m.dec.extend(s, [len(s) - 1]), m.oracle(s)[0][-1:]).max() < 5 * TOL[dtype]

    def together(steps, seed):
        rng = np.random.default_rng(seed)
        for _ in range(steps):
            new = rng.integers(0, cfg["vocab"], B).astype(np.int32)
            got = m.dec.step_batch(new)
            for i in range(B):
                seqs[i].append(int(new[i]))
        for i in range(B):
            assert kit.error(got[i:i + 1], m.oracle(seqs[i])[0][-1:]).max() < 5 * TOL[dtype], i

    together(4, 1)
    for i, n in ((0, 40), (7, 2), (10, 1)):  # slots used again
        seqs[i] = list(dk.tokens_of(cfg, n, 60 + i))
        m.dec.select(i)
        m.dec.reset()
        m.dec.extend(seqs[i])
    together(5, 2)
    m.close()


@both
@pytest.mark.parametrize("heads,kv,dim,vdim", [(17, 1, 24, 16), (40, 2, 16, 8), (2, 2, 1, 1), (3, 1, 130, 129), (2, 1, 264, 20), (2, 2, 20, 270), (8, 4, 256, 200)])
def test_head_counts_and_sizes(ctx, heads, kv, dim, vdim, dtype):
    """Groups of more heads than a CTA takes, heads too large for the tensor-core kernels, and tiny ones."""
    cfg = dk.config(40, 60, [dk.attention(heads, kv, dim, vdim, 90, 30, dim ** -0.5, None)])
    m = Model(ctx, cfg, 23, dtype, max_seq=220)
    tok = dk.tokens_of(cfg, 200, 11)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [85, 3, 1, 1, 70, 1])):
        assert close(dtype, got, want)
    m.close()


@both
def test_sequences_far_enough_apart_to_split_their_keys(ctx, dtype):
    """Steps whose sequences see many tiles, one, and none but their own token."""
    cfg = dk.config(48, 60, [dk.attention(8, 2, 24, 40, 1000, 200, 0.5, None), dk.attention(3, 3, 16, 16, 90, 40, 0.5, None)])
    m = Model(ctx, cfg, 18, dtype, max_seq=1200, batch=4)
    seqs = [list(dk.tokens_of(cfg, n, 40 + n)) for n in (1110, 999, 70, 1)]
    for i, s in enumerate(seqs):
        m.dec.select(i)
        m.dec.reset()
        m.dec.extend(s)
    rng = np.random.default_rng(1)
    got = []
    for _ in range(3):
        new = rng.integers(0, 60, 4).astype(np.int32)
        got.append(m.dec.step_batch(new))
        for s, t in zip(seqs, new):
            s.append(int(t))
    for i, s in enumerate(seqs):
        assert close(dtype, np.array([g[i] for g in got]), m.oracle(s)[0][-3:]), i
    m.close()


@both
def test_long_decoding(ctx, dtype):
    cfg = dk.SHARED
    m = Model(ctx, cfg, 19, dtype, max_seq=420)
    tok = dk.tokens_of(cfg, 400, 10)
    want, _ = m.oracle(tok)
    assert close(dtype, m.cut(tok, [10, 1]), want)
    m.close()


def greedy_is_right(m, prompt, generated, tol):
    """Every generated token's expected logit is the maximum (up to the tolerance)."""
    seq = list(prompt) + list(generated)
    want, _ = m.oracle(seq)
    spread = want.std()
    for i, t in enumerate(generated):
        row = want[len(prompt) - 1 + i]
        assert row[t] >= row.max() - tol * spread, (i, t)


@pytest.mark.parametrize("dtype,tol", [(F32, 1e-4), (BF16, 0.2)], ids=["f32", "bf16"])
def test_greedy_generation_through_the_entry_points(ctx, dtype, tol):
    cfg = dk.SHARED
    m = Model(ctx, cfg, 20, dtype, max_seq=256)
    for n in (1, 2, 37, 130):
        prompt = dk.tokens_of(cfg, n, 70 + n)
        out, metrics = m.dec.generate(prompt, 24)
        greedy_is_right(m, prompt, out, tol)
        assert metrics.launches_per_token > 0 and m.dec.kv_offset == n + 24
    prompt = dk.tokens_of(cfg, 20, 99)
    m.dec.forward(prompt)
    m.dec.continue_greedy(10)
    greedy_is_right(m, prompt, m.dec.generated_tokens(10), tol)
    m.close()
    m = Model(ctx, cfg, 20, dtype, max_seq=128, batch=3)
    prompts = [dk.tokens_of(cfg, n, 80 + n) for n in (3, 40, 1)]
    for i, p in enumerate(prompts):
        m.dec.select(i)
        m.dec.reset()
        m.dec.extend(p)
    m.dec.continue_batch(12)
    for p, out in zip(prompts, m.dec.generated_tokens_batch(12)):
        greedy_is_right(m, p, out, tol)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_command_line_and_trace_replay(tmp_path, dtype):
    cfg = dk.SHARED
    w = dk.random_weights(cfg, 21)
    model = str(tmp_path / "model")
    kit.save(model, cfg, w)
    prompts = [dk.tokens_of(cfg, 30, 90), dk.tokens_of(cfg, 7, 91)]
    r = subprocess.run([sys.executable, "-m", "loom_b200", "generate", "--model", model, "--dtype", dtype, "--max-new", "5"] +
                       [a for p in prompts for a in ("--tokens", ",".join(map(str, p)))], cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    m = type("M", (), {"oracle": lambda self, t: do.forward(cfg, w, t)})()
    for p, line in zip(prompts, r.stdout.strip().splitlines()):
        greedy_is_right(m, p, json.loads(line)["tokens"], 1e-4 if dtype == "float32" else 0.2)
    out = tmp_path / "out"
    out.mkdir()
    seq = dk.tokens_of(cfg, 50, 92).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": seq[:20], "want": [3, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": seq[20:49], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": seq[49:], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": seq[:4], "want": [3]}], "end": ["y"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", model, "--dtype", dtype, "--out", str(out), "--max-tokens", "60"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done %d" % i for i in range(4)]
    want, _ = do.forward(cfg, w, seq)
    tol = TOL[cabi.DTYPES[dtype]]
    for n, places in ((0, [3, 19]), (2, [49]), (3, [3])):
        got = np.fromfile(out / ("%d.f32" % n), "<f4").reshape(-1, cfg["vocab"])
        assert kit.error(got, want[places]).max() < tol
    assert not (out / "1.f32").exists()


def test_refusals(ctx):
    w = dk.random_weights(dk.SHARED, 22)

    def built(change):
        cfg = json.loads(json.dumps(dk.SHARED))
        change(cfg)
        models.build(ctx, cfg, kit.Weights(w), models.LoadOptions(F32, 32)).close()

    with pytest.raises(loom_b200.LoomB200Error, match="distance buckets"):
        built(lambda c: c["layers"][0]["mixer"].update(bias_max=2))
    with pytest.raises(loom_b200.LoomB200Error, match="gate cap"):
        built(lambda c: c["layers"][2]["mixer"].update(gate_cap=0.0))
    with pytest.raises(AssertionError):  # tensors of another size
        built(lambda c: c["layers"][1]["mixer"].update(conv=3))
    dec = cabi.Decoder.stack(ctx, 1, 16, 20, 1e-5, residual_alpha=1.0)
    mat = cabi.Matrix(ctx, 16, 16)
    spec = dict(mixer=cabi.MIXER_ATTENTION, heads=3, kv_heads=2, dim=8, vdim=8)
    with pytest.raises(loom_b200.LoomB200Error, match="3 heads over 2"):
        dec.set_layer(0, spec, {"in": mat, "out": mat})
    with pytest.raises(loom_b200.LoomB200Error, match="expected"):
        dec.set_layer(0, dict(spec, heads=2), {"in": mat, "out": mat, "norm1_w": np.ones(16)})
    dec.close()
