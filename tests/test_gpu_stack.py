"""Layer stacks on the GPU against the plain oracle (`stack_oracle.py`): every mechanism alone and together, in float32 and in bf16,
as whole prompts, portions, single tokens, several sequences, reused slots, and through the generation entry points.

float32 stacks are held to 2e-5 of the logits' spread (what float32 sums of this length cost), bf16 stacks to a few per cent
(two roundings of 2^-9 per product through a handful of layers), and bf16 against itself with another cut of the prompt to the
same bound.
"""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import loom_b200
import stack_oracle as so
import stackkit as kit
from loom_b200 import cabi, models

pytestmark = pytest.mark.gpu
F32, BF16 = cabi.DTYPE_F32, cabi.DTYPE_BF16
TOL = {F32: 2e-5, BF16: 0.06}

def close(cfg, dtype, got, want):
    """Rounding costs little at almost every position (a normed head output near zero magnifies it at a few).  In bf16 a token whose
    experts are a close call may go elsewhere, and the tokens after it feel that: with a real choice of experts most positions count."""
    e = kit.error(got, want)
    chooses = any(x["mlp"] and x["mlp"]["kind"] == "moe" and x["mlp"]["router"]["top"] < x["mlp"]["router"]["experts"] for x in cfg["layers"])
    if dtype == BF16 and chooses:
        return np.median(e) < TOL[dtype]
    return np.quantile(e, 0.9) < TOL[dtype] and e.max() < 10 * TOL[dtype]


ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def ctx():
    c = loom_b200.Context(0)
    yield c
    c.close()


class Model:
    def __init__(self, ctx, cfg, seed, dtype, max_seq=512, batch=1, edit=None, layers=None, **kw):
        self.cfg, self.w = cfg, kit.random_weights(cfg, seed, **kw)
        if edit:
            edit(self.w)
            self.w = {k: kit.bf16_round(v) for k, v in self.w.items()}
        self.dec = models.build(ctx, cfg, kit.Weights(self.w), models.LoadOptions(dtype, max_seq, batch, layers))
        self.dtype = dtype

    def oracle(self, tokens):
        return so.forward(self.cfg, self.w, tokens)

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


def tokens_of(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).astype(np.int32)


GLA = kit.config(56, 90, [kit.gla(3, 20, 28, 8.0, None)], taps=3)
LATENT = kit.config(72, 90, [kit.latent(5, 24, 12, 40, 0.4, None)], taps=2)
DENSE = kit.config(40, 70, [kit.gla(1, 8, 8, 4.0, kit.dense(100))], taps=1)
MOE = kit.config(48, 70, [kit.gla(1, 8, 8, 4.0, kit.moe(36, 6, 3, 0.8))], taps=4, mult=1.2)
SHARED = kit.config(64, 90, [kit.latent(2, 16, 20, 24, 0.5, kit.dense(48)), kit.gla(2, 12, 16, 4.0, None), kit.latent(3, 8, 12, 24, 0.3, None, kv_from=0),
                             kit.latent(2, 8, 8, 24, 0.6, kit.moe(24, 4, 1), kv_from=0)], taps=5)
ODD = kit.config(77, 101, [kit.latent(3, 11, 13, 19, 0.35, kit.moe(21, 5, 2, 0.5)), kit.gla(2, 37, 9, 1.0, kit.dense(33)), kit.gla(5, 3, 70, 32.0, None)],
                 taps=6, eps=3e-3, mult=0.37)
WIDE = kit.config(384, 517, [kit.gla(3, 96, 160, 16.0, kit.dense(640)), kit.latent(9, 80, 56, 144, 0.11, kit.moe(200, 12, 2)),
                             kit.gla(2, 130, 72, 5.0, kit.moe(136, 3, 3)), kit.latent(4, 48, 96, 144, 0.2, kit.dense(136), kv_from=1)], taps=4, mult=0.8)
EVERY = kit.config(96, 90, [kit.gla(2, 24, 32, 4.0, kit.moe(72, 3, 3)), kit.latent(3, 16, 24, 40, 0.3, kit.moe(40, 2, 2, 0.4))], taps=3)
ALL = {"every": EVERY, "gla": GLA, "latent": LATENT, "dense": DENSE, "moe": MOE, "shared": SHARED, "odd": ODD, "wide": WIDE}


@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(ALL))
def test_prompt_portions_and_decoding_match_the_oracle(ctx, name, dtype):
    cfg = ALL[name]
    m = Model(ctx, cfg, 3, dtype)
    tok = tokens_of(cfg, 61)
    want, after = m.oracle(tok)
    got = m.whole(tok)
    assert close(cfg, dtype, got, want)
    r = m.dec.last_residual(64)
    assert close(cfg, dtype, r, after[-1])
    for sizes in ([1], [2], [3, 17, 2, 1], [40, 1]):
        assert close(cfg, dtype, m.cut(tok, sizes), want), sizes
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
def test_long_sequences_cross_every_block_border(ctx, dtype):
    cfg = WIDE
    m = Model(ctx, cfg, 4, dtype, max_seq=640)
    tok = tokens_of(cfg, 560, 1)
    want, _ = m.oracle(tok)
    assert close(cfg, dtype, m.whole(tok), want)
    assert close(cfg, dtype, m.cut(tok, [127, 1, 1, 128, 2, 126, 64, 65, 1]), want)
    assert close(cfg, dtype, m.cut(tok, [255, 2, 3]), want)
    m.close()


def test_tensor_core_products_match_the_plain_ones(ctx):
    m = Model(ctx, WIDE, 5, BF16)
    tok = tokens_of(WIDE, 300, 2)
    a = m.whole(tok)
    ctx.set_option("dense_tc", 0)
    b = m.whole(tok)
    ctx.set_option("dense_tc", 1)
    assert kit.error(a, b.astype(np.float64)).max() < 0.03
    m.close()


def test_blocks_of_a_long_prompt(ctx):
    """More tokens than one pass holds: the states cross from pass to pass."""
    cfg = kit.config(16, 30, [kit.gla(1, 8, 8, 16.0, None), kit.latent(1, 8, 8, 8, 0.5, None)], taps=3)
    m = Model(ctx, cfg, 6, F32, max_seq=2400)
    tok = tokens_of(cfg, 2300, 3)
    m.dec.reset()
    places = list(range(5)) + list(range(2040, 2060)) + [2299]
    got = m.dec.extend(tok, places)
    want, _ = m.oracle(tok)
    assert close(cfg, F32, got, want[places])
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
def test_one_far_key_stands_out(ctx, dtype):
    """Scores so peaked that nearly all of the weight is on one key, near or far, first or at a block border: a key that is missed,
    doubled or off by one shows at once."""
    cfg = kit.config(64, 300, [kit.latent(2, 32, 24, 48, 1.0, None)], taps=2, mult=1.0)
    n = 300
    tok = tokens_of(cfg, n, 4)
    targets = {140: 0, 141: 1, 200: 127, 201: 128, 202: 129, 256: 255, 257: 256, 258: 0, 299: 128, 298: 299 - 2, 130: 127, 129: 128}
    for q, k in sorted(targets.items()):
        tok[q] = tok[k]  # equal tokens make equal normed rows, hence equal queries and keys

    def edit(w):  # no mixing over time, and queries equal to keys: the score is the squared norm where the tokens agree
        w["l0.canon1"][:] = 0
        rng = np.random.default_rng(7)
        dkv = rng.standard_normal((48, 64)) / 8
        uk = rng.standard_normal((64, 48)) / 7
        w["l0.mix.dkv"], w["l0.mix.uk"] = dkv, uk
        w["l0.mix.dkv.norm"][:] = 1.0
        w["l0.mix.q"] = uk @ dkv
        w["l0.mix.uv"] *= 3.0

    m = Model(ctx, cfg, 8, dtype, edit=edit)
    want, _ = m.oracle(tok)
    # the test is sharp: leaving out the target key moves the expected logits far beyond the tolerance
    w = {k: v.astype(np.float64) for k, v in m.w.items()}
    x = so.rms_norm(w["embed"][tok], w["embed.norm"], cfg["norm"]["eps"])
    h = so.rms_norm(x, w["l0.norm1"], cfg["norm"]["eps"])
    c = so.latent_of(h, w, "l0.mix.", cfg["norm"]["eps"])
    q, k = (h @ w["l0.mix.q"].T).reshape(n, 2, 32), (c @ w["l0.mix.uk"].T).reshape(n, 2, 32)
    for qi, ki in targets.items():
        if qi == ki or ki > qi:
            continue
        for hd in range(2):
            s = k[:qi + 1, hd] @ q[qi, hd]
            p = np.exp(s - s.max())
            p /= p.sum()
            same = p[tok[:qi + 1] == tok[ki]].sum()
            assert same > 0.5, (qi, ki, same)
    for got in (m.whole(tok), m.cut(tok, [100, 28, 1]), m.cut(tok, [129, 2, 61, 1])):
        assert close(cfg, dtype, got, want)
    m.close()


@pytest.mark.parametrize("bias,tau", [(6.0, 64.0), (-8.0, 1.0), (0.0, 2.0)], ids=["slow", "fast", "medium"])
@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
def test_decays_from_none_to_almost_all(ctx, bias, tau, dtype):
    """A state that keeps its first tokens for hundreds of positions, and one that forgets at once, over the chunks of a prompt."""
    cfg = kit.config(48, 64, [kit.gla(2, 40, 36, tau, None), kit.gla(1, 70, 20, tau, None)], taps=2)
    m = Model(ctx, cfg, 9, dtype, decay_bias=bias)
    tok = tokens_of(cfg, 330, 5)
    want, _ = m.oracle(tok)
    for got in (m.whole(tok), m.cut(tok, [63, 1, 2, 130]), m.cut(tok, [300, 1])):
        assert close(cfg, dtype, got, want)
    m.close()


def test_first_tokens_see_zeros_before_the_start(ctx):
    cfg = kit.config(40, 60, [kit.gla(1, 8, 8, 4.0, None), kit.latent(1, 8, 8, 8, 0.5, None)], taps=7)
    m = Model(ctx, cfg, 10, F32)
    for n in (1, 2, 3, 6, 7, 8):
        tok = tokens_of(cfg, n, 20 + n)
        want, _ = m.oracle(tok)
        assert close(cfg, F32, m.whole(tok), want)
        assert close(cfg, F32, m.cut(tok, [1]), want)
        assert close(cfg, F32, m.cut(tok, [2, 1]), want)
    m.close()


@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
def test_unequal_sequences_together_and_alone(ctx, dtype):
    """Eleven sequences (more than one pass) with prompts of unequal length, stepped together, against the oracle; then slots are given
    to new sequences while the others go on."""
    cfg = SHARED if dtype == F32 else kit.config(64, 90, [dict(x, mlp=None) for x in SHARED["layers"]], taps=5)
    B = 11
    m = Model(ctx, cfg, 11, dtype, max_seq=160, batch=B)
    lens = [1, 2, 3, 9, 33, 64, 65, 90, 17, 5, 128]
    seqs = [list(tokens_of(cfg, n, 30 + i)) for i, n in enumerate(lens)]
    for i, s in enumerate(seqs):
        m.dec.select(i)
        m.dec.reset()
        assert kit.error(m.dec.extend(s, [len(s) - 1]), m.oracle(s)[0][-1:]).max() < 10 * TOL[dtype]

    def together(steps, seed):
        rng = np.random.default_rng(seed)
        for _ in range(steps):
            new = rng.integers(0, cfg["vocab"], B).astype(np.int32)
            got = m.dec.step_batch(new)
            for i in range(B):
                seqs[i].append(int(new[i]))
        for i in range(B):
            assert kit.error(got[i:i + 1], m.oracle(seqs[i])[0][-1:]).max() < 10 * TOL[dtype], i

    together(4, 1)
    for i, n in ((0, 40), (7, 2), (10, 1)):  # slots used again
        seqs[i] = list(tokens_of(cfg, n, 60 + i))
        m.dec.select(i)
        m.dec.reset()
        m.dec.extend(seqs[i])
    together(5, 2)
    m.close()


def test_long_decoding(ctx):
    cfg = SHARED
    m = Model(ctx, cfg, 12, F32, max_seq=420)
    tok = tokens_of(cfg, 400, 6)
    want, _ = m.oracle(tok)
    got = m.cut(tok, [10, 1])
    assert close(cfg, F32, got, want)
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
    cfg = SHARED
    m = Model(ctx, cfg, 13, dtype, max_seq=256)
    for n in (1, 2, 37, 130):
        prompt = tokens_of(cfg, n, 70 + n)
        out, metrics = m.dec.generate(prompt, 24)
        greedy_is_right(m, prompt, out, tol)
        assert metrics.launches_per_token > 0 and m.dec.kv_offset == n + 24
    # forward / continue / read back
    prompt = tokens_of(cfg, 20, 99)
    m.dec.forward(prompt)
    m.dec.continue_greedy(10)
    greedy_is_right(m, prompt, m.dec.generated_tokens(10), tol)
    m.close()
    m = Model(ctx, cfg, 13, dtype, max_seq=128, batch=3)
    prompts = [tokens_of(cfg, n, 80 + n) for n in (3, 40, 1)]
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
    cfg = SHARED
    w = kit.random_weights(cfg, 14)
    model = str(tmp_path / "model")
    kit.save(model, cfg, w)
    prompts = [tokens_of(cfg, 30, 90), tokens_of(cfg, 7, 91)]
    r = subprocess.run([sys.executable, "-m", "loom_b200", "generate", "--model", model, "--dtype", dtype, "--max-new", "5"] +
                       [a for p in prompts for a in ("--tokens", ",".join(map(str, p)))], cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    m = type("M", (), {"oracle": lambda self, t: so.forward(cfg, w, t)})()
    for p, line in zip(prompts, r.stdout.strip().splitlines()):
        greedy_is_right(m, p, json.loads(line)["tokens"], 1e-4 if dtype == "float32" else 0.2)
    out = tmp_path / "out"
    out.mkdir()
    seq = tokens_of(cfg, 50, 92).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": seq[:20], "want": [3, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": seq[20:49], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": seq[49:], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": seq[:4], "want": [3]}], "end": ["y"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", model, "--dtype", dtype, "--out", str(out), "--max-tokens", "60"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done %d" % i for i in range(4)]
    want, _ = so.forward(cfg, w, seq)
    tol = TOL[cabi.DTYPES[dtype]]
    for n, places in ((0, [3, 19]), (2, [49]), (3, [3])):
        got = np.fromfile(out / ("%d.f32" % n), "<f4").reshape(-1, cfg["vocab"])
        assert kit.error(got, want[places]).max() < tol
    assert not (out / "1.f32").exists()


def test_refusals(ctx):
    m = Model(ctx, SHARED, 15, F32, max_seq=32)
    tok = tokens_of(SHARED, 40, 1)
    with pytest.raises(loom_b200.LoomB200Error, match="exceed MaxSeqLen"):
        m.dec.extend(tok)
    m.dec.extend(tok[:8])
    with pytest.raises(loom_b200.LoomB200Error, match="cannot be cut back"):
        m.dec.set_kv_offset(4)
    with pytest.raises(loom_b200.LoomB200Error, match="places ascend"):
        m.dec.extend(tok[:4], [2, 1])
    with pytest.raises(loom_b200.LoomB200Error, match="not for a layer stack"):
        m.dec.last_hidden()
    m.close()
    dec = cabi.Decoder.stack(ctx, 1, 16, 20, 1e-5)
    mat = cabi.Matrix(ctx, 16, 16)
    spec = dict(mixer=cabi.MIXER_LATENT, heads=1, dim=8, vdim=8, rank=8, kv_from=0, scale=1.0)
    with pytest.raises(loom_b200.LoomB200Error, match="does not come before"):
        dec.set_layer(0, spec, {"in": mat, "out": mat})
    with pytest.raises(loom_b200.LoomB200Error, match="expected"):
        dec.set_layer(0, dict(spec, mixer=cabi.MIXER_GLA, kv_from=-1, tau=1.0), {"in": mat, "out": mat, "mixer_norm": np.ones(8), "decay_w": np.ones(64),
                                                                                  "decay_b": np.ones(8)})
    with pytest.raises(loom_b200.LoomB200Error, match="has no weights|not set"):
        dec.extend([1, 2])
    dec.close()


def test_ternary_decoder_takes_portions(ctx):
    """`extend` is the decoder's own: a ternary prompt cut into portions ends in the same logits as in one call."""
    from oracle import oracle as orc
    rng = np.random.default_rng(1)
    L, H, heads, kvh, hd, I, V = 2, 256, 2, 1, 128, 384, 300
    dec = cabi.Decoder(ctx, L, H, heads, kvh, hd, I, V, 1e-5, 500000.0, cabi.ACT_SILU, 128)
    shapes = ((heads * hd, H), (kvh * hd, H), (kvh * hd, H), (H, heads * hd), (I, H), (I, H), (H, I))
    for b in range(L):
        ws = []
        for r, c in shapes:
            om = orc.Matrix.from_f32((rng.standard_normal(r * c) * 0.02).astype(np.float32), r, c)
            ws.append(ctx.upload_ternary(om.words, r, c, om.scale))
        dec.set_block(b, ws)
    emb = (rng.standard_normal((V, H)) * 0.02).astype(np.float32)
    dec.set_embeddings(ctx.to_device(emb))
    tok = rng.integers(0, V, 90).astype(np.int32)
    want = dec.forward(tok)
    dec.reset()
    at = 0
    for n in (40, 3, 1, 33, 12, 1):
        got = dec.extend(tok[at:at + n], [n - 1])[0]
        at += n
    assert np.abs(got - want).max() <= 1e-5 * np.abs(want).max()
    with pytest.raises(loom_b200.LoomB200Error, match="last token"):
        dec.extend(tok[:4], [0, 3])
    dec.close()
