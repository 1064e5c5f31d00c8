"""Suselorn on the GPU against the float64 oracle (tests/suselorn_ref.py): every mechanism alone, prompts against
single steps, portions, tile edges, slots used again, batches, generation."""
import json
import subprocess
import sys

import numpy as np
import pytest

import suselorn_ref as ref
from conftest import ROOT
from decoder_util import bf16_round, error, one_by_one, portions, tokens, whole, write_model
from suselorn_util import config, dense, latent, plain_streams, silence, weights

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 4e-2}
DTYPES = ["float32", "bfloat16"]


def build(dev, cfg, w, dtype, **kw):
    from tensorlogic_b200 import suselorn
    from tensorlogic_b200.decoder import Decoder, model_from_arrays
    kw.setdefault("max_seq", 512)
    return Decoder(dev, model_from_arrays(dev, w, dtype), suselorn.read_config(cfg), dtype, **kw)


def check(dev, cfg, w, seq, dtypes=DTYPES, tol=1.0, **kw):
    """Whole prompt and token by token, both types, against the oracle."""
    want = ref.forward(cfg, w, seq)
    for dtype in dtypes:
        dec = build(dev, cfg, w, dtype, **kw)
        for how, got in (("whole", whole(dec, seq)), ("single", one_by_one(dec, seq)), ("sevens", portions(dec, seq, [7] * len(seq)))):
            e = error(got, want)
            assert e < tol * TOL[dtype], (dtype, how, e)


# ---- mechanisms -----------------------------------------------------------------------------------

@pytest.mark.parametrize("cap", [0.7, 30.0])
def test_norm_cap_and_tied_output_alone(dev, cap):
    """Everything else silent: logits = cap of embedding table . norm(sum of the mixed streams)."""
    cfg = config([dense(latent())], width=56, vocab=67, softcap=cap)
    w = silence(weights(cfg, 1), 0, mixer=True, ff=True)
    check(dev, cfg, w, tokens(20, 67))


@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8])
@pytest.mark.parametrize("width", [48, 50])
def test_streams(dev, streams, width):
    cfg = config([dense(latent()), latent(), dense(latent(2, 8, 4, 12))], width=width, streams=streams)
    check(dev, cfg, weights(cfg, streams, gain=0.7), tokens(40, 61), tol=2.0)


def test_streams_keep_32_bits(dev):
    """Sixteen passes that each add a bias far below a bf16 step of the streams."""
    cfg = config([dense(latent())], vocab=40, softcap=1e4, loop=(0, 1, 16))
    w = plain_streams(silence(weights(cfg, 2), 0, mixer=True), 0, 3)
    step = np.random.default_rng(0).standard_normal(48).astype(np.float32)
    w["final.norm.alpha"][...] = 0.125
    w["l0.ls2"][:] = 1
    w["l0.mlp.down"][:] = 0
    w["l0.mlp.down.b"] = bf16_round(step * 2e-3)
    seq = tokens(24, 40)
    want = ref.forward(cfg, w, seq)
    moved = error(ref.forward(cfg, dict(w, **{"l0.mlp.down.b": 0 * step}), seq), want)
    for how in (whole, one_by_one):
        e = error(how(build(dev, cfg, w, "bfloat16"), seq), want)
        assert e < 0.2 * moved, (e, moved)


@pytest.mark.parametrize("ff", [40, 33, 200, 1])
def test_feed_forward_alone(dev, ff):
    cfg = config([dense(latent(), ff)])
    check(dev, cfg, silence(weights(cfg, ff, gain=1.5), 0, mixer=True), tokens(40, 61))


# heads, dim, rot, vdim, q_rank, kv_rank
SIZES = [(4, 16, 8, 16, 24, 16), (6, 24, 10, 12, 20, 40), (1, 8, 2, 8, 8, 8), (3, 40, 6, 20, 33, 17), (17, 32, 16, 48, 40, 64),
         (40, 16, 16, 16, 24, 32), (2, 128, 64, 128, 96, 512), (2, 64, 32, 192, 48, 136), (2, 130, 64, 64, 40, 264),
         (1, 192, 64, 64, 32, 32), (2, 32, 16, 32, 24, 600), (2, 48, 80, 208, 200, 72), (3, 16, 16, 80, 16, 1), (2, 16, 0, 16, 1, 24),
         (1, 7, 4, 5, 9, 12)]


@pytest.mark.parametrize("size", SIZES)
def test_attention_sizes(dev, size):
    heads, dim, rot, vdim, q_rank, kv_rank = size
    cfg = config([latent(*size, scale=1.5 * (dim + rot) ** -0.5)], width=40)
    check(dev, cfg, plain_streams(weights(cfg, heads + dim), 0, 3), tokens(150, 61))


@pytest.mark.parametrize("sink", [-1e4, 0.0, 6.0, 1e4])
def test_sink(dev, sink):
    """Far above every score the heads give nothing, far below they are a plain softmax."""
    cfg = config([latent()])
    w = plain_streams(weights(cfg, 6), 0, 3)
    w["l0.mix.sink"] = bf16_round(np.array([sink, 0.5, sink, -0.5]))
    check(dev, cfg, w, tokens(100, 61))


def test_negative_scale(dev):
    cfg = config([latent(scale=-0.4)])
    check(dev, cfg, weights(cfg, 7), tokens(100, 61))


def test_large_scores(dev):
    """Scores of some thousands, falling and rising along the keys: the running maximum moves by far more than its
    threshold, up to overflow of an unshifted exponential."""
    cfg = config([latent(2, 16, 0, 16, 24, 16, scale=300.0)])
    w, seq = plain_streams(weights(cfg, 8), 0, 3), tokens(300, 61)
    want = ref.forward(cfg, w, seq)
    for dtype in DTYPES:
        dec = build(dev, cfg, w, dtype)
        for got in (whole(dec, seq), one_by_one(dec, seq, 250), portions(dec, seq, [100, 9, 191])):
            assert np.isfinite(got).all()
            d = got - want
            rows = np.sqrt(((d - d.mean(-1, keepdims=True)) ** 2).mean(-1)) / want.std()
            # the softmax picks single keys: bf16 rounding may swap two that are close
            assert np.median(rows) < (1e-3 if dtype == "float32" else 0.1) and np.quantile(rows, 0.9) < (1e-2 if dtype == "float32" else 1.0)


def test_eps_of_the_latent_norms(dev):
    cfg = config([latent()], eps=0.4)
    check(dev, cfg, weights(cfg, 9), tokens(60, 61))


def marked_model(dim=16, vdim=16):
    """A token (7) whose key meets every query with a score far above the rest."""
    cfg = config([latent(2, dim, 2, vdim, 8, 16, base=1e9, scale=0.75)], width=32, vocab=20, streams=2, softcap=60.0)
    w = plain_streams(weights(cfg, 12), 0, 2)
    w["embed"][:, :8] = 0
    w["embed"][7, :8] = 3
    w["l0.norm1.alpha"][...] = 1
    w["l0.norm1"][:] = 1
    w["l0.norm1"][8:16] = 0
    w["l0.norm1.b"][:] = 0
    w["l0.norm1.b"][8:16] = 1                         # the same for every token: all the queries are made of it
    w["l0.mix.dq"][:, :8] = 0
    w["l0.mix.dq"][:, 16:] = 0
    w["l0.mix.dkv"][0] = 0
    w["l0.mix.dkv"][0, :8] = 4                        # latent entry 0: the mark
    w["l0.mix.dkv"][:, 8:16] = 0
    w["l0.mix.dkv"][16:] = 0                          # no rotated part
    q = w["l0.mix.dq"][:, 8:16].astype(np.float64).sum(1)
    q = w["l0.mix.uq"].astype(np.float64) @ (q / np.sqrt((q * q).mean()) * w["l0.mix.dq.norm"])
    for h in range(2):
        u = q[h * (dim + 2):h * (dim + 2) + dim]
        w["l0.mix.uk"][h * dim:(h + 1) * dim] *= 0.1
        w["l0.mix.uk"][h * dim:(h + 1) * dim, 0] = 5 * u / (u @ u)
    w["l0.mix.dkv.norm"][:] = 1
    w["l0.mix.sink"][:] = 0
    return cfg, {k: bf16_round(v).reshape(np.shape(v)) for k, v in w.items()}


@pytest.mark.parametrize("offset", [0, 1, 15, 16, 17, 31, 32, 63, 64, 65, 127, 128, 129, 190, 191, 192])
def test_one_key_that_stands_out(dev, offset):
    """Its value appears in every later row and in none before: keys far away, at the edges of tiles, and the
    newest one; a lost, doubled or early key shows."""
    cfg, w = marked_model()
    seq = [t if t != 7 else 8 for t in tokens(400, 20, 3)]
    seq[offset] = 7
    want = ref.forward(cfg, w, seq)
    plain = list(seq)
    plain[offset] = 8
    moved = np.abs(ref.forward(cfg, w, plain) - want).max(-1)
    assert moved[offset + 1:].min() > 2 and moved[:offset].max(initial=0) < 1e-9
    for dtype, tol in (("float32", 1e-3), ("bfloat16", 0.5)):
        dec = build(dev, cfg, w, dtype)
        for got in (whole(dec, seq), one_by_one(dec, seq, max(offset, 200)), one_by_one(dec, seq[:offset + 3]),
                    portions(dec, seq, [offset + 1, 2, 40, 2, 17, 400])):
            assert np.abs(got - want[:len(got)]).max() < tol


def test_two_marked_tokens_far_apart(dev):
    """The weights divide evenly between the first and the latest of two equal keys, whatever stretch they lie in."""
    cfg, w = marked_model(32, 48)
    seq = [t if t != 7 else 8 for t in tokens(500, 20, 4)]
    seq[3] = seq[330] = 7
    want = ref.forward(cfg, w, seq)
    for dtype, tol in (("float32", 1e-3), ("bfloat16", 0.5)):
        dec = build(dev, cfg, w, dtype)
        for got in (whole(dec, seq), one_by_one(dec, seq, 300), portions(dec, seq, [331, 5, 164])):
            assert np.abs(got - want).max() < tol


# ---- whole models ----------------------------------------------------------------------------------

def mixed(**kw):
    """Layers that differ in everything, the middle two run three times."""
    kw.setdefault("loop", (1, 3, 3))
    return config([dense(latent(6, 24, 16, 16, 20, 40, 100.0), 50), latent(3, 16, 16, 32, 33, 24, 20.0),
                   dense(latent(2, 40, 6, 20, 24, 17), 36), dense(latent(18, 16, 8, 8, 16, 64), 24)], width=72, vocab=91, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_layers_whole_single_and_portions(dev, dtype):
    cfg = mixed()
    w, seq = weights(cfg, 33, gain=0.7), tokens(330, 91)
    want = ref.forward(cfg, w, seq)
    dec = build(dev, cfg, w, dtype)
    ways = {"whole": whole(dec, seq), "single": one_by_one(dec, seq), "after 130": one_by_one(dec, seq, 130)}
    for sizes in ([2] * 165, [3, 64, 2, 63, 1, 65, 132], [100, 100, 130], [329, 1], [1, 329], [17, 16, 2, 18, 128, 149]):
        ways[str(sizes[:4])] = portions(dec, seq, sizes)
    for how, got in ways.items():
        assert error(got, want) < (5 if dtype == "float32" else 1) * TOL[dtype], (how, error(got, want))


@pytest.mark.parametrize("n", [63, 64, 65, 127, 128, 129, 191, 192, 193, 255, 256, 257, 384])
def test_prompt_lengths_around_tiles(dev, n):
    cfg = config([dense(latent(3, 32, 16, 32, 24, 32)), latent(2, 64, 16, 160, 24, 48)])
    w, seq = weights(cfg, n), tokens(n, 61, n)
    dec = build(dev, cfg, w, "bfloat16")
    want = ref.forward(cfg, w, seq)
    assert error(whole(dec, seq), want) < TOL["bfloat16"]
    assert error(portions(dec, seq, [n // 2, n]), want) < TOL["bfloat16"]


def test_portions_larger_than_the_row_buffers(dev):
    """A prompt runs in several passes, with more wanted rows than one pass has room for."""
    cfg = mixed()
    w, seq = weights(cfg, 34, gain=0.7), tokens(150, 91)
    want = ref.forward(cfg, w, seq)
    for dtype, tol in (("float32", 5), ("bfloat16", 1)):
        dec = build(dev, cfg, w, dtype, max_prefill=32, max_logit_rows=7)
        assert error(whole(dec, seq), want) < tol * TOL[dtype]
        for places in ([149, 3, 64], [149], [40]):
            s = dec.open()
            assert error(dec.feed(s, seq, places), want[places]) < tol * TOL[dtype]
            dec.close(s)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_used_again(dev, dtype):
    """Requests one after the other, long and short, in the same cache rows: what ran before leaves no trace."""
    cfg = config([dense(latent(3, 32, 16, 32, 24, 32)), latent()], loop=(0, 2, 2))
    w = weights(cfg, 41)
    dec = build(dev, cfg, w, dtype, max_seq=256, max_batch=3)
    first = {}
    for n in (250, 3, 100, 1, 250, 3, 100, 1):
        seq = tokens(n, 61, n)
        got = portions(dec, seq, [n // 2 + 1, n])
        if n in first:
            assert np.array_equal(got, first[n])
        else:
            first[n] = got
            assert error(got, ref.forward(cfg, w, seq)) < 2 * TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_interleaved_requests_in_different_slots(dev, dtype):
    cfg = config([dense(latent(3, 32, 16, 32, 24, 32)), dense(latent(5, 20, 6, 12))])
    w = weights(cfg, 42, gain=0.7)
    dec = build(dev, cfg, w, dtype, max_seq=200, max_batch=3)
    alone = build(dev, cfg, w, dtype)
    seqs = [tokens(n, 61, n) for n in (120, 50, 200)]
    slots, parts, at = [dec.open() for _ in seqs], [[] for _ in seqs], [0, 0, 0]
    assert len(set(slots)) == 3
    rng = np.random.default_rng(3)
    while any(a < len(s) for a, s in zip(at, seqs)):
        i, n = int(rng.integers(3)), int(rng.integers(1, 40))
        part = seqs[i][at[i]:at[i] + n]
        if part:
            parts[i].append(dec.feed(slots[i], part, range(len(part))))
            at[i] += len(part)
    for s, p in zip(seqs, parts):
        assert error(np.concatenate(p), whole(alone, s)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_decode_of_unequal_sequences(dev, dtype):
    cfg = config([dense(latent(18, 24, 8, 16, 20, 40)), latent()], loop=(0, 1, 2))
    w = weights(cfg, 43, gain=0.7)
    n, steps = (130, 7, 64, 1, 250), 9
    seqs = [tokens(k + steps, 61, k) for k in n]
    dec = build(dev, cfg, w, dtype, max_batch=5)
    alone = build(dev, cfg, w, dtype)
    want = [one_by_one(alone, s, k) for s, k in zip(seqs, n)]
    for i in range(5):
        assert dec.open() == i
        dec.feed(i, seqs[i][:n[i]])
    for t in range(steps):
        _, logits = dec.decode([s[k + t] for s, k in zip(seqs, n)], return_logits=True)
        for i in range(5):
            assert error(logits[i:i + 1], want[i][n[i] + t:n[i] + t + 1]) < TOL[dtype]


def test_long_decode(dev):
    cfg = config([dense(latent(4, 16, 8, 16, scale=0.6)), latent(2, 32, 16, 32, 24, 136)], loop=(0, 1, 2))
    w, seq = weights(cfg, 44), tokens(900, 61)
    want = ref.forward(cfg, w, seq)
    for dtype in DTYPES:
        dec = build(dev, cfg, w, dtype, max_seq=900)
        assert error(one_by_one(dec, seq, 2), want) < 2 * TOL[dtype]


@pytest.mark.parametrize("width,vocab", [(50, 61), (51, 130), (129, 33), (8, 9), (520, 40)])
def test_widths(dev, width, vocab):
    """Rows that are no whole number of 16-byte pieces; one and several wanted rows of a prompt; the sampled token."""
    cfg = config([dense(latent(3, 10, 6, 7), 37), latent(5, 13, 4, 9)], width=width, vocab=vocab)
    w, seq = weights(cfg, width, gain=0.7), tokens(40, vocab)
    check(dev, cfg, w, seq, tol=2.0)
    want = ref.forward(cfg, w, seq)
    for dtype in DTYPES:
        dec = build(dev, cfg, w, dtype)
        for place in (39, 17):
            s = dec.open()
            got = dec.feed(s, seq, [place])
            dec.close(s)
            assert error(got, want[[place]]) < 3 * TOL[dtype]
        tok, _ = dec.prefill(seq, return_logits=False)
        row = want[-1]
        assert row.max() - row[tok] < (1e-6 if dtype == "float32" else 0.2) * row.std()


def test_last_cache_row_and_beyond(dev):
    from tensorlogic_b200._lib import TensorError
    cfg = config([latent()])
    w, seq = weights(cfg, 45), tokens(64, 61)
    dec = build(dev, cfg, w, "bfloat16", max_seq=64)
    s = dec.open()
    dec.feed(s, seq[:62])
    dec.feed(s, [seq[62]], [0])
    got = dec.feed(s, [seq[63]], [0])
    assert error(got, ref.forward(cfg, w, seq)[-1:]) < TOL["bfloat16"]
    for bad in (lambda: dec.feed(s, [1], [0]), lambda: dec.prefill([1], 64), lambda: dec.prefill([61], 0)):
        with pytest.raises(TensorError):
            bad()


# ---- loading, generation, command line ---------------------------------------------------------------

def test_load_and_generate_through_the_registry(dev, tmp_path):
    from tensorlogic_b200 import registry
    cfg = mixed()
    w = weights(cfg, 55, gain=0.7)
    write_model(tmp_path, cfg, w)
    prompt = tokens(40, 91, 5)
    want = ref.greedy(cfg, w, prompt, 12)
    r = registry.load(dev, str(tmp_path), "float32", max_seq=64)
    assert list(registry.generate(r, prompt, 12)) == want
    r.prefill(prompt, return_logits=False)       # steps without a round trip to the host
    r.decode_enqueue(1, 5)
    assert r.read_state()[0][0] == want[5]


def test_bf16_generation_follows_its_own_logits(dev):
    """Greedy tokens through graph replay equal the argmax of the logits of the same sequence fed as a prompt."""
    from tensorlogic_b200 import registry
    cfg = config([dense(latent(8, 32, 16, 32, 48, 64), 96), dense(latent(8, 32, 16, 32, 48, 64), 96)], width=128, vocab=257)
    w, prompt = weights(cfg, 56), tokens(50, 257, 6)
    dec = build(dev, cfg, w, "bfloat16")
    out = list(registry.generate(dec, prompt, 40))
    full = build(dev, cfg, w, "bfloat16").prefill(prompt + out, all_rows=True)[1]
    for i, t in enumerate(out):
        row = full[len(prompt) + i - 1]
        assert row.max() - row[t] < 0.05 * row.std()
    plain = build(dev, cfg, w, "bfloat16", use_graph=False)
    assert list(registry.generate(plain, prompt, 40)) == out


def test_temperature_draws(dev):
    """The sampled token is the first whose running probability passes the draw."""
    cfg = config([latent()])
    w, prompt = weights(cfg, 57), tokens(9, 61)
    dec = build(dev, cfg, w, "float32")
    dec.set_sampling(1.3, seed=77)
    tok, logits = dec.prefill(prompt)
    pos = len(prompt) - 1
    for _ in range(10):
        p = np.exp((logits[0].astype(np.float64) - logits[0].max()) / 1.3)
        c = np.cumsum(p) / p.sum()
        u = dev.lib.tlc_sample_uniform_host(77, pos, 0)
        assert np.abs(c - u).min() < 1e-5 or tok == int(np.argmax(c > u))
        nxt, logits = dec.decode([tok], return_logits=True)
        tok, pos = int(nxt[0]), pos + 1


def test_launches_of_a_decode_step(dev):
    """Seven kernels per pass of a layer, five without a feed-forward, and embedding, logits, sample."""
    cfg = config([dense(latent()), latent(), dense(latent())], loop=(1, 3, 2))
    dec = build(dev, cfg, weights(cfg, 58), "bfloat16")
    dec.prefill(tokens(5, 61), return_logits=False)
    dec.decode_enqueue(1, 3)
    dev.synchronize()
    assert dec.launches_per_step == 7 + 2 * (5 + 7) + 3


def test_dependent_launch_changes_nothing(dev):
    cfg = mixed()
    w, seq = weights(cfg, 59, gain=0.7), tokens(120, 91)
    got = []
    for pdl in (1, 0):
        dev.set_option("pdl", pdl)
        dec = build(dev, cfg, w, "bfloat16")
        got.append(np.concatenate([whole(dec, seq), one_by_one(dec, seq, 60)]))
    dev.set_option("pdl", 1)
    assert np.array_equal(got[0], got[1])


def test_bad_models_are_refused(dev):
    from tensorlogic_b200._lib import TensorError
    cfg = config([dense(latent())])
    w = weights(cfg, 60)
    build(dev, cfg, w, "bfloat16")
    for broken in ({k: v for k, v in w.items() if k != "l0.mix.sink"}, {k: v for k, v in w.items() if k != "l0.hc2.mix"},
                   dict(w, **{"l0.mix.uk": w["l0.mix.uk"][:-1]}), dict(w, **{"final.norm.alpha": np.ones(2, np.float32)})):
        with pytest.raises(TensorError):
            build(dev, cfg, broken, "bfloat16")
    many = config([latent()], streams=9)
    with pytest.raises(TensorError):
        build(dev, many, weights(many), "bfloat16")


@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 4e-2)])
def test_trace_runner_and_command_line(tmp_path, dtype, tol):
    cfg = mixed()
    w = weights(cfg, 61, gain=0.7)
    write_model(tmp_path, cfg, w)
    seq = tokens(70, 91)
    want = ref.forward(cfg, w, seq)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": seq[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": seq[40:41], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": seq[41:], "want": []}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": seq[:2], "want": [1]}], "end": ["y"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([f"{ROOT}/bin/trace_run", "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "80"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, 91)
    assert error(read(0), want[[0, 39]]) < tol and error(read(1), want[[40]]) < tol and error(read(3), want[[1]]) < tol
    assert not (out / "2.f32").exists()
    if dtype == "bfloat16":
        return
    r = subprocess.run([sys.executable, "-m", "tensorlogic_b200", "generate", "--model", str(tmp_path), "--dtype", dtype, "--prompt",
                        ",".join(map(str, seq[:20])), "--new", "4"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == ref.greedy(cfg, w, seq[:20], 4)
