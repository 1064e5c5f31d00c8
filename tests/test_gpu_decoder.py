"""Decoder on the GPU against the float64 oracle (tests/decoder_ref.py): every mechanism alone, prompts
against single steps, portions, edges of windows and tiles, slots used again, batches, generation."""
import copy
import json
import subprocess
import sys

import numpy as np
import pytest

import decoder_ref as ref
from conftest import ROOT
from decoder_util import (attention, config, dense, error, moe, one_by_one, portions, tokens, weights, whole, write_model,
                          write_safetensors)

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 4e-2}
DTYPES = ["float32", "bfloat16"]


def build(dev, cfg, w, dtype, **kw):
    from tensorlogic_b200 import toposun
    from tensorlogic_b200.decoder import Decoder, model_from_arrays
    kw.setdefault("max_seq", 512)
    return Decoder(dev, model_from_arrays(dev, w, dtype), toposun.read_config(cfg), dtype, **kw)


def check(dev, cfg, w, seq, dtypes=DTYPES, tol=1.0, **kw):
    """Whole prompt and token by token, both types, against the oracle."""
    want = ref.forward(cfg, w, seq)
    for dtype in dtypes:
        dec = build(dev, cfg, w, dtype, **kw)
        for how, got in (("whole", whole(dec, seq)), ("single", one_by_one(dec, seq))):
            e = error(got, want)
            assert e < tol * TOL[dtype], (dtype, how, e)


def silence(w, layer, mixer=False):
    """Makes the mixer of a layer add nothing."""
    if mixer:
        w[f"l{layer}.mix.o"][:] = 0
        w[f"l{layer}.mix.o.b"][:] = 0
    return w


# ---- mechanisms -----------------------------------------------------------------------------------

def test_norm_and_tied_output_alone(dev):
    """Mixer silent, no feed-forward: logits = embedding table . layer norm(embedding); a large eps and a
    large mean tell the norm from others."""
    cfg = config([attention()], width=56, vocab=67, eps=0.3)
    w = silence(weights(cfg, 1), 0, mixer=True)
    w["embed"] = (w["embed"] + 1.5).astype(np.float32)
    from decoder_util import bf16_round
    w["embed"] = bf16_round(w["embed"])
    check(dev, cfg, w, tokens(20, 67))


def test_residual_keeps_32_bits(dev):
    """Sixteen layers that each add a bias far below a bf16 step of the residual."""
    cfg = config([attention() for _ in range(16)], width=48, vocab=40)
    w = weights(cfg, 2)
    rng = np.random.default_rng(0)
    step = rng.standard_normal(48).astype(np.float32)
    from decoder_util import bf16_round
    for i in range(16):
        w[f"l{i}.mix.o"][:] = 0
        w[f"l{i}.mix.o.b"] = bf16_round(step * 2e-3)
    seq = tokens(12, 40)
    want = ref.forward(cfg, w, seq)
    base = dict(w, **{f"l{i}.mix.o.b": 0 * step for i in range(16)})
    moved = error(ref.forward(cfg, base, seq), want)
    for how in (whole, one_by_one):
        e = error(how(build(dev, cfg, w, "bfloat16"), seq), want)
        assert e < 0.15 * moved, (e, moved)


@pytest.mark.parametrize("heads,kv,dim,rot", [(4, 2, 16, 16), (6, 1, 24, 10), (5, 5, 8, 2), (3, 3, 40, 40), (18, 1, 32, 32),
                                              (40, 2, 12, 6), (8, 2, 100, 60), (2, 1, 130, 64), (2, 2, 200, 200), (4, 1, 33, 20),
                                              (1, 1, 7, 4), (2, 1, 256, 128), (2, 1, 300, 300)])
def test_attention_sizes(dev, heads, kv, dim, rot):
    cfg = config([attention(heads, kv, dim, window=23, keep=3, rot=rot, scale=1.5 * dim ** -0.5)], width=40)
    check(dev, cfg, weights(cfg, heads + dim), tokens(90, 61))


def test_values_are_the_raw_keys(dev):
    """Norm weights and a rotation that would distort the values if they were taken after either."""
    cfg = config([attention(4, 2, 16, window=12, keep=1, base=3.0)])
    w = weights(cfg, 4)
    w["l0.mix.k.norm"] = (w["l0.mix.k.norm"] * 3 + 1).astype(np.float32)
    w["l0.mix.k.b"] = (w["l0.mix.k.b"] * 4).astype(np.float32)
    from decoder_util import bf16_round
    w = {k: bf16_round(v) for k, v in w.items()}
    check(dev, cfg, w, tokens(50, 61))


@pytest.mark.parametrize("width,vocab", [(50, 61), (51, 130), (129, 33), (8, 9), (520, 40)])
def test_widths(dev, width, vocab):
    """Rows that are no whole number of 16-byte pieces; one and several wanted rows of a prompt."""
    cfg = config([dense(attention(3, 1, 10, 12, 1, 6), 37), moe(attention(2, 2, 9, 5, 2, 4), 3, 1, 11, 5), attention(5, 1, 13, 9, 0, 12)],
                 width=width, vocab=vocab)
    w, seq = weights(cfg, width, gain=0.7), tokens(40, vocab)
    check(dev, cfg, w, seq, dtypes=["float32"], tol=5.0)
    want = ref.forward(cfg, w, seq)
    for dtype in DTYPES:
        dec = build(dev, cfg, w, dtype)
        for place in (39, 17):
            s = dec.open()
            got = dec.feed(s, seq, [place])
            dec.close(s)
            assert error(got, want[[place]]) < (5 * TOL["float32"] if dtype == "float32" else 0.2)
        tok, _ = dec.prefill(seq, return_logits=False)
        row = want[-1]
        assert row.max() - row[tok] < (1e-6 if dtype == "float32" else 0.2) * row.std()


def test_norm_spans_the_whole_projection(dev):
    """One head's rows are twenty times the others': a norm per head would equalize them."""
    cfg = config([attention(4, 4, 16, window=30, keep=0)])
    w = weights(cfg, 5)
    w["l0.mix.q"][:16] *= 16
    w["l0.mix.k"][16:32] *= 16
    check(dev, cfg, w, tokens(40, 61))


EDGES = [(1, 0), (1, 1), (2, 0), (5, 0), (7, 2), (63, 1), (64, 0), (64, 4), (65, 3), (128, 5), (129, 64), (40, 70), (500, 3)]


@pytest.mark.parametrize("window,keep", EDGES)
def test_window_edges(dev, window, keep):
    """Sharp scores: each query leans on one or two keys, so the key just inside or outside an edge shows."""
    m = dict(window=window, keep=keep, scale=1.2)
    cfg = config([attention(4, 2, 16, **m), attention(4, 1, 16, **m)])
    w, seq = weights(cfg, window + keep), tokens(300, 61, window)
    want = ref.forward(cfg, w, seq)
    for field, by in (("size", 1), ("keep_first", 1), ("size", -1), ("keep_first", -1)):
        bad = copy.deepcopy(cfg)
        for l in bad["layers"]:
            l["mixer"]["mask"][field] += by
        if bad["layers"][0]["mixer"]["mask"]["size"] < 1 or bad["layers"][0]["mixer"]["mask"]["keep_first"] < 0 or window >= 300:
            continue
        assert error(ref.forward(bad, w, seq), want) > 20 * TOL["float32"]
    dec = build(dev, cfg, w, "float32")
    assert error(whole(dec, seq), want) < 5 * TOL["float32"]
    assert error(one_by_one(dec, seq, 180), want) < 5 * TOL["float32"]
    dec = build(dev, cfg, w, "bfloat16")
    for got in (whole(dec, seq), one_by_one(dec, seq, 180), portions(dec, seq, [2, 62, 1, 63, 64, 3, 70, 100])):
        d = got - want
        rows = np.sqrt(((d - d.mean(-1, keepdims=True)) ** 2).mean(-1)) / want.std()
        # sharp scores magnify bf16 rounding of queries and keys; a wrong key would move many rows by about 1
        assert np.median(rows) < 0.05 and np.quantile(rows, 0.98) < 0.35, (np.median(rows), rows.max())


@pytest.mark.parametrize("offset", [0, 1, 20, 62, 63, 64, 65, 66, 100, 127, 128])
def test_one_key_that_stands_out(dev, offset):
    """One token's key meets every query with a score far above the rest: its value appears exactly in
    the rows that may see it (a window of 64, two kept tokens)."""
    from decoder_util import bf16_round
    cfg = config([attention(2, 1, 16, window=64, keep=2, rot=2, base=1e9, scale=0.75)], width=32, vocab=20, eps=1e-6)
    w = weights(cfg, 9)
    sign = np.array([1, -1] * 4)
    w["embed"][:, 1:8:2] = w["embed"][:, 0:8:2]      # every other token has nothing along `sign` ...
    w["embed"][7] = 0
    w["embed"][7, :8] = 2 * sign                     # ... and this one nothing else
    w["l0.mix.q"] *= 0.05
    w["l0.mix.q.b"][:] = 1.0                         # every query points along (1, .., 1)
    for n in ("l0.norm1", "l0.mix.q.norm", "l0.mix.k.norm"):
        w[n][:] = 1.0
    w["l0.mix.k.b"][:] = 0
    w["l0.mix.k"][:, :8] = sign
    w["l0.mix.o"] *= 2
    w = {k: bf16_round(v) for k, v in w.items()}
    seq = [t if t != 7 else 8 for t in tokens(200, 20, 3)]
    seq[offset] = 7
    want = ref.forward(cfg, w, seq)
    plain = list(seq)
    plain[offset] = 8
    moved = np.abs(ref.forward(cfg, w, plain) - want).max(-1)
    sees = np.array([ref.visible(i, offset, 64, 2) for i in range(200)])
    assert moved[sees].min() > 5 and moved[~sees].max(initial=0) < 1e-9
    for dtype, tol in (("float32", 1e-3), ("bfloat16", 0.3)):
        dec = build(dev, cfg, w, dtype)
        for got in (whole(dec, seq), one_by_one(dec, seq, offset + 1), portions(dec, seq, [50, 2, 30, 2, 116])):
            assert np.abs(got - want).max() < tol


@pytest.mark.parametrize("ff,limit", [(40, 1.5), (33, 0.4), (200, 7.0), (1, 1.0)])
def test_clamped_glu_alone(dev, ff, limit):
    cfg = config([dense(attention(), ff, limit)])
    w = silence(weights(cfg, ff, gain=2.0), 0, mixer=True)
    check(dev, cfg, w, tokens(40, 61))


@pytest.mark.parametrize("experts,top,ff,shared", [(5, 2, 24, 16), (8, 1, 24, 0), (3, 3, 9, 40), (70, 4, 8, 8), (1, 1, 16, 12),
                                                   (40, 33, 8, 0)])
def test_experts_alone(dev, experts, top, ff, shared):
    cfg = config([moe(attention(), experts, top, ff, shared)])
    w = silence(weights(cfg, experts, gain=1.5), 0, mixer=True)
    seq = tokens(70, 61)
    # no close calls between the last chosen and the first left out
    h = ref.layer_norm(w["embed"].astype(np.float64), w["l0.norm2"], cfg["norm"]["eps"])
    s = np.sort(h @ w["l0.mlp.router"].T.astype(np.float64), -1)[:, ::-1]
    if top < experts:
        clear = [t for t in range(61) if s[t, top - 1] - s[t, top] > 0.05]
        assert len(clear) > 4
        seq = [clear[t % len(clear)] for t in seq]
    check(dev, cfg, w, seq)


def test_parallel_branches_read_the_same_residual(dev):
    cfg = config([dense(attention(), 40), moe(attention(), 4, 1, 16, 8), attention(), dense(attention(), 24)])
    w = weights(cfg, 21)
    seq = tokens(80, 61)
    check(dev, cfg, w, seq, dtypes=["float32"], tol=3.0)


# ---- whole models ----------------------------------------------------------------------------------

def mixed(window=17, keep=3, **kw):
    """Layers that differ in everything."""
    return config([moe(attention(6, 2, 24, window, keep, 12, 100.0), 6, 2, 20, 12),
                   dense(attention(4, 1, 16, window + 50, 0), 50, 1.0),
                   attention(2, 2, 40, 5, 1, 20),
                   moe(attention(3, 1, 16, 2 * window, keep + 2, 8, 20.0), 4, 1, 16, 0)], width=72, vocab=91, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_layers_whole_single_and_portions(dev, dtype):
    cfg = mixed()
    w, seq = weights(cfg, 33, gain=0.7), tokens(260, 91)
    want = ref.forward(cfg, w, seq)
    dec = build(dev, cfg, w, dtype)
    ways = {"whole": whole(dec, seq), "single": one_by_one(dec, seq), "after 130": one_by_one(dec, seq, 130)}
    for sizes in ([2] * 130, [3, 64, 2, 63, 1, 65, 62], [100, 100, 100], [259, 1], [1, 259], [17, 16, 2, 18, 207]):
        ways[str(sizes[:4])] = portions(dec, seq, sizes)
    if dtype == "float32":
        for how, got in ways.items():
            assert error(got, want) < 5 * TOL[dtype], (how, error(got, want))
        return
    # a router call closer than bf16 rounding may go either way in a few rows
    for how, got in ways.items():
        d = got - want
        rows = np.sqrt(((d - d.mean(-1, keepdims=True)) ** 2).mean(-1)) / want.std()
        assert np.median(rows) < 0.02 and np.quantile(rows, 0.9) < 0.06, (how, np.median(rows), np.quantile(rows, 0.9))


def test_portions_larger_than_the_row_buffers(dev):
    """A prompt runs in several passes, with more wanted rows than one pass has room for."""
    cfg = mixed()
    w, seq = weights(cfg, 34, gain=0.7), tokens(150, 91)
    dec = build(dev, cfg, w, "float32", max_prefill=32, max_logit_rows=7)
    want = ref.forward(cfg, w, seq)
    assert error(whole(dec, seq), want) < 5 * TOL["float32"]
    s = dec.open()
    assert error(dec.feed(s, seq, [149, 3, 64]), want[[149, 3, 64]]) < 5 * TOL["float32"]
    dec.close(s)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_used_again(dev, dtype):
    """Requests one after the other, long and short, in the same cache rows: what ran before leaves no trace."""
    cfg = config([dense(attention(window=21, keep=3)), attention(window=70, keep=1)])
    w = weights(cfg, 41)
    dec = build(dev, cfg, w, dtype, max_seq=256, max_batch=3)
    first = {}
    for i, n in enumerate((250, 3, 100, 1, 250, 3, 100, 1)):
        seq = tokens(n, 61, n)
        got = portions(dec, seq, [n // 2 + 1, n])
        if n in first:
            assert np.array_equal(got, first[n])
        else:
            first[n] = got
            assert error(got, ref.forward(cfg, w, seq)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_interleaved_requests_in_different_slots(dev, dtype):
    cfg = config([dense(attention(window=21, keep=3)), moe(attention(window=40, keep=1), 4, 2, 16, 8)])
    w = weights(cfg, 42, gain=0.7)
    dec = build(dev, cfg, w, dtype, max_batch=3)
    alone = build(dev, cfg, w, dtype)
    seqs = [tokens(n, 61, n) for n in (120, 50, 90)]
    slots, parts = [dec.open() for _ in seqs], [[] for _ in seqs]
    assert len(set(slots)) == 3
    at = [0, 0, 0]
    rng = np.random.default_rng(3)
    while any(a < len(s) for a, s in zip(at, seqs)):
        i = int(rng.integers(3))
        n = int(rng.integers(1, 30))
        part = seqs[i][at[i]:at[i] + n]
        if part:
            parts[i].append(dec.feed(slots[i], part, range(len(part))))
            at[i] += len(part)
    for s, p in zip(seqs, parts):
        assert error(np.concatenate(p), whole(alone, s)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_decode_of_unequal_sequences(dev, dtype):
    cfg = config([dense(attention(6, 2, 24, 21, 3)), moe(attention(4, 1, 16, 40, 1), 4, 2, 16, 8)])
    w = weights(cfg, 43, gain=0.7)
    n, steps = (130, 7, 64), 9
    seqs = [tokens(k + steps, 61, k) for k in n]
    dec = build(dev, cfg, w, dtype, max_batch=3)
    alone = build(dev, cfg, w, dtype)
    want = [one_by_one(alone, s, k) for s, k in zip(seqs, n)]
    for i in range(3):
        assert dec.open() == i
        dec.feed(i, seqs[i][:n[i]])
    for t in range(steps):
        _, logits = dec.decode([s[k + t] for s, k in zip(seqs, n)], return_logits=True)
        for i in range(3):
            assert error(logits[i:i + 1], want[i][n[i] + t:n[i] + t + 1]) < TOL[dtype]


def test_long_decode(dev):
    cfg = config([dense(attention(4, 2, 16, 37, 3, scale=0.6)), attention(4, 2, 16, 130, 0)])
    w, seq = weights(cfg, 44), tokens(900, 61)
    want = ref.forward(cfg, w, seq)
    for dtype in DTYPES:
        dec = build(dev, cfg, w, dtype, max_seq=900)
        assert error(one_by_one(dec, seq, 2), want) < 2 * TOL[dtype]


def test_last_cache_row_and_beyond(dev):
    from tensorlogic_b200._lib import TensorError
    cfg = config([attention(window=9)])
    w, seq = weights(cfg, 45), tokens(64, 61)
    dec = build(dev, cfg, w, "bfloat16", max_seq=64)
    s = dec.open()
    dec.feed(s, seq[:62])
    dec.feed(s, [seq[62]], [0])
    got = dec.feed(s, [seq[63]], [0])
    assert error(got, ref.forward(cfg, w, seq)[-1:]) < TOL["bfloat16"]
    with pytest.raises(TensorError):
        dec.feed(s, [1], [0])
    with pytest.raises(TensorError):
        dec.prefill([1], 64)
    with pytest.raises(TensorError):
        dec.prefill([61], 0)
    dec.close(s)
    with pytest.raises(TensorError):
        dec.prefill([1], 5)      # nothing of the sequence is in the cache yet


# ---- loading, generation, command line ---------------------------------------------------------------

@pytest.mark.parametrize("file_type", ["BF16", "F16", "F32"])
def test_load_and_generate_through_the_registry(dev, tmp_path, file_type):
    from tensorlogic_b200 import registry
    cfg = mixed()
    w = weights(cfg, 55, gain=0.7)
    if file_type == "F16":
        w = {k: v.astype(np.float16).astype(np.float32) for k, v in w.items()}
    write_model(tmp_path, cfg, w, file_type)
    prompt = tokens(40, 91, 5)
    want = ref.greedy(cfg, w, prompt, 12)
    r = registry.load(dev, str(tmp_path), "float32", max_seq=64)
    assert list(registry.generate(r, prompt, 12)) == want
    stop = want[4]
    assert list(registry.generate(r, prompt, 12, stop=[stop])) == want[:want.index(stop) + 1]
    # steps without a round trip to the host
    r.prefill(prompt, return_logits=False)
    r.decode_enqueue(1, 5)
    assert r.read_state()[0][0] == want[5]


def test_bf16_generation_follows_its_own_logits(dev):
    """Greedy tokens through graph replay equal the argmax of the logits of the same sequence fed as a prompt."""
    from tensorlogic_b200 import registry
    cfg = config([dense(attention(8, 2, 32, 30, 2), 96), dense(attention(8, 2, 32, 300, 0), 96)], width=128, vocab=257)
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
    cfg = config([attention()])
    w, prompt = weights(cfg, 57), tokens(9, 61)
    dec = build(dev, cfg, w, "float32")
    dec.set_sampling(1.3, seed=77)
    tok, logits = dec.prefill(prompt)
    pos = len(prompt) - 1
    for _ in range(20):
        p = np.exp((logits[0].astype(np.float64) - logits[0].max()) / 1.3)
        c = np.cumsum(p) / p.sum()
        u = dev.lib.tlc_sample_uniform_host(77, pos, 0)
        assert np.abs(c - u).min() < 1e-5 or tok == int(np.argmax(c > u))
        nxt, logits = dec.decode([tok], return_logits=True)
        tok, pos = int(nxt[0]), pos + 1


def test_launches_of_a_decode_step(dev):
    """Three kernels per layer, four with experts, and embedding, logits, sample."""
    cfg = config([dense(attention()), moe(attention()), attention()])
    dec = build(dev, cfg, weights(cfg, 58), "bfloat16")
    dec.prefill(tokens(5, 61), return_logits=False)
    dec.decode_enqueue(1, 3)
    dev.synchronize()
    assert dec.launches_per_step == 3 + 3 + 4 + 3


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


def test_bad_files_are_refused(dev, tmp_path):
    from tensorlogic_b200._lib import TensorError
    from tensorlogic_b200.decoder import load_safetensors
    cfg = config([attention()])
    w = weights(cfg, 60)
    good = tmp_path / "m.safetensors"
    write_safetensors(good, w)
    m = load_safetensors(dev, good)
    assert sorted(m.names()) == sorted(w)
    raw = good.read_bytes()
    n = int.from_bytes(raw[:8], "little")
    head = json.loads(raw[8:8 + n])

    def variant(change):
        h = copy.deepcopy(head)
        change(h)
        text = json.dumps(h).encode()
        p = tmp_path / "bad.safetensors"
        p.write_bytes(len(text).to_bytes(8, "little") + text + raw[8 + n:])
        return p
    cases = [variant(lambda h: h["embed"].update(dtype="I64")), variant(lambda h: h["embed"].update(shape=[61, 47])),
             variant(lambda h: h["embed"].update(data_offsets=[0, 10**12])), variant(lambda h: h["embed"].pop("shape"))]
    for p in cases:
        with pytest.raises(TensorError):
            load_safetensors(dev, p)
    for blob in (b"", b"\xff" * 8, raw[:8 + n // 2], (2**60).to_bytes(8, "little"), raw[:-10]):
        p = tmp_path / "bad.safetensors"
        p.write_bytes(blob)
        with pytest.raises(TensorError):
            load_safetensors(dev, p)
    with pytest.raises(TensorError):           # a tensor is missing
        build(dev, cfg, {k: v for k, v in w.items() if k != "l0.mix.o.b"}, "bfloat16")
    with pytest.raises(TensorError):           # a tensor of another shape
        build(dev, cfg, dict(w, **{"l0.mix.q": w["l0.mix.q"][:-1]}), "bfloat16")


def test_trace_runner_and_command_line(tmp_path):
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
    r = subprocess.run([f"{ROOT}/bin/trace_run", "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "80"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                       timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, 91)
    assert error(read(0), want[[0, 39]]) < 1e-4 and error(read(1), want[[40]]) < 1e-4 and error(read(3), want[[1]]) < 1e-4
    assert not (out / "2.f32").exists()
    r = subprocess.run([sys.executable, "-m", "tensorlogic_b200", "generate", "--model", str(tmp_path), "--dtype", "float32",
                        "--prompt", ",".join(map(str, seq[:20])), "--new", "4"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [int(t) for t in r.stdout.split()] == ref.greedy(cfg, w, seq[:20], 4)


def test_llama_files_through_the_registry(dev, tmp_path):
    from gguf_util import write_gguf
    from tensorlogic_b200 import registry
    from tensorlogic_b200.model import Llama, LlamaArch, synthetic_host_weights
    arch = LlamaArch(n_layers=2, d_model=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn_dim=512, vocab=512)
    p = tmp_path / "m.gguf"
    write_gguf(p, synthetic_host_weights(arch, seed=1), arch)
    r = registry.load(dev, str(p), max_seq=64, max_prefill=16)
    assert isinstance(r, Llama) and abs(r.arch.rms_eps - 1e-5) < 1e-9
    r.arch.rms_eps = arch.rms_eps        # the file holds 32 bits of it
    assert r.arch == arch
    out = list(registry.generate(r, [3, 1, 4, 1, 5], 6))
    assert len(out) == 6
    from tensorlogic_b200._lib import TensorError
    with pytest.raises(TensorError):
        registry.load(dev, str(p), "float32")
