"""Decoder, parts that need no GPU: the configuration reader, the registry, trace replay, and that the
oracle's mechanisms are told apart by the inputs the GPU tests use."""
import copy
import json

import numpy as np
import pytest

import decoder_ref as ref
from decoder_util import attention, config, dense, error, moe, shapes, tokens, weights, write_model


def test_config_reader_takes_every_size_from_the_file():
    from tensorlogic_b200 import toposun
    cfg = config([dense(attention(6, 3, 20, 11, 1, 8, 77.0, 0.31), 50, 2.5), moe(attention(2, 1, 12, 5, 0, 12), 7, 3, 18, 0),
                  moe(attention(), 4, 1, 8, 12), attention()], width=40, vocab=33, eps=3e-4)
    a = toposun.read_config(cfg)
    assert (a.width, a.vocab, a.norm_eps, len(a.layers)) == (40, 33, 3e-4, 4)
    l = a.layers[0]
    assert (l.heads, l.kv_heads, l.dim, l.window, l.keep_first, l.rot_dims, l.rot_base, l.scale) == (6, 3, 20, 11, 1, 8, 77.0, 0.31)
    assert (l.ff_kind, l.ff, l.limit) == ("clamped_glu", 50, 2.5)
    l = a.layers[1]
    assert (l.ff_kind, l.experts, l.top, l.expert_ff, l.shared_ff) == ("moe", 7, 3, 18, 0)
    assert a.layers[2].shared_ff == 12 and a.layers[3].ff_kind == "none"
    flat = {n: (1,) + s if len(s) == 1 else s for n, s in shapes(cfg).items()}
    assert a.tensor_shapes() == flat


@pytest.mark.parametrize("change", ["type", "kind", "vdim", "missing"])
def test_config_reader_refuses_what_it_does_not_know(change):
    from tensorlogic_b200 import toposun
    from tensorlogic_b200._lib import TensorError
    cfg = config([dense(attention())])
    layer = cfg["layers"][0]
    if change == "type":
        layer["type"] = "recurrent"
    elif change == "kind":
        layer["mlp"]["kind"] = "sparse"
    elif change == "vdim":
        layer["mixer"]["vdim"] = layer["mixer"]["dim"] + 8
    else:
        del layer["mixer"]["scale"]
    with pytest.raises(TensorError):
        toposun.read_config(cfg)


def test_registry_names_the_class(tmp_path, lib, capsys):
    from tensorlogic_b200 import __main__ as cli
    from tensorlogic_b200 import registry
    from tensorlogic_b200._lib import TensorError
    cfg = config([attention()])
    write_model(tmp_path, cfg, weights(cfg))
    assert registry.identify(str(tmp_path)) == ("Toposun", cfg)
    assert cli.main(["info", "--model", str(tmp_path)]) == 0
    assert "Toposun" in capsys.readouterr().out
    (tmp_path / "config.json").write_text(json.dumps(dict(cfg, architecture="Other")))
    with pytest.raises(TensorError):
        registry.identify(str(tmp_path))


def test_gguf_files_keep_their_class(tmp_path, lib):
    from gguf_util import write_gguf
    from tensorlogic_b200 import registry
    p = tmp_path / "m.gguf"
    write_gguf(p, {"output_norm.weight": (0, np.ones((1, 32)))})
    assert registry.identify(str(p)) == ("llama", None)


def test_the_decoder_part_of_the_library_is_complete(lib):
    """The part that serves decoder models alone loads and exports what their runner calls."""
    import ctypes
    import os
    from tensorlogic_b200 import build, registry
    assert registry.ARCHITECTURES["Toposun"].part == "decoder"
    path = build.build(part="decoder")
    assert path != build.LIB and os.path.exists(path)
    part = ctypes.CDLL(path, mode=os.RTLD_NOW)
    for name in ("tlc_init", "tlc_model_load_safetensors", "tlc_decoder_create", "tlc_decoder_prefill", "tlc_decoder_decode_host",
                 "tlc_decoder_release", "tlc_synchronize"):
        assert hasattr(part, name)
    assert not hasattr(part, "tlc_llama_create")


class FakeRunner:
    def __init__(self):
        self.free, self.seen, self.closed = [0], {}, []

    def open(self):
        return self.free.pop()

    def close(self, seq):
        self.closed.append(seq)
        self.free.append(seq)
        self.seen[seq] = []

    def feed(self, seq, toks, want):
        past = self.seen.setdefault(seq, [])
        rows = []
        for i, t in enumerate(toks):
            past.append(t)
            if i in want:
                rows.append([len(past), sum(past)])
        return np.array(rows, np.float32)


def test_trace_replay_writes_and_reports_every_step(tmp_path):
    from tensorlogic_b200 import trace
    steps = [{"step": 0, "entries": [{"id": "u", "tokens": [4, 5, 6], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "u", "tokens": [7], "want": []}], "end": ["u"]},
             {"step": 2, "entries": [{"id": "v", "tokens": [1, 2], "want": [1]}], "end": ["v"]}]
    said, r = [], FakeRunner()
    trace.replay(r, [json.dumps(s) + "\n" for s in steps], str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and r.closed == [0, 0]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [1, 4, 3, 15]
    assert not (tmp_path / "1.f32").exists()
    assert np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [2, 3]


# ---- the oracle ---------------------------------------------------------------------------------

def test_rotation_keeps_distances_and_lengths():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 1, 10)), rng.standard_normal((1, 1, 10))

    def score(p, j):
        return float((ref.rotate_half(q, [p], 6, 100.0) * ref.rotate_half(k, [j], 6, 100.0)).sum())
    assert abs(score(7, 3) - score(104, 100)) < 1e-9
    assert abs(np.linalg.norm(ref.rotate_half(q, [5], 6, 100.0)) - np.linalg.norm(q)) < 1e-12
    r = ref.rotate_half(q, [2], 6, 100.0)[0, 0]
    a = 2 * 100.0 ** (-2 / 6)
    assert abs(r[1] - (q[0, 0, 1] * np.cos(a) - q[0, 0, 4] * np.sin(a))) < 1e-12
    assert abs(r[4] - (q[0, 0, 4] * np.cos(a) + q[0, 0, 1] * np.sin(a))) < 1e-12
    assert np.array_equal(r[6:], q[0, 0, 6:])


def test_visible_keys_by_counting():
    seen = [[j for j in range(12) if ref.visible(i, j, 3, 2)] for i in range(12)]
    assert seen[1] == [0, 1] and seen[3] == [0, 1, 2, 3] and seen[4] == [0, 1, 2, 3, 4] and seen[5] == [0, 1, 3, 4, 5]
    assert seen[11] == [0, 1, 9, 10, 11]


def test_attention_core_against_one_loop():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 4, 6)), rng.standard_normal((9, 2, 6)), rng.standard_normal((9, 2, 5))
    out = ref.attention_core(q, k, v, np.arange(9), 0.7, 3, 1)
    for i in range(9):
        for h in range(4):
            js = [j for j in range(9) if ref.visible(i, j, 3, 1)]
            e = np.exp([0.7 * float(q[i, h] @ k[j, h // 2]) for j in js])
            want = sum(c * v[j, h // 2] for c, j in zip(e / e.sum(), js))
            assert np.allclose(out[i, h], want)


def test_clamped_glu_by_hand():
    out = ref.clamped_glu(np.array([3.0, -4.0, 0.5]), np.array([9.0, -9.0, 0.25]), 2.0)
    s = lambda z: 1 / (1 + np.exp(-z))
    assert np.allclose(out, [2 * s(3.404) * 3.0, -4 * s(-6.808) * -1.0, 0.5 * s(0.851) * 1.25])


def test_expert_weight_scales_the_input():
    cfg = config([moe(attention(), experts=3, top=2, ff=8, shared=0)])
    w = {k: v.astype(np.float64) for k, v in weights(cfg, 3).items()}
    h = np.random.default_rng(5).standard_normal((2, 48))
    out = ref.moe_ff(h, w, "l0.mlp.", cfg["layers"][0]["mlp"])
    for t in range(2):
        s = ref.sigmoid(w["l0.mlp.router"] @ h[t])
        want = 0
        for e in np.argsort(-s)[:2]:
            x = s[e] * h[t]
            g = w[f"l0.mlp.e{e}.gate"] @ x
            want = want + w[f"l0.mlp.e{e}.down"] @ (g / (1 + np.exp(-g)) * (w[f"l0.mlp.e{e}.up"] @ x))
        assert np.allclose(out[t], want)


MISTAKES = {
    "window + 1": lambda m: m["mask"].__setitem__("size", m["mask"]["size"] + 1),
    "window - 1": lambda m: m["mask"].__setitem__("size", m["mask"]["size"] - 1),
    "kept + 1": lambda m: m["mask"].__setitem__("keep_first", m["mask"]["keep_first"] + 1),
    "kept - 1": lambda m: m["mask"].__setitem__("keep_first", m["mask"]["keep_first"] - 1),
    "scale": lambda m: m.__setitem__("scale", m["scale"] * 1.2),
    "base": lambda m: m["rot"].__setitem__("base", m["rot"]["base"] * 1.5),
    "rotated": lambda m: m["rot"].__setitem__("dims", m["rot"]["dims"] - 2),
}


@pytest.mark.parametrize("name", sorted(MISTAKES))
def test_planted_mistakes_show(name):
    """With sharp scores (a large scale) an edge that is one token off moves the logits far beyond the
    tolerances of the GPU tests."""
    cfg = config([attention(window=9, keep=2, scale=2.0), attention(window=9, keep=2, scale=2.0)])
    w, seq = weights(cfg, 11), tokens(60, 61)
    bad = copy.deepcopy(cfg)
    for l in bad["layers"]:
        MISTAKES[name](l["mixer"])
    assert error(ref.forward(bad, w, seq), ref.forward(cfg, w, seq)) > 0.1
