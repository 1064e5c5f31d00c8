"""Suselorn, parts that need no GPU: the configuration reader, the registry, and that the oracle's mechanisms
are what they are meant to be and are told apart by the inputs the GPU tests use."""
import copy
import math

import numpy as np
import pytest

import suselorn_ref as ref
from decoder_util import error, tokens, write_model
from suselorn_util import config, dense, latent, shapes, weights


def test_config_reader_takes_every_size_from_the_file():
    from tensorlogic_b200 import suselorn
    cfg = config([dense(latent(6, 20, 10, 12, 28, 36, 77.0, 0.31), 50), latent(2, 12, 4, 14, 9, 11)], width=40, vocab=33, streams=5,
                 softcap=12.5, eps=3e-4, loop=(1, 2, 3))
    a = suselorn.read_config(cfg)
    assert (a.width, a.vocab, a.norm_eps, a.streams, a.logit_softcap, a.runs) == (40, 33, 3e-4, 5, 12.5, [0, 1, 1, 1])
    l = a.layers[0]
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.rot_base, l.scale) == (6, 20, 10, 12, 28, 36, 77.0, 0.31)
    assert (l.ff_kind, l.ff) == ("silu_glu", 50) and a.layers[1].ff_kind == "none"
    flat = {n: (1, 1) if s == () else (1,) + s if len(s) == 1 else s for n, s in shapes(cfg).items()}
    assert a.tensor_shapes() == flat


@pytest.mark.parametrize("loop,runs", [(None, [0, 1, 2, 3]), ((0, 4, 1), [0, 1, 2, 3]), ((1, 3, 3), [0, 1, 2, 1, 2, 1, 2, 3]),
                                       ((0, 4, 2), [0, 1, 2, 3] * 2), ((3, 4, 2), [0, 1, 2, 3, 3]), ((2, 2, 5), [0, 1, 2, 3])])
def test_order_of_a_loop(loop, runs):
    from tensorlogic_b200 import suselorn
    cfg = config([latent() for _ in range(4)], loop=loop)
    assert suselorn.read_config(cfg).runs == runs and ref.order(cfg) == runs


@pytest.mark.parametrize("change", ["type", "kind", "rot", "missing", "streams", "loop"])
def test_config_reader_refuses_what_it_does_not_know(change):
    from tensorlogic_b200 import suselorn
    from tensorlogic_b200._lib import TensorError
    cfg = config([dense(latent())], loop=(0, 1, 2))
    layer = cfg["layers"][0]
    if change == "type":
        layer["type"] = "recurrent"
    elif change == "kind":
        layer["mlp"]["kind"] = "moe"
    elif change == "rot":
        layer["mixer"]["rot"]["dims"] = 4
    elif change == "missing":
        del layer["mixer"]["kv_rank"]
    elif change == "streams":
        del cfg["streams"]
    else:
        cfg["loop"]["stop"] = 3
    with pytest.raises(TensorError):
        suselorn.read_config(cfg)


def test_registry_names_the_class(tmp_path, lib, capsys):
    from tensorlogic_b200 import __main__ as cli
    from tensorlogic_b200 import registry
    cfg = config([latent()])
    write_model(tmp_path, cfg, weights(cfg))
    assert registry.identify(str(tmp_path)) == ("Suselorn", cfg)
    assert registry.ARCHITECTURES["Suselorn"].part == "decoder"
    assert cli.main(["info", "--model", str(tmp_path)]) == 0
    assert "Suselorn" in capsys.readouterr().out


# ---- the oracle ---------------------------------------------------------------------------------

def test_neighbours_rotate_together():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 1, 6)), rng.standard_normal((1, 1, 6))

    def score(p, j):
        return float((ref.rotate_pairs(q, [p], 50.0) * ref.rotate_pairs(k, [j], 50.0)).sum())
    assert abs(score(7, 3) - score(104, 100)) < 1e-9 and abs(score(7, 3) - score(7, 4)) > 1e-3
    r, a = ref.rotate_pairs(q, [2], 50.0)[0, 0], 2 * 50.0 ** (-2 / 6)
    assert abs(r[2] - (q[0, 0, 2] * math.cos(a) - q[0, 0, 3] * math.sin(a))) < 1e-12
    assert abs(r[3] - (q[0, 0, 3] * math.cos(a) + q[0, 0, 2] * math.sin(a))) < 1e-12


def test_sink_takes_weight_and_gives_nothing():
    w = ref.softmax_with_sink(np.array([0.5, -np.inf, 2.0]), 1.0)
    z = math.exp(0.5) + math.exp(2.0) + math.exp(1.0)
    assert np.allclose(w, [math.exp(0.5) / z, 0.0, math.exp(2.0) / z])
    assert np.allclose(ref.softmax_with_sink(np.array([900.0, 899.0]), -900.0).sum(), 1.0)


def test_latent_attention_against_one_loop():
    cfg = config([latent(3, 6, 4, 5, 7, 8)])
    mix, w = cfg["layers"][0]["mixer"], {k: v.astype(np.float64) for k, v in weights(cfg, 2).items()}
    h, m = np.random.default_rng(4).standard_normal((5, 48)), "l0.mix."
    out = ref.latent_attention(h, w, m, mix, 1e-5)

    def norm(v, g):
        return v / np.sqrt(np.mean(v * v) + 1e-5) * g

    def turn(v, pos):
        return np.concatenate([[v[2 * i] * math.cos(pos * 300.0 ** (-i / 2)) - v[2 * i + 1] * math.sin(pos * 300.0 ** (-i / 2)),
                                v[2 * i + 1] * math.cos(pos * 300.0 ** (-i / 2)) + v[2 * i] * math.sin(pos * 300.0 ** (-i / 2))]
                               for i in range(2)])
    for t in range(5):
        heads = []
        q = w[m + "uq"] @ norm(w[m + "dq"] @ h[t], w[m + "dq.norm"])
        for n in range(3):
            qn, qr = q[10 * n:10 * n + 6], turn(q[10 * n + 6:10 * n + 10], t)
            e, vals = [], []
            for j in range(t + 1):
                z = w[m + "dkv"] @ h[j]
                c = norm(z[:8], w[m + "dkv.norm"])
                e.append(math.exp(mix["scale"] * float(qn @ (w[m + "uk"][6 * n:6 * n + 6] @ c) + qr @ turn(z[8:], j))))
                vals.append(w[m + "uv"][5 * n:5 * n + 5] @ c)
            heads.append(sum(a * v for a, v in zip(e, vals)) / (sum(e) + math.exp(w[m + "sink"][n])))
        assert np.allclose(out[t], w[m + "o"] @ np.concatenate(heads))


def test_streams_by_hand():
    rng = np.random.default_rng(5)
    x = rng.standard_normal((2, 3, 4))
    w = {"in": np.array([0.5, -1.0]), "out": np.array([2.0, 3.0]), "mix": np.array([[1.0, 0.25], [-0.5, 0.75]])}
    out = ref.hyper(x, w, "", lambda u: 10 * u)
    y = 10 * (0.5 * x[0] - x[1])
    assert np.allclose(out[0], x[0] - 0.5 * x[1] + 2 * y)
    assert np.allclose(out[1], 0.25 * x[0] + 0.75 * x[1] + 3 * y)


def test_feed_forward_norm_and_cap_by_hand():
    w = {"gate": np.array([[2.0]]), "gate.b": np.array([1.0]), "up": np.array([[-1.0]]), "up.b": np.array([0.5]), "down": np.array([[3.0]]),
         "down.b": np.array([0.25])}
    z = 2 * 1.5 + 1
    assert np.allclose(ref.silu_glu(np.array([[1.5]]), w, ""), 3 * (z / (1 + math.exp(-z)) * (-1.5 + 0.5)) + 0.25)
    assert np.allclose(ref.tanh_norm(np.array([0.3, -4.0]), 0.5, np.array([2.0, 1.0]), np.array([0.1, 0.2])),
                       [2 * math.tanh(0.15) + 0.1, math.tanh(-2.0) + 0.2])
    assert np.allclose(ref.softcap(np.array([40.0]), 8.0), 8 * math.tanh(5.0))


def _no_sink(cfg, w):
    for n in w:
        if n.endswith("sink"):
            w[n] = w[n] * 0 - 1e9


def _transposed_mix(cfg, w):
    for n in w:
        if n.endswith(".mix"):
            w[n] = w[n].T


def _halves(cfg, w):
    """The rotated entries in the order a half-split rotation would pair them."""
    for i, l in enumerate(cfg["layers"]):
        m = l["mixer"]
        order = np.arange(m["rot_dim"]).reshape(2, -1).T.reshape(-1)
        q = w[f"l{i}.mix.uq"].reshape(m["heads"], m["dim"] + m["rot_dim"], -1).copy()
        q[:, m["dim"]:] = q[:, m["dim"]:][:, order]
        w[f"l{i}.mix.uq"] = q.reshape(w[f"l{i}.mix.uq"].shape)
        kv = w[f"l{i}.mix.dkv"].copy()
        kv[m["kv_rank"]:] = kv[m["kv_rank"]:][order]
        w[f"l{i}.mix.dkv"] = kv


def _ones(*ends):
    def change(cfg, w):
        for n in w:
            if n.endswith(ends):
                w[n] = np.ones_like(w[n])
    return change


def _zeros(*ends):
    def change(cfg, w):
        for n in w:
            if n.endswith(ends):
                w[n] = np.zeros_like(w[n])
    return change


def _mixer(key, factor):
    def change(cfg, w):
        for l in cfg["layers"]:
            if key == "base":
                l["mixer"]["rot"]["base"] *= factor
            else:
                l["mixer"][key] *= factor
    return change


MISTAKES = {
    "no sink": _no_sink, "mix by [to, from]": _transposed_mix, "half-split rotation": _halves, "base": _mixer("base", 1.5),
    "scale": _mixer("scale", 1.2), "no scale of the mixer": _ones("ls1"), "no scale of the feed-forward": _ones("ls2"),
    "no weight of the query norm": _ones("dq.norm"), "no weight of the latent norm": _ones("dkv.norm"),
    "no norm bias": _zeros("norm1.b", "norm2.b", "final.norm.b"), "no alpha": _ones("alpha"), "no gate bias": _zeros("gate.b"),
    "no up bias": _zeros("up.b"), "no down bias": _zeros("down.b"),
    "one pass less": lambda cfg, w: cfg["loop"].__setitem__("times", 1),
    "cap": lambda cfg, w: cfg.__setitem__("logit_softcap", 1e6),
    "streams in": _ones("hc1.in", "hc2.in"), "streams out": _ones("hc1.out", "hc2.out"),
}


@pytest.mark.parametrize("name", sorted(MISTAKES))
def test_planted_mistakes_show(name):
    """What the GPU tests' tolerances (0.04 at most) must be able to tell apart."""
    cfg = config([dense(latent(scale=1.0)), latent(3, 12, 6, 10, 20, 14, scale=1.0)], loop=(0, 2, 2))
    w, seq = weights(cfg, 11), tokens(60, 61)
    bad, bw = copy.deepcopy(cfg), {k: v.copy() for k, v in w.items()}
    MISTAKES[name](bad, bw)
    assert error(ref.forward(bad, bw, seq), ref.forward(cfg, w, seq)) > 0.08
