"""Small Suselorn configurations and random weights."""
import numpy as np

from decoder_util import bf16_round


def latent(heads=4, dim=16, rot=8, vdim=16, q_rank=24, kv_rank=16, base=300.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "rot": {"dims": rot, "base": base}, "scale": (dim + rot) ** -0.5 if scale is None else scale},
            "mlp": None}


def dense(layer, ff=40):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def config(layers, width=48, vocab=61, streams=3, softcap=9.0, eps=1e-5, loop=None):
    cfg = {"architecture": "Suselorn", "layers": layers, "logit_softcap": softcap, "norm": {"eps": eps}, "streams": streams,
           "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def shapes(cfg):
    w, s = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], w)}

    def norm(name):
        out.update({name: (w,), name + ".b": (w,), name + ".alpha": ()})
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        h = m["heads"]
        x = p + "mix."
        out.update({x + "dq": (m["q_rank"], w), x + "dq.norm": (m["q_rank"],), x + "uq": (h * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                    x + "dkv": (m["kv_rank"] + m["rot_dim"], w), x + "dkv.norm": (m["kv_rank"],),
                    x + "uk": (h * m["dim"], m["kv_rank"]), x + "uv": (h * m["vdim"], m["kv_rank"]), x + "sink": (h,),
                    x + "o": (w, h * m["vdim"])})
        for q in (1, 2) if l["mlp"] else (1,):
            norm(f"{p}norm{q}")
            out.update({f"{p}ls{q}": (w,), f"{p}hc{q}.in": (s,), f"{p}hc{q}.out": (s,), f"{p}hc{q}.mix": (s, s)})
        if l["mlp"]:
            ff, x = l["mlp"]["ff"], p + "mlp."
            out.update({x + "gate": (ff, w), x + "gate.b": (ff,), x + "up": (ff, w), x + "up.b": (ff,), x + "down": (w, ff),
                        x + "down.b": (w,)})
    return out


def weights(cfg, seed=0, gain=1.0):
    """bf16-valued random weights; ``gain`` multiplies the matrices."""
    rng = np.random.default_rng(seed)
    s, out = cfg["streams"], {}
    for name, shape in shapes(cfg).items():
        a, last = rng.standard_normal(shape), name.rsplit(".", 1)[-1]
        if last == "alpha":
            a = 0.7 + 0.2 * a
        elif last == "in":
            a = (1.0 + 0.4 * a) / s
        elif last == "out":
            a = 0.7 + 0.3 * a
        elif last == "mix":
            a = 0.8 * np.eye(s) + 0.25 * a
        elif last == "sink":
            a = 1.0 + a
        elif last in ("ls1", "ls2"):
            a = 1.0 + 0.3 * a
        elif last == "b":
            a = 0.3 * a
        elif "norm" in name:
            a = 1.0 + 0.2 * a
        elif name != "embed":
            a = a * gain * shape[-1] ** -0.5
        out[name] = bf16_round(a).reshape(shape)
    return out


def silence(w, layer, mixer=False, ff=False):
    """Makes a sublayer add nothing (the streams still mix)."""
    for q, on in ((1, mixer), (2, ff)):
        if on:
            w[f"l{layer}.ls{q}"][:] = 0
    return w


def plain_streams(w, layer, streams):
    """The streams of both sublayers: u is the first stream, every stream receives y."""
    for q in (1, 2):
        if f"l{layer}.hc{q}.in" in w:
            w[f"l{layer}.hc{q}.in"][:] = np.eye(streams)[0]
            w[f"l{layer}.hc{q}.out"][:] = 1
            w[f"l{layer}.hc{q}.mix"][:] = np.eye(streams)
    return w
