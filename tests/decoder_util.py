"""Small configurations, random weights, files and ways to feed a runner for the decoder tests."""
import json
import struct

import numpy as np


def bf16_round(a):
    """Nearest bf16 (ties to even) as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.view(np.float32)


def attention(heads=4, kv=2, dim=16, window=9, keep=2, rot=None, base=500.0, scale=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "mask": {"size": window, "keep_first": keep},
                      "rot": {"dims": dim if rot is None else rot, "base": base},
                      "scale": dim ** -0.5 if scale is None else scale},
            "mlp": None}


def dense(layer, ff=40, limit=1.5):
    return dict(layer, mlp={"kind": "dense", "ff": ff, "limit": limit})


def moe(layer, experts=5, top=2, ff=24, shared=16):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return dict(layer, mlp=m)


def config(layers, width=48, vocab=61, eps=1e-5):
    return {"architecture": "Toposun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def shapes(cfg):
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "final.norm": (w,)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        q, k = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        out.update({p + "norm1": (w,), p + "mix.q": (q, w), p + "mix.q.b": (q,), p + "mix.q.norm": (q,), p + "mix.k": (k, w),
                    p + "mix.k.b": (k,), p + "mix.k.norm": (k,), p + "mix.o": (w, q), p + "mix.o.b": (w,)})
        mlp = l.get("mlp")
        if not mlp:
            continue
        out[p + "norm2"] = (w,)
        units = [(p + "mlp.", mlp["ff"])] if mlp["kind"] == "dense" else []
        if mlp["kind"] == "moe":
            out[p + "mlp.router"] = (mlp["router"]["experts"], w)
            units += [(f"{p}mlp.e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            if mlp.get("shared"):
                units.append((p + "mlp.shared.", mlp["shared"]["ff"]))
                out[p + "mlp.shared.sg"] = (1, w)
        for at, n in units:
            out.update({at + "gate": (n, w), at + "up": (n, w), at + "down": (w, n)})
    return out


def weights(cfg, seed=0, gain=1.0):
    """bf16-valued random weights; ``gain`` multiplies the matrices."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        a = rng.standard_normal(shape)
        if "norm" in name:
            a = 1.0 + 0.2 * a
        elif name.endswith(".b"):
            a = 0.3 * a
        elif name == "embed":
            a = a.astype(np.float32)
        else:
            a = a * gain * shape[-1] ** -0.5
        out[name] = bf16_round(a)
    return out


def tokens(n, vocab, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, vocab, n).tolist()


def write_safetensors(path, tensors, dtype="BF16"):
    head, blobs, at = {"__metadata__": {"made by": "a \"test\" \\u00e9"}}, [], 0
    for name, a in tensors.items():
        a = np.ascontiguousarray(a, np.float32)
        raw = (a.view(np.uint32) >> 16).astype("<u2").tobytes() if dtype == "BF16" else \
            a.astype("<f2").tobytes() if dtype == "F16" else a.astype("<f4").tobytes()
        head[name] = {"dtype": dtype, "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    text += b" " * (-len(text) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))


def write_model(folder, cfg, w, dtype="BF16"):
    with open(folder / "config.json", "w") as f:
        json.dump(cfg, f)
    write_safetensors(folder / "model.safetensors", w, dtype)


def error(got, want):
    """Worst row: root mean square of the difference (mean taken off) over the rows' typical size."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape, (got.shape, want.shape)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    size = np.sqrt(((want - want.mean(-1, keepdims=True)) ** 2).mean())
    return float(np.sqrt((d * d).mean(-1)).max() / size)


# ---- ways to feed a sequence to a runner -------------------------------------------------------------

def whole(dec, seq):
    s = dec.open()
    out = dec.feed(s, seq, range(len(seq)))
    dec.close(s)
    return out


def one_by_one(dec, seq, first=1):
    s = dec.open()
    rows = [dec.feed(s, seq[:first], range(first))]
    rows += [dec.feed(s, [t], [0]) for t in seq[first:]]
    dec.close(s)
    return np.concatenate(rows)


def portions(dec, seq, sizes):
    s, at, rows = dec.open(), 0, []
    for n in sizes:
        part = seq[at:at + n]
        if len(part):
            rows.append(dec.feed(s, part, range(len(part))))
        at += n
    assert at >= len(seq)
    dec.close(s)
    return np.concatenate(rows)
