"""Suselorn: reader of its config.json.

Layers of latent attention (queries and keys / values through normalized latents, a rotated key part all
heads share, a softmax sink per head) and SiLU GLU feed-forwards over several residual streams
(hyper-connections) under tanh norms, with layer scales; a stretch of layers may run several times;
the embedding table is the output projection too, under a soft cap of the logits.
"""
from __future__ import annotations

from ._lib import ERR_LOAD, TensorError
from .decoder import DecoderArch, LatentLayerArch

NAME = "Suselorn"


def _refuse(what: str):
    raise TensorError(ERR_LOAD, f"{NAME} configuration: {what}")


def _get(d: dict, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        _refuse(f"{where} has no '{key}'")
    return d[key]


def _layer(entry: dict, at: str) -> LatentLayerArch:
    kind = _get(entry, "type", at)
    if kind != "latent_attention":
        _refuse(f"{at} is of type '{kind}' (known: latent_attention)")
    mix = _get(entry, "mixer", at)
    m = at + ".mixer"
    rot, rot_dim = _get(mix, "rot", m), int(_get(mix, "rot_dim", m))
    if int(_get(rot, "dims", m + ".rot")) != rot_dim:
        _refuse(f"{m}: the whole rotated part turns, rot.dims {rot['dims']} is not rot_dim {rot_dim}")
    arch = LatentLayerArch(int(_get(mix, "heads", m)), int(_get(mix, "dim", m)), rot_dim, int(_get(mix, "vdim", m)),
                           int(_get(mix, "q_rank", m)), int(_get(mix, "kv_rank", m)), float(_get(rot, "base", m + ".rot")),
                           float(_get(mix, "scale", m)))
    mlp = entry.get("mlp")
    if mlp is not None:
        kind = _get(mlp, "kind", at + ".mlp")
        if kind != "dense":
            _refuse(f"{at}.mlp is of kind '{kind}' (known: dense)")
        arch.ff_kind, arch.ff = "silu_glu", int(_get(mlp, "ff", at + ".mlp"))
    return arch


def _runs(loop, n: int) -> list[int]:
    if loop is None:
        return list(range(n))
    start, stop, times = (int(_get(loop, k, "loop")) for k in ("start", "stop", "times"))
    if not (0 <= start <= stop <= n and times >= 1):
        _refuse(f"loop of layers {start} .. {stop}, {times} times, over {n} layers")
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


def read_config(cfg: dict) -> DecoderArch:
    layers = [_layer(e, f"layers[{i}]") for i, e in enumerate(_get(cfg, "layers", "config"))]
    return DecoderArch(int(_get(cfg, "width", "config")), int(_get(cfg, "vocab", "config")),
                       float(_get(_get(cfg, "norm", "config"), "eps", "norm")), layers, streams=int(_get(cfg, "streams", "config")),
                       logit_softcap=float(_get(cfg, "logit_softcap", "config")), runs=_runs(cfg.get("loop"), len(layers)))
