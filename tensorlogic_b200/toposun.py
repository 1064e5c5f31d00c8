"""Toposun: reader of its config.json.

Layers of grouped-query attention (sliding window with kept first tokens, values = keys, norm over
the whole query / key projection, half-split rotation) in parallel with a clamped GLU, a mixture of
experts or nothing, under two layer norms; the embedding table is the output projection too.
"""
from __future__ import annotations

from ._lib import ERR_LOAD, TensorError
from .decoder import DecoderArch, LayerArch

NAME = "Toposun"


def _get(d: dict, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise TensorError(ERR_LOAD, f"{NAME} configuration: {where} has no '{key}'")
    return d[key]


def _layer(entry: dict, at: str) -> LayerArch:
    kind = _get(entry, "type", at)
    if kind != "attention":
        raise TensorError(ERR_LOAD, f"{NAME} configuration: {at} is of type '{kind}' (known: attention)")
    mix = _get(entry, "mixer", at)
    at = at + ".mixer"
    dim = int(_get(mix, "dim", at))
    if int(mix.get("vdim", dim)) != dim:
        raise TensorError(ERR_LOAD, f"{NAME} configuration: {at}: values are the keys, vdim {mix['vdim']} is not dim {dim}")
    mask, rot = _get(mix, "mask", at), _get(mix, "rot", at)
    arch = LayerArch(int(_get(mix, "heads", at)), int(_get(mix, "kv_heads", at)), dim, int(_get(mask, "size", at + ".mask")),
                     int(_get(mask, "keep_first", at + ".mask")), int(_get(rot, "dims", at + ".rot")),
                     float(_get(rot, "base", at + ".rot")), float(_get(mix, "scale", at)))
    mlp = entry.get("mlp")
    if mlp is None:
        return arch
    at = at[:-len("mixer")] + "mlp"
    kind = _get(mlp, "kind", at)
    if kind == "dense":
        arch.ff_kind, arch.ff, arch.limit = "clamped_glu", int(_get(mlp, "ff", at)), float(_get(mlp, "limit", at))
    elif kind == "moe":
        router = _get(mlp, "router", at)
        arch.ff_kind = "moe"
        arch.experts, arch.top = int(_get(router, "experts", at + ".router")), int(_get(router, "top", at + ".router"))
        arch.expert_ff = int(_get(_get(mlp, "expert", at), "ff", at + ".expert"))
        if mlp.get("shared") is not None:
            arch.shared_ff = int(_get(mlp["shared"], "ff", at + ".shared"))
    else:
        raise TensorError(ERR_LOAD, f"{NAME} configuration: {at} is of kind '{kind}' (known: dense, moe)")
    return arch


def read_config(cfg: dict) -> DecoderArch:
    layers = [_layer(e, f"layers[{i}]") for i, e in enumerate(_get(cfg, "layers", "config"))]
    return DecoderArch(int(_get(cfg, "width", "config")), int(_get(cfg, "vocab", "config")),
                       float(_get(_get(cfg, "norm", "config"), "eps", "norm")), layers)
