"""Which model class serves which files.

    load(dev, path, dtype=None, **options) -> runner

``path`` is a GGUF file, whose ``general.architecture`` names the model, or a folder with config.json
(its ``architecture``) and model.safetensors.  Every runner has prefill / decode / set_sampling;
``generate`` drives any of them.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Iterator, Sequence

from . import decoder, suselorn, toposun
from ._lib import ERR_LOAD, TensorError
from .api import Device
from .model import Llama, LlamaArch, load_model


@dataclass(frozen=True)
class Entry:
    dtypes: tuple[str, ...]              # what a runner can compute in; the first is the default
    load: Callable[..., object]          # (dev, path, config or None, dtype, options) -> runner
    part: str | None = None              # the part of the library that is enough (build.PARTS); None: all of it


def _llama(dev: Device, path: str, _config, _dtype: str, options: dict) -> Llama:
    model = load_model(dev, path)
    options = {k: v for k, v in options.items() if k in ("max_seq", "max_batch", "max_prefill", "use_graph", "logits_all_rows")}
    return Llama(dev, model, LlamaArch.from_model(model), **options)


def _decoder(read_config) -> Callable[..., object]:
    def load(dev: Device, path: str, config: dict, dtype: str, options: dict) -> decoder.Decoder:
        arch = read_config(config)
        model = decoder.load_safetensors(dev, os.path.join(path, "model.safetensors"), dtype)
        return decoder.Decoder(dev, model, arch, dtype, **options)
    return load


ARCHITECTURES: dict[str, Entry] = {
    "llama": Entry(("float16",), _llama),
    toposun.NAME: Entry(decoder.Decoder.dtypes, _decoder(toposun.read_config), "decoder"),
    suselorn.NAME: Entry(decoder.Decoder.dtypes, _decoder(suselorn.read_config), "decoder"),
}


def identify(path: str) -> tuple[str, dict | None]:
    """(architecture, config.json's contents or None for a GGUF file)."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
        name = config.get("architecture")
    else:
        import ctypes as C
        from . import _lib
        lib, g = _lib.load(), C.c_void_p()
        _lib.check(lib.tlc_gguf_open(str(path).encode(), C.byref(g)))
        raw = lib.tlc_gguf_meta_str(g, b"general.architecture")
        name, config = (raw.decode() if raw else None), None
        lib.tlc_gguf_close(g)
    if name not in ARCHITECTURES:
        raise TensorError(ERR_LOAD, f"'{path}': unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return name, config


def load(dev: Device, path: str, dtype: str | None = None, **options):
    """The runner for the model at ``path`` (options: max_seq, max_batch, max_prefill, ...)."""
    path = str(path)
    name, config = identify(path)
    entry = ARCHITECTURES[name]
    dtype = dtype or entry.dtypes[0]
    if dtype not in entry.dtypes:
        raise TensorError(ERR_LOAD, f"{name} models run in {', '.join(entry.dtypes)}, not in {dtype}")
    return entry.load(dev, path, config, dtype, options)


def generate(runner, prompt: Sequence[int], max_new_tokens: int, stop: Sequence[int] = ()) -> Iterator[int]:
    """Continues ``prompt`` token by token (sampling as set on the runner), up to a token of ``stop``."""
    token, _ = runner.prefill(list(prompt), return_logits=False)
    for i in range(max_new_tokens):
        yield int(token)
        if token in stop or i + 1 == max_new_tokens:
            return
        token = int(runner.decode([token])[0][0])
