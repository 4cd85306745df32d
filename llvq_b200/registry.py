"""Which class serves a model. A model is a sealed archive file (LLVQ codes with its config.json inside) or a folder
with config.json and model.safetensors; config.json names the architecture. `load_model` is the one way in for the
command line and for trace replay.

An architecture registers a loader `fn(config, source, dtype, capacity, device, **options)`: `source` is the opened
archive or the folder's SafetensorsFile, and the result is a TokenLoop.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Tuple


class UnsupportedDtype(ValueError):
    """The architecture is known but does not run in the element type asked for."""


@dataclass(frozen=True)
class Architecture:
    name: str
    container: str           # "archive" or "folder"
    dtypes: Tuple[str, ...]
    load: Callable


_ARCHITECTURES: Dict[str, Architecture] = {}


def register(name: str, container: str, dtypes: Tuple[str, ...], aliases: Tuple[str, ...] = ()):
    def add(fn):
        arch = Architecture(name, container, dtypes, fn)
        for n in (name, *aliases):
            _ARCHITECTURES[n.lower()] = arch
        return fn
    return add


def architectures() -> Dict[str, Architecture]:
    from . import hybrid, latent, model  # noqa: F401  (they register themselves)
    return dict(_ARCHITECTURES)


def architecture_of(config: dict, default: str = "") -> Architecture:
    """By `architecture`, else the first of `architectures`, else `model_type`."""
    names = [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type"), default]
    known = architectures()
    for n in names:
        if n and n.lower() in known:
            return known[n.lower()]
    raise ValueError(f"config.json names no known architecture ({[n for n in names if n]}); known: {sorted(known)}")


def load_model(path: str, capacity: int, dtype: str = "", device: int = 0, **options):
    """A TokenLoop with room for `capacity` tokens. `dtype` "" takes the architecture's own."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            config = json.load(f)
        arch, source, container = architecture_of(config), None, "folder"
    else:
        from .archive import LvqArchive
        source = LvqArchive(path=path)
        blobs = dict(source.blob(i) for i in range(source.n_blobs))
        if "config.json" not in blobs:
            raise ValueError(f"{path} carries no config.json: not a sealed, self-contained file")
        config, container = json.loads(blobs["config.json"]), "archive"
        arch = architecture_of(config, default="qwen3")
    if arch.container != container:
        raise ValueError(f"{arch.name} is served from a {arch.container}, {path} is a {container}")
    if dtype and dtype not in arch.dtypes:
        raise UnsupportedDtype(f"{arch.name} runs in {', '.join(arch.dtypes)}, not in {dtype}")
    if source is None:
        from .safetensors import SafetensorsFile
        source = SafetensorsFile(os.path.join(path, "model.safetensors"))
    return arch.load(config, source, dtype or arch.dtypes[0], capacity, device, **options)
