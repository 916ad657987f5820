"""Which class reads a checkpoint, and which engine serves it.

A checkpoint names its architecture in the ``config.json`` of its folder (``"architecture"``); a single
``.safetensors`` / ``.pt`` file is a speech checkpoint in the reference's format (src/vui/model.py:1155-1219 in
fluxions-ai/vui).  A model class is added with ``register``; model and engine modules are imported when first needed.
"""

from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass

SPEECH = "Vui"


@dataclass(frozen=True)
class Entry:
    model: str    # "module:class" with from_checkpoint(path, device=..., **kw)
    engine: str   # "module:class" taking (model=..., max_rows=..., max_seq=..., ...)


_REGISTRY: dict[str, Entry] = {}


def register(architecture: str, model: str, engine: str) -> None:
    _REGISTRY[architecture] = Entry(model, engine)


def architectures() -> list[str]:
    return sorted(_REGISTRY)


def architecture_of(path: str) -> str:
    if not os.path.isdir(path):
        return SPEECH
    with open(os.path.join(path, "config.json")) as f:
        name = json.load(f).get("architecture")
    if name not in _REGISTRY:
        raise ValueError(f"'{path}' has architecture {name!r}; known are {', '.join(architectures())}")
    return name


def _resolve(spec: str):
    mod, cls = spec.split(":")
    return getattr(importlib.import_module(mod, __package__), cls)


def load_model(path: str, device="cuda", **kw):
    """The model at ``path``, as the class its configuration names."""
    return _resolve(_REGISTRY[architecture_of(path)].model).from_checkpoint(path, device=device, **kw)


def open_engine(model, **kw):
    """An engine for a model object, or for a checkpoint path (loaded first; ``dtype=`` goes to the loader)."""
    if isinstance(model, (str, os.PathLike)):
        load_kw = {k: kw.pop(k) for k in ("device", "dtype") if k in kw}
        model = load_model(os.fspath(model), **load_kw)
    return _resolve(_REGISTRY[model.architecture].engine)(model=model, **kw)


register(SPEECH, ".model:VuiB200", ".engine:Engine")
register("Vidotar", ".token_lm:Vidotar", ".token_engine:TokenEngine")
register("Medirax", ".token_lm:Medirax", ".token_engine:TokenEngine")
