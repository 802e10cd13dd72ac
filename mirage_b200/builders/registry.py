"""Which runner serves a checkpoint: the architecture its config.json names -> runner class."""
from __future__ import annotations

import json
import os
from typing import Tuple

import torch

# architecture name -> (runner class in builders.runner, kernel family it runs on, activation types)
_RUNNERS = {
    "bebuzen": ("BebuzenRunner", "hybrid", (torch.bfloat16, torch.float32)),
    "lofirax": ("LofiraxRunner", "hybrid", (torch.bfloat16, torch.float32)),
    "palarax": ("PalaraxRunner", "hybrid", (torch.bfloat16, torch.float32)),
    "ruludra": ("RuludraRunner", "hybrid", (torch.bfloat16, torch.float32)),
    "qwen3forcausallm": ("Qwen3Runner", "decoder", (torch.bfloat16,)),
}


class UnsupportedDtype(ValueError):
    """The model has no graph in the requested activation type."""


def _entry(path: str):
    with open(os.path.join(path, "config.json")) as f:
        c = json.load(f)
    names = [c["architecture"]] if "architecture" in c else list(c.get("architectures") or [])
    for n in names:
        if n.lower() in _RUNNERS:
            return _RUNNERS[n.lower()]
    raise KeyError(f"{path}: no runner for architecture {names} (known: {sorted(_RUNNERS)})")


def kernel_family(path: str) -> str:
    """Target of mirage_b200/build.py that a checkpoint's graph needs beside the core library."""
    return _entry(path)[1]


def runner_class(path: str) -> Tuple[type, tuple]:
    """(runner class, activation types it supports) for a checkpoint directory."""
    from . import runner
    name, _, dtypes = _entry(path)
    return getattr(runner, name), dtypes


def load_runner(path: str, dtype: torch.dtype = torch.bfloat16, **kw):
    """The checkpoint's runner, built.  Keyword arguments are those of `from_checkpoint` of the runner class."""
    cls, dtypes = runner_class(path)
    if dtype not in dtypes:
        raise UnsupportedDtype(f"{cls.__name__} has no {dtype} graph")
    if len(dtypes) > 1:
        kw["dtype"] = dtype
    return cls.from_checkpoint(path, **kw)
