"""Model families by the architecture name in a model folder's config.json: which kernels library a family needs, how
its weights are loaded, which dtypes it runs in, and the session that generates with it.  Families are imported on
first use, so serving one does not load another."""
from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class UnsupportedDtype(RuntimeError):
    """The family does not run in the requested dtype."""


@dataclass(frozen=True)
class Family:
    library: str                       # key of build.LIBRARIES
    module: str                        # module with load(folder, config, dtype, context_len, device)
    loader: str
    dtypes: tuple = ("bfloat16", "float32")


FAMILIES: dict[str, Family] = {
    # fp32 activations enter the packed products as two fp16 terms: not a 32-bit mode
    "PackedGPT": Family("packed", "nativebit_b200.generate", "load_folder", ("bfloat16",)),
    "Nerulorn": Family("layered", "nativebit_b200.nerulorn", "load"),
    "Nabalix": Family("layered", "nativebit_b200.nabalix", "load"),
}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def family(config: dict) -> Family:
    name = config.get("architecture")
    if name not in FAMILIES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(FAMILIES)}")
    return FAMILIES[name]


def build_for(config: dict) -> None:
    """Compiles the kernels the family needs, if they are missing or out of date."""
    from .build import build_library
    build_library(which=family(config).library)


def load_model(folder: str, dtype: str = "bfloat16", context_len: int = 4096, device="cuda"):
    """The model of a folder (config.json and weights), ready for `open_session`."""
    config = read_config(folder)
    fam = family(config)
    if dtype not in fam.dtypes:
        raise UnsupportedDtype(f"{config['architecture']} runs in {', '.join(fam.dtypes)}, not in {dtype}")
    load = getattr(importlib.import_module(fam.module), fam.loader)
    return load(folder, config, DTYPES[dtype], context_len, torch.device(device))


def open_session(model, batch_size: int = 1, **options):
    """The family's generation session (session.Session) over a model."""
    return model.session(batch_size, **options)
