"""Model classes by the name a checkpoint's config.json gives in "architecture", and loading a checkpoint folder."""
from __future__ import annotations

import json
import os

from . import _lib
from .checkpoint import read_safetensors
from .dotanex import DotanexConfig, DotanexModel
from .numuzen import NumuzenConfig, NumuzenModel
from .sakinex import SakinexConfig, SakinexModel
from .tofazen import TofazenConfig, TofazenModel

# architecture -> (configuration class, model class with ``from_tensors``)
ARCHITECTURES = {"Tofazen": (TofazenConfig, TofazenModel), "Numuzen": (NumuzenConfig, NumuzenModel), "Dotanex": (DotanexConfig, DotanexModel),
                 "Sakinex": (SakinexConfig, SakinexModel)}

DEFAULT_MAX_SEQ = 8192      # for designs without a largest position

DTYPES = {"bfloat16": _lib.BF16, "float32": _lib.F32}


class UnknownArchitecture(ValueError):
    pass


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        return json.load(f)


def resolve(config: dict):
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise UnknownArchitecture(f"architecture {name!r} is not one of {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[name]


def load_model(dev, folder: str, dtype: int = _lib.BF16, max_slots: int = 64, max_seq: int | None = None, cache_budget: int = 64 << 30):
    """Loads config.json and model.safetensors from `folder`.  `max_slots` concurrent sequences of `max_seq` positions
    (default: all the model has, or DEFAULT_MAX_SEQ when its design sets no limit); fewer slots when they would take more than `cache_budget` bytes."""
    config = read_config(folder)
    config_class, model_class = resolve(config)
    cfg = config_class.from_dict(config)
    limit = getattr(cfg, "max_positions", None)
    seq = max_seq or limit or DEFAULT_MAX_SEQ
    if limit:
        seq = min(seq, limit)
    max_slots = max(1, min(max_slots, cache_budget // max(1, cfg.bytes_per_slot(dtype, seq))))
    return model_class.from_tensors(dev, config, read_safetensors(os.path.join(folder, "model.safetensors")), dtype, max_slots, seq)
