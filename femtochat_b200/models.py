"""Model registry: which class runs a folder of config.json + model.safetensors.

config.json names the model in "architecture".  A registered class offers
`from_weights(config_json, tensors, compute_type=..., **options)` and the face that generation uses: `params`, `config`
(`vocab_size`, `sequence_len`), `index_base`, `state(B)`."""
from __future__ import annotations

import json
import os

from .decoder import Decoder
from .gpt import GPT
from .weights import SafeTensors

MODELS = {"GPT": GPT, "Virolorn": Decoder, "Zurevik": Decoder}


def register(architecture: str, cls) -> None:
    MODELS[architecture] = cls


def load_model(path: str, compute_type="bfloat16", **options):
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    name = config.get("architecture")
    if name not in MODELS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(MODELS))}")
    return MODELS[name].from_weights(config, SafeTensors(os.path.join(path, "model.safetensors")), compute_type=compute_type, **options)
