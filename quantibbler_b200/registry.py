"""Which decoder serves a model: a folder with config.json is looked up by its ``architecture``
key; a folder with manifest.toml or a single-file blob is the factorized Llama-shaped decoder."""

from __future__ import annotations

import json
import os

from . import blob, model_dir, safetensors, virudra, vogizen
from .decoder import Decoder
from .layered import LayeredDecoder


def _load_vogizen(ctx, config: dict, tensors: dict, **settings):
    vogizen.check_tensors(config, tensors)
    return LayeredDecoder(ctx, vogizen.parse(config, **settings), tensors)


def _load_virudra(ctx, config: dict, tensors: dict, **settings):
    virudra.check_tensors(config, tensors)
    return LayeredDecoder(ctx, virudra.parse(config, **settings), tensors)


ARCHITECTURES = {"Virudra": _load_virudra, "Vogizen": _load_vogizen}


class UnknownArchitecture(ValueError):
    pass


def load_decoder(ctx, path: str, **settings):
    """A decoder for the model at ``path``.  ``settings``: ``serving`` ("float32" or "bfloat16"),
    ``max_seq``, ``max_batch``, ``prefill_chunk`` and the decoder's other serving settings."""
    path = os.fspath(path)
    config_path = os.path.join(path, "config.json")
    if os.path.isfile(config_path):
        with open(config_path) as f:
            config = json.load(f)
        name = config.get("architecture")
        if name not in ARCHITECTURES:
            raise UnknownArchitecture(f"{config_path}: architecture {name!r} is not served; known: "
                                      + ", ".join(sorted(ARCHITECTURES)))
        tensors = safetensors.load(os.path.join(path, "model.safetensors"))
        return ARCHITECTURES[name](ctx, config, tensors, **settings)
    cfg, weights = model_dir.decoder_inputs(blob.load_any(path), **settings)
    return Decoder(ctx, cfg, weights)
