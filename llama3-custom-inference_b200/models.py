"""The model registry: which decoder serves a model folder, chosen by its config.json.

An architecture brings its configuration reader, its weight mapping (checkpoint tensors -> what the decoder takes), its
decoder class and the build targets its kernels live in.
"""
from __future__ import annotations

from dataclasses import dataclass
from types import SimpleNamespace
from typing import Callable

import torch

from . import build, checkpoint, decode_loop, nibelorn, rupotar


@dataclass(frozen=True)
class Architecture:
    read_config: Callable     # config.json as a dict -> the decoder's configuration
    map_weights: Callable     # (checkpoint tensors, configuration) -> the decoder's `weights`
    decoder: type
    libraries: tuple          # build targets of the forward pass (token choice needs "extension" besides)
    dtypes: tuple = (torch.bfloat16,)


ARCHITECTURES = {
    "LlamaForCausalLM": Architecture(
        read_config=lambda c: decode_loop.config_from_hf(SimpleNamespace(**c)),
        map_weights=decode_loop.weights_from_hf, decoder=decode_loop.Llama3Decoder, libraries=("library", "extension")),
    "Nibelorn": Architecture(
        read_config=nibelorn.config_from_json, map_weights=lambda tensors, cfg: tensors,
        decoder=nibelorn.NibelornDecoder, libraries=("mixers",), dtypes=(torch.bfloat16, torch.float32)),
    "Rupotar": Architecture(
        read_config=rupotar.config_from_json, map_weights=lambda tensors, cfg: tensors,
        decoder=rupotar.RupotarDecoder, libraries=("mixers",), dtypes=(torch.bfloat16, torch.float32)),
}


def architecture_of(config: dict) -> Architecture:
    names = [config["architecture"]] if "architecture" in config else list(config.get("architectures") or [])
    for name in names:
        if name in ARCHITECTURES:
            return ARCHITECTURES[name]
    raise ValueError(f"no decoder for architecture {names}; known: {sorted(ARCHITECTURES)}")


def load_model(folder, device, max_batch: int, max_len: int, dtype=torch.bfloat16, ext=None):
    """The decoder of a model folder (config.json, model.safetensors) with its weights, ready to run.  Builds the
    libraries it needs if they are missing or older than their sources."""
    config = checkpoint.read_config(folder)
    arch = architecture_of(config)
    if dtype not in arch.dtypes:
        raise NotImplementedError(f"{arch.decoder.__name__} does not run in {dtype}")
    build.ensure(*arch.libraries)
    cfg = arch.read_config(config)
    weights = arch.map_weights(checkpoint.read_weights(folder), cfg)
    return arch.decoder(ext, cfg, device, max_batch, max_len, weights=weights, dtype=dtype)
