"""Checkpoints described by a ``config.json`` of their own form (a top-level ``architecture`` name) rather than by Hugging
Face's: readers that turn one into the attribute object the engine works with."""
from __future__ import annotations

import copy
import json
import os
import struct
from glob import glob
from types import SimpleNamespace
from typing import Any

import torch


def tensor_shapes(path: str) -> dict[str, list[int]]:
    """Name -> shape over every safetensors header of a directory (no tensor data is read)."""
    shapes: dict[str, list[int]] = {}
    for file in sorted(glob(os.path.join(path, "*.safetensors"))):
        with open(file, "rb") as f:
            (n,) = struct.unpack("<Q", f.read(8))
            header = json.loads(f.read(n))
        shapes.update({k: v["shape"] for k, v in header.items() if k != "__metadata__"})
    return shapes


def fupupel_config(config: dict, shapes: dict[str, list[int]] | None = None, dtype: torch.dtype = torch.bfloat16,
                   max_position_embeddings: int = 4096) -> SimpleNamespace:
    """The ranks of the delta rule's two low-rank projections are given by tensor shapes alone; without a checkpoint they
    come from the mixer's ``decay_rank`` / ``gate_rank`` (default: its ``dim``)."""
    layers = copy.deepcopy(config["layers"])
    for i, layer in enumerate(layers):
        if layer["type"] != "parallel":
            continue
        right = layer["mixer"]["right"]
        for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
            tensor = f"l{i}.mix.right.{name}"
            if shapes and tensor in shapes:
                right[key] = shapes[tensor][0]
            else:
                right.setdefault(key, right["dim"])
    return SimpleNamespace(
        architectures=["Fupupel"], dtype=dtype, layers=layers, num_hidden_layers=len(layers), hidden_size=config["width"],
        vocab_size=config["vocab"], rms_norm_eps=config["norm"]["eps"], logit_softcap=config.get("logit_softcap"),
        max_position_embeddings=max_position_embeddings, eos_token_id=config.get("eos_token_id"))


def vebonex_config(config: dict, shapes: dict[str, list[int]] | None = None, dtype: torch.dtype = torch.bfloat16,
                   max_position_embeddings: int = 4096) -> SimpleNamespace:
    """Positions are a learned table, so its size is the model's and not the engine's.  The rank of a decay's low-rank pair is given by
    tensor shapes alone; without a checkpoint it comes from the mixer's ``decay_rank`` (default: its ``dim``)."""
    layers = copy.deepcopy(config["layers"])
    for i, layer in enumerate(layers):
        if layer["type"] != "gla":
            continue
        tensor = f"l{i}.mix.a1"
        if shapes and tensor in shapes:
            layer["mixer"]["decay_rank"] = shapes[tensor][0]
        else:
            layer["mixer"].setdefault("decay_rank", layer["mixer"]["dim"])
    return SimpleNamespace(
        architectures=["Vebonex"], dtype=dtype, layers=layers, num_hidden_layers=len(layers), hidden_size=config["width"],
        vocab_size=config["vocab"], rms_norm_eps=config["norm"]["eps"], norm_groups=config["norm"]["groups"], streams=config["streams"],
        max_position_embeddings=config["max_positions"], learned_positions=config["max_positions"], eos_token_id=config.get("eos_token_id"))


def sunulorn_config(config: dict, shapes: dict[str, list[int]] | None = None, dtype: torch.dtype = torch.bfloat16,
                    max_position_embeddings: int = 4096) -> SimpleNamespace:
    """Positions are rotated or biased, so the engine's longest request sets how many there are."""
    layers = copy.deepcopy(config["layers"])
    return SimpleNamespace(
        architectures=["Sunulorn"], dtype=dtype, layers=layers, num_hidden_layers=len(layers), hidden_size=config["width"],
        vocab_size=config["vocab"], rms_norm_eps=config["norm"]["eps"], embedding_scale=config["embedding"]["scale"],
        max_position_embeddings=max_position_embeddings, eos_token_id=config.get("eos_token_id"))


def rasezen_config(config: dict, shapes: dict[str, list[int]] | None = None, dtype: torch.dtype = torch.bfloat16,
                   max_position_embeddings: int = 4096) -> SimpleNamespace:
    """Positions are rotated, so the engine's longest request sets how many there are."""
    layers = copy.deepcopy(config["layers"])
    return SimpleNamespace(
        architectures=["Rasezen"], dtype=dtype, layers=layers, num_hidden_layers=len(layers), hidden_size=config["width"],
        vocab_size=config["vocab"], rms_norm_eps=config["norm"]["eps"], max_position_embeddings=max_position_embeddings,
        eos_token_id=config.get("eos_token_id"))


_READERS = {"Fupupel": fupupel_config, "Vebonex": vebonex_config, "Sunulorn": sunulorn_config, "Rasezen": rasezen_config}


def read_native(path: str, dtype: torch.dtype | None, max_position_embeddings: int) -> Any:
    """The attribute object of the checkpoint in ``path``, or None if its config.json is not of this kind."""
    file = os.path.join(path, "config.json")
    if not os.path.isfile(file):
        return None
    with open(file) as f:
        config = json.load(f)
    reader = _READERS.get(config.get("architecture"))
    if reader is None:
        return None
    return reader(config, tensor_shapes(path), dtype or torch.bfloat16, max_position_embeddings)
