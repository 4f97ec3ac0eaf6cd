"""Model registry: which configuration and model class serve a checkpoint directory.

A family registers the names its ``config.json`` goes by; :func:`load_target` reads the file, picks the family and
loads the weights.  Names come from ``architecture`` (one string), ``architectures`` (Hugging Face's list) or
``model_type``; a file that names none of the registered families is read as Qwen3, the framework's first family.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass

import torch


@dataclass(frozen=True)
class ModelFamily:
    name: str
    config_cls: type
    model_cls: type


_FAMILIES: dict = {}
_DEFAULT = "qwen3"


def register_family(name: str, config_cls: type, model_cls: type, aliases=()) -> None:
    fam = ModelFamily(name, config_cls, model_cls)
    for key in (name, *aliases):
        _FAMILIES[key.lower()] = fam


def family_names() -> list:
    return sorted({f.name for f in _FAMILIES.values()})


def family_of(config: dict) -> ModelFamily:
    """The family a parsed ``config.json`` belongs to."""
    names = [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type")]
    for n in names:
        if isinstance(n, str) and n.lower() in _FAMILIES:
            return _FAMILIES[n.lower()]
    if isinstance(config.get("architecture"), str):
        raise ValueError(f"unknown architecture {config['architecture']!r}; registered: {family_names()}")
    return _FAMILIES[_DEFAULT]


def family_of_path(path: str) -> ModelFamily:
    with open(os.path.join(path, "config.json")) as f:
        return family_of(json.load(f))


def is_model(obj) -> bool:
    """True for an instance of a registered model class (engines also accept one instead of a directory)."""
    return isinstance(obj, tuple({f.model_cls for f in _FAMILIES.values()}))


def load_target(model_name_or_path, device="cuda", dtype=torch.bfloat16, attn_implementation: str = "auto",
                **_unused):
    """Load a target LM and its tokenizer from a local directory (``config.json`` + safetensors).

    Counterpart of the reference's ``load_target`` (``jetspec/models/qwen3.py:38-71``).
    ``attn_implementation`` is accepted for signature compatibility; attention is
    always this framework's own backend.  The tokenizer is ``None`` when the
    directory has no tokenizer files (token-id prompts still work).
    """
    model = family_of_path(model_name_or_path).model_cls.from_pretrained(model_name_or_path, dtype=dtype, device=device)
    return model, load_tokenizer(model_name_or_path)


def load_tokenizer(path: str):
    has_tok = any(os.path.exists(os.path.join(path, f))
                  for f in ("tokenizer.json", "tokenizer_config.json", "vocab.json"))
    if not has_tok:
        return None
    from transformers import AutoTokenizer
    return AutoTokenizer.from_pretrained(path)
