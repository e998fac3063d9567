"""Model registry: which model class a ``config.json`` asks for, and how a folder with ``config.json`` and
``model.safetensors`` becomes a model.

An entry names itself, recognises a parsed config, turns it into the model's configuration object and builds the model.
``register`` adds one; ``resolve`` picks the first that recognises the config (later registrations win).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, List

import torch


@dataclass(frozen=True)
class Architecture:
    name: str
    matches: Callable[[dict], bool]
    config: Callable          # (parsed config, dtype) -> configuration object; with ``shapes``, (.., name -> shape of the weights)
    build: Callable           # (configuration object, device) -> model with load_safetensors
    kernels: str = ""         # group of translation units that serves it (build.GROUPS); empty: the whole library
    shapes: bool = False      # some sizes are only in the weights


_REGISTRY: List[Architecture] = []


def register(arch: Architecture) -> None:
    _REGISTRY.insert(0, arch)


def architectures() -> List[str]:
    return [a.name for a in _REGISTRY]


def resolve(obj: dict) -> Architecture:
    for a in _REGISTRY:
        if a.matches(obj):
            return a
    raise ValueError(f"no registered model takes this config (known: {', '.join(architectures())})")


def read_config(path: str) -> dict:
    try:
        with open(path, "r", encoding="utf-8") as f:
            obj = json.load(f)
    except OSError as e:
        raise ValueError(f"cannot read {path}: {e}") from None
    except json.JSONDecodeError as e:
        raise ValueError(f"{path}: malformed JSON ({e})") from None
    if not isinstance(obj, dict):
        raise ValueError(f"{path}: top-level JSON value must be an object")
    return obj


def load_config(path: str, dtype: torch.dtype):
    """(architecture, configuration object) of a config.json."""
    obj = read_config(path)
    arch = resolve(obj)
    return arch, arch.config(obj, dtype)


def tensor_shapes(path: str) -> dict:
    from ..io.safetensors import SafeTensors
    with SafeTensors.open(path) as st:
        return {k: st.info(k)[1] for k in st.keys()}


def load_model(config_path: str, weights_path: str, dtype: torch.dtype, device=None):
    obj = read_config(config_path)
    arch = resolve(obj)
    cfg = arch.config(obj, dtype, tensor_shapes(weights_path)) if arch.shapes else arch.config(obj, dtype)
    model = arch.build(cfg, device)
    model.load_safetensors(weights_path)
    return model


def load_pretrained(folder: str, dtype: torch.dtype, device=None):
    return load_model(os.path.join(folder, "config.json"), os.path.join(folder, "model.safetensors"), dtype, device)


def _llama_config(obj: dict, dtype: torch.dtype):
    from .llama import LlamaConfig
    cfg = LlamaConfig.from_json(json.dumps(obj))
    cfg.dtype = dtype
    return cfg


def _llama_build(cfg, device):
    from .llama import LlamaModel
    return LlamaModel(cfg, device=device)


def _is_llama(obj: dict) -> bool:
    archs = obj.get("architectures") or []
    return ("architecture" not in obj and "hidden_size" in obj
            and (not archs or any(str(a).startswith(("Llama", "Mixtral")) for a in archs)))


def _fozelix_config(obj: dict, dtype: torch.dtype):
    from . import fozelix
    return fozelix.config_from_dict(obj, dtype)


def _fozelix_build(cfg, device):
    from . import fozelix
    return fozelix.build(cfg, device)


def _polosun_config(obj: dict, dtype: torch.dtype):
    from . import polosun
    return polosun.config_from_dict(obj, dtype)


def _polosun_build(cfg, device):
    from . import polosun
    return polosun.build(cfg, device)


def _vobotar_config(obj: dict, dtype: torch.dtype, shapes=None):
    from . import vobotar
    return vobotar.config_from_dict(obj, dtype, shapes)


def _vobotar_build(cfg, device):
    from . import vobotar
    return vobotar.build(cfg, device)


def _tonilix_config(obj: dict, dtype: torch.dtype, shapes=None):
    from . import tonilix
    return tonilix.config_from_dict(obj, dtype, shapes)


def _tonilix_build(cfg, device):
    from . import tonilix
    return tonilix.build(cfg, device)


register(Architecture("Llama", _is_llama, _llama_config, _llama_build))
register(Architecture("Fozelix", lambda o: o.get("architecture") == "Fozelix", _fozelix_config, _fozelix_build,
                      kernels="fozelix"))
register(Architecture("Polosun", lambda o: o.get("architecture") == "Polosun", _polosun_config, _polosun_build,
                      kernels="polosun"))
register(Architecture("Vobotar", lambda o: o.get("architecture") == "Vobotar", _vobotar_config, _vobotar_build,
                      kernels="vobotar", shapes=True))
register(Architecture("Tonilix", lambda o: o.get("architecture") == "Tonilix", _tonilix_config, _tonilix_build,
                      kernels="tonilix", shapes=True))
