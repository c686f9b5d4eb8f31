"""Model registry keyed on HF ``config.json: model_type`` (reference: lightllm/models/registry.py)."""
from __future__ import annotations

from typing import Callable, Dict, Optional

_REGISTRY: Dict[str, list] = {}
_CONFIGS: Dict[str, Callable[[dict], dict]] = {}


def register_config(architecture: str):
    """For designs whose config.json is not in HF spelling: the decorated function turns a config with
    `"architecture": architecture` (and no model_type) into one with the keys the framework reads."""
    def deco(fn):
        _CONFIGS[architecture] = fn
        return fn

    return deco


def native_config(config: dict) -> dict:
    if config.get("model_type") or not isinstance(config.get("architecture"), str):
        return config
    from . import _load_all  # noqa: F401

    fn = _CONFIGS.get(config["architecture"])
    if fn is None:
        raise ValueError(f"unsupported architecture {config['architecture']!r}; known: {sorted(_CONFIGS)}")
    return fn(config)


def register_model(*model_types: str, condition: Optional[Callable[[dict], bool]] = None, is_multimodal=False):
    def deco(cls):
        for mt in model_types:
            _REGISTRY.setdefault(mt, []).append((condition, cls, is_multimodal))
        return cls

    return deco


def get_model_class(config: dict):
    from . import _load_all  # noqa: F401  (imports every model module once)

    mt = native_config(config).get("model_type")
    cands = _REGISTRY.get(mt)
    if not cands:
        raise ValueError(f"unsupported model_type {mt!r}; known: {sorted(_REGISTRY)}")
    # conditional entries first
    for cond, cls, _ in cands:
        if cond is not None and cond(config):
            return cls
    for cond, cls, _ in cands:
        if cond is None:
            return cls
    raise ValueError(f"no registered variant of {mt!r} accepts this config")


def is_multimodal(config: dict) -> bool:
    from . import _load_all  # noqa: F401

    cands = _REGISTRY.get(config.get("model_type"), [])
    for cond, _, mm in cands:   # the variant that `get_model_class` would pick
        if cond is not None and cond(config):
            return bool(mm)
    return any(mm for cond, _, mm in cands if cond is None)


def supported_model_types():
    from . import _load_all  # noqa: F401

    return sorted(_REGISTRY)


def get_model(config: dict, **kvargs):
    return get_model_class(config)(config, **kvargs)
