"""Model classes by architecture name (``YvConfig.architecture``; the empty name is the Yv trunk) and the cache layout
that a model's layers ask for."""
from __future__ import annotations

from typing import Any, Callable, Dict, List, Optional, Tuple

_BUILDERS: Dict[str, Callable[[], type]] = {}


def register_model(name: str, builder: Callable[[], type]) -> None:
    """``builder`` returns the ``nn.Module`` class (called late, so that registration imports nothing)."""
    _BUILDERS[name] = builder


def model_class(cfg: Any) -> type:
    if cfg.architecture not in _BUILDERS:
        raise ValueError(f"no model class for architecture {cfg.architecture!r}; known: {sorted(_BUILDERS)}")
    return _BUILDERS[cfg.architecture]()


def latent_cache_layout(cfg: Any) -> Tuple[List[int], Optional[int]]:
    """(numbers per token of every layer's cache row, tokens the widest layer reads back or None)."""
    rows = [s["mixer"]["kv_rank"] + s["mixer"]["rot_dim"] for s in cfg.layer_specs]
    windows = [s["mixer"]["window"] for s in cfg.layer_specs]
    return rows, (max(windows) if all(windows) else None)


def _yv() -> type:
    from .model import YvModelForCausalLM
    return YvModelForCausalLM


def _layered() -> type:
    from .layered import YvLayeredForCausalLM
    return YvLayeredForCausalLM


register_model("", _yv)
register_model("Gebelorn", _layered)
