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


def cache_layout(cfg: Any) -> Tuple[List[Dict[str, int]], Optional[int]]:
    """(what every layer run of a layered model stores per token, tokens the widest layer reads back or None): either
    ``{"row": numbers}`` or ``{"heads", "dim", "vdim"}`` of keys and values."""
    layouts, reach = [], []
    for i, _, _ in cfg.layer_runs():
        m = cfg.layer_specs[i]["mixer"]
        if m["kind"] == "latent_attention":
            layouts.append({"row": m["kv_rank"] + m["rot_dim"]})
        else:
            layouts.append({"heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"]})
        reach.append(m.get("window"))
    return layouts, (max(reach) if all(reach) else None)


def kernel_families(cfg: Any) -> Tuple[str, ...]:
    """The operator families (``ops.build.FAMILIES``) that serve a model; empty = the whole library."""
    return tuple(sorted({s["mixer"]["kind"] for s in cfg.layer_specs}))


def _yv() -> type:
    from .model import YvModelForCausalLM
    return YvModelForCausalLM


def _layered() -> type:
    from .layered import YvLayeredForCausalLM
    return YvLayeredForCausalLM


register_model("", _yv)
register_model("Gebelorn", _layered)
register_model("Pitolix", _layered)
