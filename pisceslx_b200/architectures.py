"""Architectures named by a checkpoint folder's ``config.json`` (key ``architecture``): how the file's keys map onto
``YvConfig`` fields.  The model classes are registered under the same names in ``models.registry``.

A layered architecture lists its layers one by one; each entry becomes a ``layer_specs`` item

    {"mixer": {"kind": ..., sizes and constants}, "mlp": {"kind": ..., "ff": ...} or None}

whose ``kind`` names a mixer or feed-forward of ``models.layered``, so that a new design made of known parts needs an
adapter here and nothing else."""
from __future__ import annotations

from typing import Any, Callable, Dict, List

_ADAPTERS: Dict[str, Callable[[Dict[str, Any]], Dict[str, Any]]] = {}


def register_architecture(name: str, adapter: Callable[[Dict[str, Any]], Dict[str, Any]]) -> None:
    _ADAPTERS[name] = adapter


def known_architectures() -> List[str]:
    return sorted(_ADAPTERS)


def config_fields(d: Dict[str, Any]) -> Dict[str, Any]:
    """``config.json`` of a named architecture -> ``YvConfig`` keyword arguments."""
    name = d["architecture"]
    if name not in _ADAPTERS:
        raise ValueError(f"unknown architecture {name!r}; known: {known_architectures()}")
    return _ADAPTERS[name](d)


def _rotation(rot: Dict[str, Any]) -> Dict[str, Any]:
    out: Dict[str, Any] = {"dims": int(rot["dims"]), "base": float(rot["base"])}
    sc = rot.get("scaling")
    if sc:
        out["yarn"] = {k: float(sc[k]) for k in ("factor", "original", "fast", "slow")}
    return out


def _gebelorn(d: Dict[str, Any]) -> Dict[str, Any]:
    """Windowed latent attention (query latent, shared rotary key part, per-head output gate) and plain GELU
    feed-forwards, normed before and after, with a per-layer token input; every layer has its own sizes."""
    specs = []
    for i, entry in enumerate(d["layers"]):
        if entry["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        m = entry["mixer"]
        rot = _rotation(m["rot"])
        if rot["dims"] != int(m["rot_dim"]):
            raise ValueError(f"layer {i}: the rotation covers the whole rotary part ({rot['dims']} != {m['rot_dim']})")
        mask = m.get("mask") or {}
        mixer = {"kind": "latent_attention", "heads": int(m["heads"]), "dim": int(m["dim"]), "rot_dim": int(m["rot_dim"]),
                 "vdim": int(m["vdim"]), "kv_rank": int(m["kv_rank"]), "q_rank": int(m["q_rank"]),
                 "scale": float(m["scale"]), "window": int(mask["size"]) if mask.get("size") else None, "rotation": rot,
                 "output_gate": True}
        mlp = None
        if entry.get("mlp"):
            if entry["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {entry['mlp']['kind']!r}")
            mlp = {"kind": "dense_gelu", "ff": int(entry["mlp"]["ff"])}
        specs.append({"mixer": mixer, "mlp": mlp})
    first = specs[0]["mixer"]
    side = d.get("token_side") or {}
    return dict(
        architecture=d["architecture"], model_type=d["architecture"].lower(), vocab_size=int(d["vocab"]),
        hidden_size=int(d["width"]), n_layer=len(specs), layer_specs=specs, layer_norm_eps=float(d["norm"]["eps"]),
        n_head=first["heads"], n_kv_head=first["heads"], head_dim=first["dim"] + first["rot_dim"],
        intermediate_size=max([s["mlp"]["ff"] for s in specs if s["mlp"]], default=1),
        token_side_dim=int(side.get("dim", 0)), moe_num_experts=0, moe_shared_experts=0, tie_word_embeddings=False,
        use_mla=True, kv_lora_rank=first["kv_rank"], mla_q_lora_rank=first["q_rank"], mla_rope_dim=first["rot_dim"],
        use_gradient_checkpointing=False, bos_token_id=-1, eos_token_id=-1, pad_token_id=0)


register_architecture("Gebelorn", _gebelorn)
