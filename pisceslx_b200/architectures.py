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


def _dense(entry: Dict[str, Any], i: int, kind: str) -> Any:
    """The feed-forward of a layer entry (None for none); every design here names one kind, ``dense``."""
    if not entry.get("mlp"):
        return None
    if entry["mlp"]["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward kind {entry['mlp']['kind']!r}")
    return {"kind": kind, "ff": int(entry["mlp"]["ff"])}


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
        specs.append({"mixer": mixer, "mlp": _dense(entry, i, "dense_gelu")})
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


def _pitolix(d: Dict[str, Any]) -> Dict[str, Any]:
    """Two kinds of grouped-query attention (normed queries and keys with a position-dependent temperature, a sink and a
    gate per number, against rotation, biases and a gate per head) beside a SwiGLU feed-forward that reads the same
    stream; a run of layers is passed through several times."""
    specs = []
    for i, entry in enumerate(d["layers"]):
        m = entry["mixer"]
        mixer = {"kind": "grouped_attention", "heads": int(m["heads"]), "kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]),
                 "vdim": int(m["vdim"]), "scale": float(m["scale"]), "rotation": None}
        if entry["type"] == "attention":
            mixer.update(qk_norm=True, sink=True, output_gate="element")
            temp = m.get("q_temp")
            if temp:
                mixer["temperature"] = {"coef": float(temp["coef"]), "every": int(temp["every"])}
        elif entry["type"] == "attention_2":
            mixer.update(bias=True, output_gate="head", rotation=_rotation(m["rot"]) if m.get("rot") else None)
        else:
            raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        specs.append({"mixer": mixer, "mlp": _dense(entry, i, "dense_swiglu")})
    first, loop = specs[0]["mixer"], d.get("loop")
    if loop:
        loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
        if not 0 <= loop["start"] < loop["stop"] <= len(specs) or loop["times"] < 1:
            raise ValueError(f"loop {loop} does not fit {len(specs)} layers")
    return dict(
        architecture=d["architecture"], model_type=d["architecture"].lower(), vocab_size=int(d["vocab"]),
        hidden_size=int(d["width"]), n_layer=len(specs), layer_specs=specs, layer_norm_eps=float(d["norm"]["eps"]),
        layer_block="parallel", layer_loop=loop or None, norm_offset=1.0, embedding_norm=False,
        embedding_scale=float(d["embedding"]["scale"]), n_head=first["heads"], n_kv_head=first["kv_heads"],
        head_dim=first["dim"], intermediate_size=max([s["mlp"]["ff"] for s in specs if s["mlp"]], default=1),
        moe_num_experts=0, moe_shared_experts=0, tie_word_embeddings=False, use_gradient_checkpointing=False,
        bos_token_id=-1, eos_token_id=-1, pad_token_id=0)


register_architecture("Gebelorn", _gebelorn)
register_architecture("Pitolix", _pitolix)
