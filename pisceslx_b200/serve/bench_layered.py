"""Prefill and decode throughput of a layered design beside the Yv trunk's closest configuration at equal size
(``bench.py --design gebelorn`` or ``pitolix``).

* Gebelorn: the Yv trunk with dense feed-forwards and its low-rank attention (``use_mla`` with the shared rotary slice):
  same width, layers, heads, ranks and vocabulary, a SwiGLU feed-forward of the same number of parameters, full causal
  attention (the design's window covers the whole context of the decode case).
* Pitolix: the Yv trunk with dense SwiGLU feed-forwards and grouped-query attention: same width, query and key/value heads,
  head size, feed-forward and vocabulary, as many layers as the design has layer runs (two layers are passed twice).

Both run random weights through the serving engine: a prompt is one ``run_tokens`` call, a decode step one replay of a
captured step.  Times are CUDA events around the calls after three warm-ups; weights and caches are larger than L2."""
from __future__ import annotations

import json
import time
from typing import Any, Callable, Dict, List, Tuple

import torch

VOCAB = 32000
GEBELORN_SIZES: Dict[str, Dict[str, int]] = {
    "w1024": dict(width=1024, heads=16, dim=64, rot=32, vdim=64, kv_rank=256, q_rank=512, ff=4096, side=64, window=1024,
                  layers=8, prompt=8192, batch=64, context=4096),
    "w2048": dict(width=2048, heads=16, dim=128, rot=64, vdim=128, kv_rank=512, q_rank=1536, ff=8192, side=256,
                  window=4096, layers=8, prompt=8192, batch=64, context=4096),
    "w4096": dict(width=4096, heads=32, dim=128, rot=64, vdim=128, kv_rank=512, q_rank=1536, ff=16384, side=256,
                  window=4096, layers=4, prompt=8192, batch=64, context=4096),
}
PITOLIX_SIZES: Dict[str, Dict[str, int]] = {
    "w1024": dict(width=1024, heads=16, kv_heads=4, dim=64, rot=32, ff=2816, runs=8, prompt=8192, batch=64, context=4096),
    "w2048": dict(width=2048, heads=16, kv_heads=4, dim=128, rot=64, ff=5632, runs=8, prompt=8192, batch=64, context=4096),
    "w4096": dict(width=4096, heads=32, kv_heads=8, dim=128, rot=64, ff=11264, runs=5, prompt=8192, batch=64, context=4096),
}


def gebelorn_config(s: Dict[str, int]):
    from ..config import YvConfig
    layer = {"type": "latent_attention",
             "mixer": {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot"], "vdim": s["vdim"], "kv_rank": s["kv_rank"],
                       "q_rank": s["q_rank"], "scale": (s["dim"] + s["rot"]) ** -0.5, "mask": {"size": s["window"]},
                       "rot": {"dims": s["rot"], "base": 10000.0,
                               "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}},
             "mlp": {"kind": "dense", "ff": s["ff"]}}
    return YvConfig.from_dict({"architecture": "Gebelorn", "layers": [layer] * s["layers"], "norm": {"eps": 1e-6},
                               "vocab": VOCAB, "width": s["width"], "token_side": {"dim": s["side"]}})


def gebelorn_closest(s: Dict[str, int]):
    from ..config import YvConfig
    return YvConfig(vocab_size=VOCAB, hidden_size=s["width"], n_layer=s["layers"], n_head=s["heads"], n_kv_head=s["heads"],
                    head_dim=128 if s["dim"] > 64 else 64, intermediate_size=(s["ff"] * 2 // 3 + 63) // 64 * 64,
                    moe_num_experts=0, moe_shared_experts=0, use_mla=True, kv_lora_rank=s["kv_rank"],
                    mla_q_lora_rank=s["q_rank"], mla_rope_dim=s["rot"], use_enhanced_mla=True, tie_word_embeddings=False,
                    max_position_embeddings=16384, use_gradient_checkpointing=False, eos_token_id=-1)


def pitolix_config(s: Dict[str, int]):
    """One layer in three has normed queries and keys, the others rotate; layers 0 and 1 are passed twice."""
    from ..config import YvConfig
    base = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5}
    mlp = {"kind": "dense", "ff": s["ff"]}
    rotated = {"type": "attention_2", "mixer": {**base, "rot": {"dims": s["rot"], "base": 10000.0}}, "mlp": mlp}
    normed = {"type": "attention", "mixer": {**base, "q_temp": {"coef": 0.2, "every": 1024}}, "mlp": mlp}
    layers = [normed if i % 3 == 2 else rotated for i in range(s["runs"] - 2)]
    return YvConfig.from_dict({"architecture": "Pitolix", "layers": layers, "norm": {"eps": 1e-6}, "vocab": VOCAB,
                               "width": s["width"], "embedding": {"scale": s["width"] ** 0.5},
                               "loop": {"start": 0, "stop": 2, "times": 2}})


def pitolix_closest(s: Dict[str, int]):
    from ..config import YvConfig
    return YvConfig(vocab_size=VOCAB, hidden_size=s["width"], n_layer=s["runs"], n_head=s["heads"], n_kv_head=s["kv_heads"],
                    head_dim=s["dim"], intermediate_size=s["ff"], moe_num_experts=0, moe_shared_experts=0,
                    tie_word_embeddings=False, max_position_embeddings=16384, use_gradient_checkpointing=False,
                    eos_token_id=-1)


# name -> (sizes, the design's configuration, the closest Yv configuration)
DESIGNS: Dict[str, Tuple[Dict[str, Dict[str, int]], Callable[..., Any], Callable[..., Any]]] = {
    "gebelorn": (GEBELORN_SIZES, gebelorn_config, gebelorn_closest),
    "pitolix": (PITOLIX_SIZES, pitolix_config, pitolix_closest),
}


def _kernel_shares(fn, top: int = 12) -> List[Tuple[str, float, int]]:
    """(kernel, device microseconds, launches) of one call, largest first."""
    from torch.profiler import ProfilerActivity, profile
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        fn()
        torch.cuda.synchronize()
    rows = [(e.key.replace("(anonymous namespace)::", "").split("(")[0].replace("void ", "")[:90], e.self_device_time_total, e.count) for e in prof.key_averages()
            if e.self_device_time_total > 0]
    return sorted(rows, key=lambda r: -r[1])[:top]


def measure(cfg, s: Dict[str, int], steps: int, warmup: int, shares: bool) -> Dict[str, Any]:
    from ..models import build_model
    from ..ops import check_status
    from .engine import YvEngineConfig, YvInferenceEngine
    dev = torch.device("cuda", 0)
    model = build_model(cfg, dev, torch.bfloat16, seed=0).eval()
    pages = s["batch"] * (-(-(s["context"] + 64) // 64) + 1) + -(-s["prompt"] // 64) + 8
    eng = YvInferenceEngine(model, cfg=YvEngineConfig(max_num_seqs=s["batch"], num_blocks=pages, eos_token_id=-1,
                                                      max_model_len=max(s["prompt"], s["context"] + 64), graph_max_seq_len=s["context"] + 64))
    gen = torch.Generator().manual_seed(1)
    prompt = torch.randint(0, cfg.vocab_size, (s["prompt"],), generator=gen).tolist()

    def prefill(n: int = 0) -> None:
        eng.cache.add_sequence(-5)
        eng.run_tokens(-5, prompt[:n or len(prompt)], [(n or len(prompt)) - 1])
        eng.cache.free_sequence(-5)

    def timed(fn, count: int) -> float:
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(count):
            fn()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) / count

    for _ in range(warmup):
        prefill()
    pre_ms = timed(prefill, steps)
    seqs = list(range(s["batch"]))
    for i in seqs:                                       # every sequence starts with the same context length
        eng.cache.add_sequence(i)
        eng.run_tokens(i, prompt[: s["context"]], [])
    last = [7] * s["batch"]

    def decode() -> None:
        eng.graph.step(last, seqs)

    for _ in range(warmup):
        decode()
    dec_ms = timed(decode, max(8, 4 * steps))
    out = {"parameters": sum(p.numel() for p in model.parameters()), "cache_bytes_per_token": eng.cache.bytes() // (pages * 64),
           "prefill_ms": pre_ms, "prefill_tokens_per_s": s["prompt"] / pre_ms * 1e3, "decode_ms_per_step": dec_ms,
           "decode_tokens_per_s": s["batch"] / dec_ms * 1e3, "decode_graph": eng.graph.disabled_reason is None}
    if shares:
        out["prefill_kernels_us"] = _kernel_shares(prefill)
        out["decode_kernels_us"] = _kernel_shares(decode)
    check_status(dev)
    del eng, model
    torch.cuda.empty_cache()
    return out


def run(design: str, steps: int, warmup: int, names: List[str], shares: bool) -> Dict[str, Any]:
    from ..ops import load_extension
    load_extension()
    sizes, config, closest = DESIGNS[design]
    res: Dict[str, Any] = {"metric": f"prefill and decode tokens/s, {design.capitalize()} beside the closest Yv model",
                           "dtype": "bf16", "data": "synthetic uniform-random token ids, random-init weights", "steps": steps,
                           "warmup": warmup, "time": time.strftime("%Y-%m-%dT%H:%M:%SZ", time.gmtime()), "sizes": {}}
    with torch.no_grad():
        for name in names or list(sizes):
            s = sizes[name]
            res["sizes"][name] = {"shape": s, design: measure(config(s), s, steps, warmup, shares),
                                  "closest_yv": measure(closest(s), s, steps, warmup, shares)}
    return res


def main(design: str, steps: int, warmup: int, sizes: str = "", shares: bool = False) -> None:
    print(json.dumps(run(design, steps, warmup, [x for x in sizes.split(",") if x], shares)))
