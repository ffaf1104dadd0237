"""Small configurations and random weights of the Gebelorn design, and the schedules the tests run them through."""
import torch

import gebelorn_oracle as oracle

YARN = {"factor": 6.0, "original": 48, "fast": 8.0, "slow": 1.0}


def layer(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, ff, scale, base=1000.0, scaling=YARN):
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": scale, "mask": {"size": window}, "rot": rot},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, vocab, width, side, eps):
    return {"architecture": "Gebelorn", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "token_side": {"dim": side}}


def mixed():
    """Every size differs between the layers; one layer has no feed-forward, one rotates without scaling."""
    return config([layer(3, 24, 8, 16, 40, 32, 7, 104, 0.31),
                   layer(2, 16, 16, 40, 64, 56, 70, None, 0.2, base=300.0, scaling=None),
                   layer(5, 40, 24, 24, 136, 48, 33, 64, 0.17, scaling={"factor": 3.5, "original": 20, "fast": 4.0, "slow": 0.5})],
                  vocab=104, width=80, side=8, eps=3e-5)


def odd():
    """Sizes that no 16-byte vector divides, and a window of one."""
    return config([layer(3, 10, 6, 9, 21, 13, 1, 35, 0.4), layer(1, 7, 2, 5, 11, 19, 41, 22, 0.5)],
                  vocab=61, width=50, side=3, eps=1e-4)


def wide():
    """Heads, latent and parts at the upper sizes of the tensor-core kernels."""
    return config([layer(18, 128, 64, 128, 256, 64, 150, 128, 0.09), layer(20, 72, 40, 120, 200, 96, 90, 128, 0.12)],
                  vocab=128, width=128, side=16, eps=1e-6)


def weights(cfg, seed=0):
    """bf16-representable random weights, scaled so that attention is peaked and every branch contributes."""
    g = torch.Generator().manual_seed(seed)
    C, V = cfg["width"], cfg["vocab"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / i ** 0.5).bfloat16()

    def norm(n):
        return (1.0 + 0.3 * torch.randn(n, generator=g)).bfloat16()

    W = {"embed": torch.randn(V, C, generator=g).bfloat16(), "embed.norm": norm(C), "final.norm": norm(C), "head": lin(V, C)}
    S = (cfg.get("token_side") or {}).get("dim", 0)
    if S:
        W["side.embed"] = torch.randn(V, S * len(cfg["layers"]), generator=g).bfloat16()
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        W[p + "norm1"], W[p + "norm1b"] = norm(C), norm(C)
        W[p + "mix.dq"], W[p + "mix.dq.norm"] = lin(m["q_rank"], C), norm(m["q_rank"])
        W[p + "mix.uq"] = lin(m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.6)
        W[p + "mix.dkv"], W[p + "mix.dkv.norm"] = lin(m["kv_rank"] + m["rot_dim"], C, 1.5), norm(m["kv_rank"])
        W[p + "mix.uk"] = lin(m["heads"] * m["dim"], m["kv_rank"], 1.6)
        W[p + "mix.uv"] = lin(m["heads"] * m["vdim"], m["kv_rank"])
        W[p + "mix.g"], W[p + "mix.o"] = lin(m["heads"], C, 2.0), lin(C, m["heads"] * m["vdim"])
        if e["mlp"]:
            W[p + "norm2"], W[p + "norm2b"] = norm(C), norm(C)
            W[p + "mlp.up"], W[p + "mlp.down"] = lin(e["mlp"]["ff"], C, 1.5), lin(C, e["mlp"]["ff"])
        if S:
            W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"] = lin(S, C, 2.0), lin(C, S), norm(C)
    return W


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def build(cfg, W, device="cpu", dtype=torch.float32):
    from pisceslx_b200 import YvConfig
    from pisceslx_b200.models import build_model
    m = build_model(YvConfig.from_dict(cfg), device, dtype).eval()
    assert m.load_reference_state_dict(W) == []
    return m


def engine(model, blocks=24, block_size=64, **kw):
    from pisceslx_b200.serve.engine import YvEngineConfig, YvInferenceEngine
    return YvInferenceEngine(model, cfg=YvEngineConfig(num_blocks=blocks, block_size=block_size, eos_token_id=-1,
                                                       max_model_len=1024, **kw))


def run_cut(eng, seq_id, toks, cuts):
    """Logits of every position when ``toks`` arrives in portions of the given sizes (the last one repeats)."""
    eng.cache.add_sequence(seq_id)
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(eng.run_tokens(seq_id, toks[at:at + n], list(range(n))).float().cpu().clone())
        at, i = at + n, i + 1
    eng.cache.free_sequence(seq_id)
    return torch.cat(out, 0)


def expected(cfg, W, toks, dtype=torch.float64, layers_out=None):
    with torch.no_grad():
        return oracle.forward(cfg, W, toks, dtype, layers_out).float()


def error(got, want):
    """Per position: root mean square over the vocabulary, means taken off, relative to the logits' spread."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


def rounding_limit(cfg, W, toks, want, times=3.0):
    """Per position: what weights off by one bf16 rounding do to the plain logits (some positions are badly
    conditioned), not below the median over positions, times a factor."""
    g = torch.Generator().manual_seed(77)
    noise = torch.stack([error(expected(cfg, {k: v.float() * (1 + 2 ** -9 * torch.randn(v.shape, generator=g))
                                              for k, v in W.items()}, toks, torch.float32), want)
                         for _ in range(4)]).amax(0)
    return times * noise.clamp_min(noise.median())


CUTS = {"whole": [10_000], "token by token": [1], "pairs": [2], "uneven": [5, 64, 1, 1, 3, 130, 2, 17], "pages": [64],
        "prompt then decode": [100, 1]}
