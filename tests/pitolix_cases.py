"""Small configurations and random weights of the Pitolix design, and the schedules the tests run them through."""
import torch

import pitolix_oracle as oracle
from gebelorn_cases import engine, error, run_cut, tokens                                           # noqa: F401


def normed(heads, kv_heads, dim, vdim, ff, scale, temp=(0.4, 16)):
    """Unit queries and keys, temperature, sink, a gate per number."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        mixer["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def rotated(heads, kv_heads, dim, vdim, ff, scale, dims, base=900.0):
    """Rotation of a part of the head, biases, a gate per head."""
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                             "rot": {"dims": dims, "base": base}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, vocab, width, eps, scale=1.0, loop=None):
    cfg = {"architecture": "Pitolix", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab,
           "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def mixed():
    """Every size differs between the layers; the loop starts and ends inside; a layer without feed-forward in it."""
    return config([rotated(6, 2, 24, 16, 104, 0.3, 8), normed(4, 4, 40, 24, None, 1.9), rotated(8, 1, 16, 72, 56, 0.25, 16, 200.0),
                   normed(3, 1, 64, 40, 88, 2.4, (0.7, 5))], vocab=104, width=80, eps=3e-5, scale=2.5, loop=(1, 3, 3))


def odd():
    """Sizes that no 16-byte vector divides, a temperature step at every position, no loop."""
    return config([normed(3, 3, 10, 9, 35, 1.5, (0.2, 1)), rotated(4, 2, 7, 5, 22, 0.5, 6), normed(2, 1, 6, 11, None, 2.0, None)],
                  vocab=61, width=50, eps=1e-4, scale=0.5)


def wide():
    """Heads at the upper sizes of the tensor-core kernels, groups of more than sixteen heads, a whole-model loop."""
    return config([normed(20, 1, 128, 128, 192, 3.0, (0.5, 64)), rotated(6, 2, 128, 64, 128, 0.09, 128),
                   rotated(10, 2, 48, 128, 128, 0.2, 16)], vocab=128, width=128, eps=1e-6, scale=11.0, loop=(0, 3, 2))


def plain():
    """One key/value head per query head, a loop that runs once, unit scales."""
    return config([rotated(2, 2, 32, 32, 64, 1.0, 32, 50.0), normed(2, 2, 32, 32, 64, 1.0, (1.0, 100))], vocab=72, width=64,
                  eps=1e-5, loop=(1, 2, 1))


def weights(cfg, seed=0):
    """bf16-representable random weights, scaled so that attention is peaked and every branch contributes."""
    g = torch.Generator().manual_seed(seed)
    C, V = cfg["width"], cfg["vocab"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / i ** 0.5).bfloat16()

    def vec(n, gain):
        return (gain * torch.randn(n, generator=g)).bfloat16()

    W = {"embed": torch.randn(V, C, generator=g).bfloat16(), "final.norm": vec(C, 0.3), "head": lin(V, C)}
    if cfg.get("loop"):
        W["loop.step"] = (0.5 * torch.randn(cfg["loop"]["times"], C, generator=g)).bfloat16()
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        W[p + "norm1"] = vec(C, 0.3)
        for n, rows, gain in (("q", H * d, 1.6), ("k", G * d, 1.6), ("v", G * vd, 1.0)):
            W[p + "mix." + n] = lin(rows, C, gain)
            if e["type"] == "attention_2":
                W[p + f"mix.{n}.b"] = vec(rows, 0.5)
        if e["type"] == "attention":
            W[p + "mix.sink"], W[p + "mix.g"] = vec(H, 2.0), lin(H * vd, C, 2.0)
        else:
            W[p + "mix.g"] = lin(H, C, 2.0)
        W[p + "mix.o"] = lin(C, H * vd)
        if e["mlp"]:
            W[p + "norm2"] = vec(C, 0.3)
            for n in ("gate", "up"):
                W[p + "mlp." + n] = lin(e["mlp"]["ff"], C, 1.3)
            W[p + "mlp.down"] = lin(C, e["mlp"]["ff"])
    return W


def build(cfg, W, device="cpu", dtype=torch.float32):
    from pisceslx_b200 import YvConfig
    from pisceslx_b200.models import build_model
    m = build_model(YvConfig.from_dict(cfg), device, dtype).eval()
    assert m.load_reference_state_dict(W) == []
    return m


def expected(cfg, W, toks, dtype=torch.float64, layers_out=None):
    with torch.no_grad():
        return oracle.forward(cfg, W, toks, dtype, layers_out).float()


def rounding_limit(cfg, W, toks, want, times=3.0):
    """Per position: what weights off by one bf16 rounding do to the plain logits (some positions are badly
    conditioned), not below the median over positions, times a factor."""
    g = torch.Generator().manual_seed(77)
    noise = torch.stack([error(expected(cfg, {k: v.float() * (1 + 2 ** -9 * torch.randn(v.shape, generator=g))
                                              for k, v in W.items()}, toks, torch.float32), want)
                         for _ in range(4)]).amax(0)
    return times * noise.clamp_min(noise.median())


CUTS = {"whole": [10_000], "token by token": [1], "pairs": [2], "uneven": [5, 64, 1, 1, 3, 130, 2, 17], "pages": [64],
        "prompt then decode": [100, 1], "inside a page": [63, 2, 65, 1, 127, 1, 2]}
