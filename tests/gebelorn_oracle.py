"""Plain, slow statement of the Gebelorn design for the tests: one function per mechanism, fp64 or fp32 arithmetic on
the CPU, no code shared with the package.  Weights are a dict ``name -> tensor``; ``cfg`` is the parsed config.json."""
import math

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotary_frequencies(rot):
    """(angle per position of every pair, factor on cos and sin)."""
    dims, base = rot["dims"], float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return plain, 1.0

    def turns_to_dim(t):
        return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turns_to_dim(sc["fast"])), 0)
    hi = min(math.ceil(turns_to_dim(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """x [..., dims] at one position."""
    freq, m = rotary_frequencies(rot)
    a = torch.tensor([pos * f for f in freq], dtype=torch.float64)
    c, s = (torch.cos(a) * m).to(x.dtype), (torch.sin(a) * m).to(x.dtype)
    half = rot["dims"] // 2
    u, v = x[..., :half], x[..., half:]
    return torch.cat([u * c - v * s, v * c + u * s], -1)


def visible(i, n, window):
    """Key positions that query position i sees among the first n tokens."""
    return [j for j in range(n) if j <= i and (window is None or i - j < window)]


def attend(qn, qr, kn, kr, v, scale):
    """One query position: qn [H, dim], qr [H, rot], keys kn [J, H, dim], kr [J, rot] (shared by the heads), values
    v [J, H, vdim] -> [H, vdim]."""
    s = (torch.einsum("hd,jhd->hj", qn, kn) + torch.einsum("hd,jd->hj", qr, kr)) * scale
    return torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v)


def latent_attention(h, W, p, mx, eps):
    """h [T, width] (normed input, positions 0..T-1) -> [T, width]."""
    T = h.shape[0]
    H, dim, rd, vd, r = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    cq = rms(h @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    q = (cq @ W[p + "uq"].T).view(T, H, dim + rd)
    kv = h @ W[p + "dkv"].T
    c = rms(kv[:, :r], W[p + "dkv.norm"], eps)
    kr = torch.stack([rotate(kv[t, r:], t, mx["rot"]) for t in range(T)])
    kn = (c @ W[p + "uk"].T).view(T, H, dim)
    v = (c @ W[p + "uv"].T).view(T, H, vd)
    gate = torch.sigmoid(h @ W[p + "g"].T)
    window = (mx.get("mask") or {}).get("size")
    out = torch.zeros(T, H, vd, dtype=h.dtype)
    for t in range(T):
        js = visible(t, T, window)
        lo, hi = js[0], js[-1] + 1                       # the visible keys are one run
        out[t] = attend(q[t, :, :dim], rotate(q[t, :, dim:], t, mx["rot"]), kn[lo:hi], kr[lo:hi], v[lo:hi],
                        mx["scale"]) * gate[t][:, None]
    return out.reshape(T, H * vd) @ W[p + "o"].T


def dense_ff(h, W, p):
    return gelu_erf(h @ W[p + "up"].T) @ W[p + "down"].T


def token_side(x, tokens, W, p, side_embed, i, dim, eps):
    e = side_embed[tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return x + rms(y, W[p + "side.norm"], eps)


def forward(cfg, W, tokens, dtype=torch.float64, layers_out=None):
    """tokens (list) -> logits [T, vocab]; ``layers_out`` (a list) receives the residual stream after every layer."""
    W = {k: v.to(dtype) for k, v in W.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = rms(W["embed"][tokens], W["embed.norm"], eps)
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        a = latent_attention(rms(x, W[p + "norm1"], eps), W, p + "mix.", spec["mixer"], eps)
        x = x + rms(a, W[p + "norm1b"], eps)
        if spec.get("mlp"):
            x = x + rms(dense_ff(rms(x, W[p + "norm2"], eps), W, p + "mlp."), W[p + "norm2b"], eps)
        if cfg.get("token_side"):
            x = token_side(x, tokens, W, p, W["side.embed"], i, cfg["token_side"]["dim"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, W["final.norm"], eps) @ W["head"].T
