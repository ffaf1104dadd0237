"""Plain, slow statement of the Pitolix design for the tests: one function per mechanism, fp64 or fp32 arithmetic on the
CPU, no code shared with the package.  Weights are a dict ``name -> tensor``; ``cfg`` is the parsed config.json."""
import math

import torch


def unit(x, eps):
    """x over its root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """The weight is stored as its distance from one."""
    return unit(x, eps) * (1.0 + w)


def rotate(x, pos, rot):
    """x [..., dim] at one position: pairs (i, i + dims / 2) of the first ``dims`` numbers turn, the rest stays."""
    dims, half = rot["dims"], rot["dims"] // 2
    a = torch.tensor([pos * float(rot["base"]) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def temperature(pos, temp):
    """Factor on the query at a position: grows by a step every ``every`` positions."""
    return 1.0 + temp["coef"] * math.log((pos + 1) // temp["every"] + 1)


def weights_of(scores, sink=None):
    """Softmax over the last dimension; ``sink`` [H] adds exp(sink) to every denominator of its head."""
    top = scores.amax(-1, keepdim=True)
    if sink is not None:
        top = torch.maximum(top, sink[:, None])
    e = torch.exp(scores - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink[:, None] - top)
    return e / total


def attend(q, k, v, scale, sink=None):
    """One query position: q [H, dim] over keys k [J, G, dim] and values v [J, G, vdim], H / G heads to a group."""
    per = q.shape[0] // k.shape[1]
    kh, vh = k.repeat_interleave(per, 1), v.repeat_interleave(per, 1)
    w = weights_of(torch.einsum("hd,jhd->hj", q, kh) * scale, sink)
    return torch.einsum("hj,jhd->hd", w, vh)


def mixer(kind, h, W, p, mx, eps):
    """h [T, width] (normed input, positions 0..T-1) -> [T, width]."""
    T, H, G, d, vd = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    proj = lambda n: h @ W[p + n].T + (W[p + n + ".b"] if kind == "attention_2" else 0.0)
    q, k, v = proj("q").view(T, H, d), proj("k").view(T, G, d), proj("v").view(T, G, vd)
    gate = torch.sigmoid(h @ W[p + "g"].T)
    sink = None
    if kind == "attention":
        q, k, sink = unit(q, eps), unit(k, eps), W[p + "sink"]
        if mx.get("q_temp"):
            q = torch.stack([q[t] * temperature(t, mx["q_temp"]) for t in range(T)])
        gate = gate.view(T, H, vd)
    else:
        q = torch.stack([rotate(q[t], t, mx["rot"]) for t in range(T)])
        k = torch.stack([rotate(k[t], t, mx["rot"]) for t in range(T)])
        gate = gate.view(T, H, 1)
    o = torch.stack([attend(q[t], k[:t + 1], v[:t + 1], mx["scale"], sink) for t in range(T)]) * gate
    return o.reshape(T, H * vd) @ W[p + "o"].T


def feed_forward(h, W, p):
    z = h @ W[p + "gate"].T
    return (z * torch.sigmoid(z) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def layer(x, W, i, spec, eps):
    """Both branches read the same stream."""
    y = mixer(spec["type"], norm(x, W[f"l{i}.norm1"], eps), W, f"l{i}.mix.", spec["mixer"], eps)
    if spec.get("mlp"):
        y = y + feed_forward(norm(x, W[f"l{i}.norm2"], eps), W, f"l{i}.mlp.")
    return x + y


def order(cfg):
    """(layer, pass or None, first layer of its pass) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None, False) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t, i == a) for i in range(a, b)]
    return out + [(i, None, False) for i in range(b, n)]


def forward(cfg, W, tokens, dtype=torch.float64, layers_out=None):
    """tokens (list) -> logits [T, vocab]; ``layers_out`` (a list) receives the residual stream after every layer run."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    start = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = start
    for i, t, first in order(cfg):
        if first:
            x = x + (start if t > 0 else 0.0) + W["loop.step"][t]
        x = layer(x, W, i, cfg["layers"][i], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, W["final.norm"], eps) @ W["head"].T
