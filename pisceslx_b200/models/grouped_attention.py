"""``YvGroupedAttention``: grouped-query attention of layered models, served from pages of keys and values.

Options of the spec, each on its own: sizes of a query / key head (``dim``) and of a value head (``vdim``), projection
biases, RMS norm of every query and key head without a weight, rotation of a part of the head, a query factor that grows
with the position, a learned sink in the softmax, and a sigmoid gate on the output per head or per number.

The projections that share the input are one product, ``in_proj`` = [queries | keys | values | gate].  ``grouped_prep``
finishes queries in place and stores keys and values in the pages; a portion of a prompt (any start) and a decode step
both attend over what the pages hold, so a position's result does not depend on how the sequence was cut.  The gated
heads can be written straight into a wider buffer (``attend``), which is how a block joins this layer's output product
with the feed-forward's."""
from __future__ import annotations

from typing import Any, Dict, Optional

import torch
import torch.nn as nn

from ..ops import grouped as G
from ..ops import latent as L
from .attention import AttnContext
from .norms import YvRotaryEmbedding


def _up8(n: int) -> int:
    return -(-n // 8) * 8


class YvGroupedAttention(nn.Module):
    def __init__(self, hidden: int, spec: Dict[str, Any], layer_idx: int, eps: float,
                 rotary: Optional[YvRotaryEmbedding], init_std: float = 0.02, own_output: bool = True):
        super().__init__()
        self.layer_idx, self.eps, self.rotary = layer_idx, eps, rotary
        self.heads, self.kv_heads, self.dim, self.vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not divide over {self.kv_heads} key/value heads")
        self.scale = float(spec["scale"])
        self.qk_norm, self.temperature = bool(spec.get("qk_norm", False)), spec.get("temperature")
        self.gate_kind: Optional[str] = spec.get("output_gate")
        self.out_width = self.heads * self.vdim
        gate = {None: 0, "head": self.heads, "element": self.out_width}[self.gate_kind]
        # every part starts 16 bytes aligned and the product has a whole number of 16-byte columns
        sizes = {"q": self.heads * self.dim, "k": self.kv_heads * self.dim, "v": self.kv_heads * self.vdim, "g": gate}
        self.parts, at = {}, 0
        for name, n in sizes.items():
            self.parts[name] = slice(at, at + n)
            at += _up8(n)
        mk = lambda *s: nn.Parameter(torch.empty(*s).normal_(std=init_std), requires_grad=False)
        self.in_proj = mk(at, hidden)
        self.in_bias = nn.Parameter(torch.zeros(at), requires_grad=False) if spec.get("bias") else None
        end = 0
        for sl in self.parts.values():                       # rows between the parts belong to none
            self.in_proj.data[end:sl.start].zero_()
            end = sl.stop
        self.in_proj.data[end:].zero_()
        self.sink = mk(self.heads) if spec.get("sink") else None
        self.o_proj = mk(hidden, self.out_width) if own_output else None

    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        """Checkpoint name (without the layer's prefix) -> view of the parameter that holds it."""
        out = {n: self.in_proj[self.parts[n]] for n in ("q", "k", "v")}
        if self.in_bias is not None:
            out.update({n + ".b": self.in_bias[self.parts[n]] for n in ("q", "k", "v")})
        if self.gate_kind is not None:
            out["g"] = self.in_proj[self.parts["g"]]
        if self.sink is not None:
            out["sink"] = self.sink
        if self.o_proj is not None:
            out["o"] = self.o_proj
        return out

    def attend(self, h: torch.Tensor, ctx: AttnContext, run: Optional[int], out: torch.Tensor) -> None:
        """h [T, hidden] (normed input, packed tokens) -> gated heads in ``out`` [T, heads * vdim] (a column range)."""
        y = L.project(h, self.in_proj)
        T, P = y.shape[0], self.parts
        cos = sin = None
        rot = 0
        if self.rotary is not None:
            rot = self.rotary.rot_dim
            cos, sin = self.rotary.tables(ctx.max_position or ctx.max_len, h.device)
        if ctx.cache is not None:
            k, v = ctx.cache.layer(self.layer_idx if run is None else run)
            slots = ctx.slot_map
        else:
            k = torch.empty(T, 1, self.kv_heads, self.dim, dtype=y.dtype, device=y.device)
            v = torch.empty(T, 1, self.kv_heads, self.vdim, dtype=y.dtype, device=y.device)
            slots = None
        q = y[:, P["q"]]
        G.grouped_prep(q, y[:, P["k"]], y[:, P["v"]], self.in_bias, [P[n].start for n in "qkv"], self.heads, self.kv_heads,
                       k, v, slots, ctx.positions, cos, sin, rot, self.qk_norm, self.temperature, self.eps)
        gate = y[:, P["g"]] if self.gate_kind is not None else None
        if ctx.decode:
            G.grouped_decode(q, k, v, ctx.block_table, ctx.seq_lens, self.heads, self.scale, self.sink, gate, out)
            return
        table, lens = ctx.pages() if ctx.cache is not None else (None, None)
        G.grouped_attention(q, k, v, table, lens, ctx.cu_seqlens, ctx.max_len, self.heads, self.scale, self.sink, gate, out)

    def forward(self, h: torch.Tensor, ctx: AttnContext, run: Optional[int] = None) -> torch.Tensor:
        out = torch.empty(h.shape[0], self.out_width, dtype=h.dtype, device=h.device)
        self.attend(h, ctx, run, out)
        return L.project(out, self.o_proj)
