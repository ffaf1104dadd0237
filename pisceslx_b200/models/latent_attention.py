"""``YvWindowedLatentAttention``: attention over a low-rank latent with a sliding window, served from latent pages.

Per token the layer keeps ``[c | r]``: the normed key/value latent (``kv_rank``) and one rotated key part shared by the
heads (``rot_dim``).  With per-head maps K_h, V_h of the latent the score of query q and cached token s is
``(q_plain . K_h c_s + q_rot . r_s) * scale`` and the output ``sum_s w_s V_h c_s`` times a sigmoid gate per head.

* A portion of a prompt (any start) reconstructs keys and values of its own tokens and of the window in front of it
  from the pages and runs the flash kernel.
* A decode step folds K_h into the query and applies V_h to the weighted latent, so that it reads only the pages.

Both read what the pages hold, so a position's result does not depend on how the sequence was cut.  The projections
that share an input are one product: ``in_proj`` = query latent, key/value latent with the shared key part, gate;
``kv_up`` = all heads' keys, then all heads' values."""
from __future__ import annotations

import math
from typing import Any, Dict, Optional, Tuple

import torch
import torch.nn as nn

from ..ops import latent as L
from .attention import AttnContext
from .norms import YvRotaryEmbedding


def rotary_for(spec: Dict[str, Any]) -> YvRotaryEmbedding:
    """Angle tables of a layer's ``rotation`` entry (``dims``, ``base`` and optionally ``yarn``)."""
    y = spec.get("yarn")
    if not y:
        return YvRotaryEmbedding(spec["dims"], 1024, spec["base"])
    return YvRotaryEmbedding(spec["dims"], 1024, spec["base"], "yarn", y["factor"], y["original"],
                             {"beta_fast": y["fast"], "beta_slow": y["slow"], "ramp_end": spec["dims"] - 1,
                              "magnitude": 0.1 * math.log(y["factor"]) + 1.0})


class YvWindowedLatentAttention(nn.Module):
    def __init__(self, hidden: int, spec: Dict[str, Any], layer_idx: int, eps: float, rotary: YvRotaryEmbedding,
                 init_std: float = 0.02):
        super().__init__()
        self.layer_idx, self.eps, self.rotary = layer_idx, eps, rotary
        self.heads, self.dim, self.rot_dim = spec["heads"], spec["dim"], spec["rot_dim"]
        self.vdim, self.kv_rank, self.q_rank = spec["vdim"], spec["kv_rank"], spec["q_rank"]
        self.window: Optional[int] = spec["window"]
        self.scale = float(spec["scale"])
        self.gated = bool(spec.get("output_gate", False))
        self.row = self.kv_rank + self.rot_dim
        gate_rows = self.heads if self.gated else 0
        # the gate's columns start 16 bytes aligned and the product has a whole number of 16-byte columns
        self.gate_col = -(-(self.q_rank + self.row) // 8) * 8
        self.in_rows = -(-(self.gate_col + gate_rows) // 8) * 8
        H, hd = self.heads, self.dim + self.rot_dim
        mk = lambda *s: nn.Parameter(torch.empty(*s).normal_(std=init_std), requires_grad=False)
        self.in_proj = mk(self.in_rows, hidden)
        self.in_proj.data[self.q_rank + self.row:self.gate_col].zero_()
        self.in_proj.data[self.gate_col + gate_rows:].zero_()
        self.q_norm = nn.Parameter(torch.ones(self.q_rank), requires_grad=False)
        self.kv_norm = nn.Parameter(torch.ones(self.kv_rank), requires_grad=False)
        self.q_up = mk(H * hd, self.q_rank)
        self.kv_up = mk(H * (self.dim + self.vdim), self.kv_rank)
        self.o_proj = mk(hidden, H * self.vdim)
        self._key_map: Optional[torch.Tensor] = None

    # -- weights ---------------------------------------------------------------------------------------------------
    @property
    def k_up(self) -> torch.Tensor:
        return self.kv_up[: self.heads * self.dim]

    @property
    def v_up(self) -> torch.Tensor:
        return self.kv_up[self.heads * self.dim:]

    def key_map(self) -> torch.Tensor:
        """[heads, kv_rank, dim]: the key map of every head transposed, built once (decode folds it into the query)."""
        m = self._key_map
        if m is None or m.device != self.kv_up.device or m.dtype != self.kv_up.dtype:
            m = self.k_up.view(self.heads, self.dim, self.kv_rank).transpose(1, 2).contiguous()
            self._key_map = m
        return m

    def checkpoint_slices(self) -> Dict[str, torch.Tensor]:
        """Checkpoint name (without the layer's prefix) -> view of the parameter that holds it."""
        q, g = self.q_rank, self.gate_col
        out = {"dq": self.in_proj[:q], "dq.norm": self.q_norm, "uq": self.q_up, "dkv": self.in_proj[q:q + self.row],
               "dkv.norm": self.kv_norm, "uk": self.k_up, "uv": self.v_up, "o": self.o_proj}
        if self.gated:
            out["g"] = self.in_proj[g:g + self.heads]
        return out

    def weights_changed(self) -> None:
        self._key_map = None

    # -- forward -----------------------------------------------------------------------------------------------------
    def _angles(self, ctx: AttnContext, device: torch.device) -> Tuple[torch.Tensor, torch.Tensor]:
        return self.rotary.tables(ctx.max_position or ctx.max_len, device)

    def forward(self, h: torch.Tensor, ctx: AttnContext, run: Optional[int] = None) -> torch.Tensor:
        """h [T, hidden] (normed input, packed tokens) -> [T, hidden]; ``run`` names the cache of a layer that runs more
        than once."""
        cos, sin = self._angles(ctx, h.device)
        y = L.project(h, self.in_proj)
        cache = ctx.cache.rows(self.layer_idx if run is None else run) if ctx.cache is not None else None
        cq, rows = L.latent_prep(y, self.q_rank, self.kv_rank, self.rot_dim, self.q_norm, self.kv_norm, cos, sin,
                                 ctx.positions, self.eps, cache, ctx.slot_map, want_rows=not ctx.decode)
        gate = y[:, self.gate_col:self.gate_col + self.heads] if self.gated else None
        q = L.project(cq, self.q_up)
        if ctx.decode:
            o = self._decode(q, gate, cache, cos, sin, ctx)
        else:
            o = self._portion(q, rows, gate, cache, cos, sin, ctx)
        return L.project(o, self.o_proj)

    def _portion(self, q, rows, gate, cache, cos, sin, ctx: AttnContext) -> torch.Tensor:
        q = L.latent_query(q, self.heads, self.dim, self.rot_dim, cos, sin, ctx.positions)
        slots, cu_k = ctx.visible_context(self.window)
        if slots is not None:                       # the portion continues a sequence: its window starts in the pages
            rows = L.latent_gather(cache, slots)
        kv = L.project(rows[:, :self.kv_rank], self.kv_up)
        nk = self.heads * self.dim
        return L.latent_attention(q, kv[:, :nk], kv[:, nk:], rows[:, self.kv_rank:], gate, ctx.cu_seqlens, cu_k,
                                  ctx.max_len, self.heads, self.window, self.scale)

    def _decode(self, q, gate, cache, cos, sin, ctx: AttnContext) -> torch.Tensor:
        B = q.shape[0]
        q_lat = L.latent_query_absorbed(q, self.key_map(), self.rot_dim, cos, sin, ctx.positions)
        o_lat = L.latent_decode(q_lat, cache, self.kv_rank, ctx.block_table, ctx.seq_lens, self.window, self.scale)
        return L.latent_values(o_lat, self.v_up.view(self.heads, self.vdim, self.kv_rank), gate, B)
