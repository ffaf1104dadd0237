"""Operators of grouped-query attention over pages of keys and values, with heads of any size, sinks and output gates
(serving: no autograd).

CUDA tensors run the kernels of ``csrc/grouped.cu``: tensor-core kernels in bf16, CUDA-core forms in fp32 and for sizes
the tensor-core kernels do not take; CPU tensors run the plain math of ``ops.reference``."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from . import kernels, reference as ref, status_word
from .functional import paged_splits


def _st(t: torch.Tensor) -> torch.Tensor:
    return status_word(t.device)


def grouped_prep(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, bias: Optional[torch.Tensor], bias_at: List[int],
                 heads: int, kv_heads: int, k_pages: torch.Tensor, v_pages: torch.Tensor, slots: Optional[torch.Tensor],
                 positions: torch.Tensor, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor], rot_dims: int,
                 unit: bool, temperature: Optional[Dict[str, float]], eps: float) -> None:
    """Finishes the projections q [T, heads * dim], k [T, kv_heads * dim], v [T, kv_heads * vdim] (column ranges of one
    product): adds ``bias`` (their parts start at ``bias_at``), divides every query and key head by its root mean square
    (``unit``), rotates the first ``rot_dims`` numbers of every query and key head, and multiplies the queries by
    ``1 + coef ln(floor((position + 1) / every) + 1)`` (``temperature``).  Queries stay in place; keys and values go to
    the pages [blocks, block, kv_heads, size] at flat ``slots`` (-1 = not stored; None: token t at slot t)."""
    if not q.is_cuda:
        ref.grouped_prep(q, k, v, bias, bias_at, heads, kv_heads, k_pages, v_pages, slots, positions, cos, sin, rot_dims,
                         unit, temperature, eps)
        return
    coef, every = (float(temperature["coef"]), int(temperature["every"])) if temperature else (0.0, 0)
    kernels().grouped_prep(q, k, v, bias, bias_at[0], bias_at[1], bias_at[2], heads, kv_heads, k_pages, v_pages, slots,
                           positions, cos, sin, rot_dims, unit, coef, every, eps, _st(q))


def grouped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, table: Optional[torch.Tensor],
                      lens: Optional[torch.Tensor], cu_q: torch.Tensor, max_q: int, heads: int, scale: float,
                      sink: Optional[torch.Tensor], gate: Optional[torch.Tensor], out: torch.Tensor,
                      simt: bool = False) -> None:
    """Causal attention of packed portions over pages: q [Tq, heads * dim], pages k [blocks, block, kv_heads, dim] and
    v [.., vdim], block ``table`` [B, W] with ``lens`` [B] tokens (the last query of a sequence sits at its last token;
    without a table the tokens of the batch are the slots, one after the other).  ``sink`` [heads]: logits that only
    count in the denominator.  ``gate`` [Tq, heads] or [Tq, heads * vdim]: logits of a sigmoid on the output.  The
    result goes to ``out`` [Tq, heads * vdim], which may be a column range."""
    if not q.is_cuda:
        ref.grouped_attention(q, k, v, table, lens, cu_q, heads, scale, sink, gate, out)
        return
    kernels().grouped_attn(q, k, v, table, lens, cu_q, max_q, heads, scale, sink, gate, out, simt, _st(q))


def grouped_decode(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, table: torch.Tensor, lens: torch.Tensor, heads: int,
                   scale: float, sink: Optional[torch.Tensor], gate: Optional[torch.Tensor], out: torch.Tensor,
                   simt: bool = False, splits: int = 0) -> None:
    """One query token per sequence: q [B, heads * dim] over the pages -> ``out`` [B, heads * vdim] (a column range);
    sinks and gates as in ``grouped_attention``."""
    if not q.is_cuda:
        cu = torch.arange(q.shape[0] + 1, dtype=torch.int32)
        ref.grouped_attention(q, k, v, table, lens, cu, heads, scale, sink, gate, out)
        return
    B, kv_heads, vdim = q.shape[0], k.shape[2], v.shape[3]
    if splits <= 0:
        small = max(q.shape[1] // heads, vdim) <= 64
        splits = paged_splits(B * kv_heads * -(-(heads // kv_heads) // 16), table.shape[1], 2 if small else 1)
    po = pml = None
    if splits > 1:
        po = torch.empty(B * heads * splits * vdim, dtype=torch.float32, device=q.device)
        pml = torch.empty(B * heads * splits * 2, dtype=torch.float32, device=q.device)
    kernels().grouped_decode(q, k, v, table, lens, heads, scale, sink, gate, out, po, pml, splits, simt, _st(q))
