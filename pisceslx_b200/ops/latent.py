"""Operators of latent attention and of the fp32 residual stream of layered models (serving: no autograd).

CUDA tensors run the kernels of ``csrc/latent.cu``, ``csrc/stream.cu`` and the tcgen05 GEMM in bf16, or their
CUDA-core forms in fp32 (true 32-bit products); CPU tensors run the plain math of ``ops.reference``."""
from __future__ import annotations

from typing import Optional, Sequence, Tuple

import torch

from . import kernels, reference as ref, status_word
from . import functional as F_

_BF16 = torch.bfloat16
_ROW_TILE = 128


def _st(t: torch.Tensor) -> torch.Tensor:
    return status_word(t.device)


# --------------------------------------------------------------------------------------------------
# products
# --------------------------------------------------------------------------------------------------
def _mappable(*ts: torch.Tensor) -> bool:
    """True when every operand can be described by a tensor map: 16-byte base and row pitch."""
    return all(t.data_ptr() % 16 == 0 and t.stride(-2) * t.element_size() % 16 == 0 for t in ts)


def project(x: torch.Tensor, w: torch.Tensor, out_fp32: bool = False) -> torch.Tensor:
    """x [T, K] @ w [N, K]^T -> [T, N] in x's dtype (or fp32).  bf16 runs on the tensor cores; fp32, and operands
    whose pitch no tensor map takes, run the CUDA-core product."""
    if not x.is_cuda:
        y = torch.nn.functional.linear(x, w.to(x.dtype))
        return y.float() if out_fp32 else y
    T, N = x.shape[0], w.shape[0]
    if x.dtype == _BF16 and _mappable(x, w) and (N * (4 if out_fp32 else 2)) % 16 == 0:
        return F_.linear(x, w, out_fp32=out_fp32)
    out = torch.empty(T, N, dtype=torch.float32 if out_fp32 else x.dtype, device=x.device)
    kernels().linear_simt(x.unsqueeze(0), w.unsqueeze(0), out.unsqueeze(0))
    return out


def project_onto(x: torch.Tensor, z: torch.Tensor, w: torch.Tensor) -> Optional[torch.Tensor]:
    """x += z [T, K] @ w [N, K]^T on the fp32 stream x [T, N].  The tensor-core product adds to x itself; a skinny one
    is cut along K and returns its fp32 parts [slices, rows, N] for ``stream_add`` to sum (as do products that run on
    the CUDA cores or the CPU, in one part): None means that x already holds the sum."""
    if not x.is_cuda:
        return torch.nn.functional.linear(z, w.to(z.dtype)).float()
    if z.dtype == _BF16 and _mappable(z, w) and x.shape[1] % 4 == 0:
        parts = F_.skinny_parts(z, w)
        if parts is None:
            kernels().gemm(z, w, x, False, False, True, 0, _st(z))
        return parts
    out = torch.empty_like(x)
    kernels().linear_simt(z.unsqueeze(0), w.unsqueeze(0), out.unsqueeze(0))
    return out


def head_rows(batch: int, like: torch.Tensor) -> int:
    """Rows to allocate per head for ``project_heads``: the tensor-core product takes whole 128-row tiles."""
    return -(-batch // _ROW_TILE) * _ROW_TILE if like.is_cuda and like.dtype == _BF16 else batch


def project_heads(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, rows: int) -> None:
    """out[h, :rows] = a[h, :rows] @ w[h]^T for every head; a [H, R, K], w [H, N, K], out [H, R, N] (row-pitched views
    of stacked heads).  Rows past ``rows`` are padding: their content is not defined."""
    if not a.is_cuda:
        out[:, :rows] = torch.einsum("hmk,hnk->hmn", a[:, :rows], w.to(a.dtype))
        return
    stacked = all(t.stride(0) == t.shape[1] * t.stride(1) for t in (a, w, out))
    if a.dtype == _BF16 and a.shape[1] % _ROW_TILE == 0 and stacked and _mappable(a, w, out):
        kernels().gemm_batched(a, w, out, False, False, False, 0, _st(a))
        return
    kernels().linear_simt(a[:, :rows], w, out[:, :rows])


# --------------------------------------------------------------------------------------------------
# residual stream
# --------------------------------------------------------------------------------------------------
def stream_norm(x: torch.Tensor, y: Optional[torch.Tensor], w_y: Optional[torch.Tensor], w_h: Optional[torch.Tensor],
                eps: float, dtype: torch.dtype, rows: Optional[torch.Tensor] = None, start: bool = False,
                want_h: bool = True) -> Optional[torch.Tensor]:
    """One pass over the fp32 stream ``x`` [T, C], updated in place: ``x += rms(y) * w_y`` (``start``: ``x = ...``;
    ``rows``: row t of the branch is ``y[rows[t]]``), then returns ``rms(x) * w_h`` (or ``x`` itself when ``w_h`` is
    None) in ``dtype``."""
    if not x.is_cuda:
        if y is not None:
            b = ref.rms_norm((y if rows is None else y[rows]).float(), w_y.float(), eps)
            x.copy_(b if start else x + b)
        if not want_h:
            return None
        return (x if w_h is None else ref.rms_norm(x, w_h.float(), eps)).to(dtype, copy=True)
    h = torch.empty(x.shape, dtype=dtype, device=x.device) if want_h else None
    kernels().stream_norm(x, y, rows, w_y, w_h, h, start, eps, _st(x))
    return h


def stream_add(x: torch.Tensor, parts: Optional[torch.Tensor], norms: Sequence[torch.Tensor], offset: float, eps: float,
               dtype: torch.dtype, table: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None,
               table_scale: float = 1.0, vec: Optional[torch.Tensor] = None, start: bool = False) -> Tuple[torch.Tensor, ...]:
    """One pass over the fp32 stream ``x`` [T, C], updated in place: ``x += sum(parts) + table_scale * table[rows] + vec``
    (each optional; ``start``: ``x = ...``).  ``parts`` is [T, C], or [slices, rows >= T, C] to be summed.  Returns
    ``x / sqrt(mean(x^2) + eps) * (offset + w)`` in ``dtype`` for each of up to two ``norms``."""
    if not x.is_cuda:
        new = torch.zeros_like(x) if start else x.clone()
        if parts is not None:
            new += parts.float() if parts.dim() == 2 else parts[:, :x.shape[0]].float().sum(0)
        if table is not None:
            new += table[rows].float() * table_scale
        if vec is not None:
            new += vec.float()
        x.copy_(new)
        return tuple(ref.rms_norm(x, offset + w.float(), eps).to(dtype, copy=True) for w in norms)
    hs = tuple(torch.empty(x.shape, dtype=dtype, device=x.device) for _ in norms)
    two = len(norms) > 1
    kernels().stream_add(x, parts, table, rows if table is not None else None, table_scale, vec, start,
                         norms[0] if norms else None, norms[1] if two else None, offset, eps, hs[0] if norms else None,
                         hs[1] if two else None, _st(x))
    return hs


def swiglu(gate_up: torch.Tensor, out: torch.Tensor) -> None:
    """out [T, F] (a column range) = silu(gate) * up of gate_up [T, 2 F] = [gate | up]."""
    if not gate_up.is_cuda:
        out.copy_(ref.swiglu(gate_up))
        return
    kernels().gated_silu(gate_up, out)


def gelu(x: torch.Tensor) -> torch.Tensor:
    """x * Phi(x) with the error function."""
    if not x.is_cuda:
        return torch.nn.functional.gelu(x)
    out = torch.empty_like(x)
    kernels().gelu(x, out)
    return out


def token_gate(a: torch.Tensor, table: torch.Tensor, offset: int, tokens: torch.Tensor) -> torch.Tensor:
    """gelu_tanh(a) * table[tokens, offset : offset + a.shape[1]]"""
    if not a.is_cuda:
        e = table[tokens][:, offset:offset + a.shape[1]]
        return (torch.nn.functional.gelu(a.float(), approximate="tanh") * e.float()).to(a.dtype)
    out = torch.empty(a.shape, dtype=a.dtype, device=a.device)
    kernels().token_gate(a, table, offset, tokens, out, _st(a))
    return out


# --------------------------------------------------------------------------------------------------
# latent attention
# --------------------------------------------------------------------------------------------------
def latent_prep(y: torch.Tensor, q_rank: int, kv_rank: int, rot_dim: int, w_q: torch.Tensor, w_kv: torch.Tensor,
                cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor, eps: float,
                cache: Optional[torch.Tensor] = None, slot_map: Optional[torch.Tensor] = None,
                want_rows: bool = True) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """y [T, >= q_rank + kv_rank + rot_dim] = [query latent | key/value latent | shared key part | ...] ->
    (normed query latent [T, q_rank], rows [T, kv_rank + rot_dim] = [normed latent | rotated key part]); the rows are
    also stored at ``slot_map`` of the paged ``cache`` (-1 = not stored)."""
    T, row = y.shape[0], kv_rank + rot_dim
    if not y.is_cuda:
        cq = ref.rms_norm(y[:, :q_rank], w_q, eps)
        c = ref.rms_norm(y[:, q_rank:q_rank + kv_rank], w_kv, eps)
        kr = ref.apply_rope(y[:, q_rank + kv_rank:q_rank + row].unsqueeze(1), cos, sin, positions, rot_dim).squeeze(1)
        rows = torch.cat([c, kr], 1)
        if cache is not None:
            keep = slot_map >= 0
            cache.view(-1, row)[slot_map[keep].long()] = rows[keep]
        return cq, rows if want_rows else None
    cq = torch.empty(T, q_rank, dtype=y.dtype, device=y.device)
    rows = torch.empty(T, row, dtype=y.dtype, device=y.device) if want_rows else None
    kernels().latent_prep(y, q_rank, kv_rank, rot_dim, w_q, w_kv, cos, sin, positions, cq, rows, cache,
                          slot_map if cache is not None else None, eps, _st(y))
    return cq, rows


def latent_query(q: torch.Tensor, heads: int, dim: int, rot_dim: int, cos: torch.Tensor, sin: torch.Tensor,
                 positions: torch.Tensor) -> torch.Tensor:
    """Rotates the last ``rot_dim`` numbers of every head of q [T, heads * (dim + rot_dim)]; returns q (in place on a
    GPU)."""
    if not q.is_cuda:
        T = q.shape[0]
        x = q.view(T, heads, dim + rot_dim)
        return torch.cat([x[..., :dim], ref.apply_rope(x[..., dim:], cos, sin, positions, rot_dim)], -1).reshape(T, -1)
    kernels().latent_query(q, heads, dim, rot_dim, cos, sin, positions, None, None, _st(q))
    return q


def latent_query_absorbed(q: torch.Tensor, w_uk: torch.Tensor, rot_dim: int, cos: torch.Tensor, sin: torch.Tensor,
                          positions: torch.Tensor) -> torch.Tensor:
    """The latent-space query of a decode step: q [B, heads * (dim + rot_dim)], w_uk [heads, kv_rank, dim] (the key map
    transposed per head) -> [heads, R, kv_rank + rot_dim] = [W_uk^T q | rotated part], R >= B rows."""
    heads, r, dim = w_uk.shape
    B = q.shape[0]
    R = head_rows(B, q)
    q_lat = torch.empty(heads, R, r + rot_dim, dtype=q.dtype, device=q.device)
    if not q.is_cuda:
        x = q.view(B, heads, dim + rot_dim)
        nope = x[..., :dim].transpose(0, 1).contiguous()
        q_lat[:, :, r:] = ref.apply_rope(x[..., dim:], cos, sin, positions, rot_dim).transpose(0, 1)
    else:
        nope = torch.empty(heads, R, dim, dtype=q.dtype, device=q.device)
        kernels().latent_query(q, heads, dim, rot_dim, cos, sin, positions, nope, q_lat, _st(q))
    project_heads(nope, w_uk, q_lat[:, :, :r], B)
    return q_lat


def latent_gather(cache: torch.Tensor, slots: torch.Tensor) -> torch.Tensor:
    """Rows of the paged cache at flat ``slots`` (int32)."""
    row = cache.shape[-1]
    if not cache.is_cuda:
        return cache.view(-1, row)[slots.long()]
    out = torch.empty(slots.numel(), row, dtype=cache.dtype, device=cache.device)
    kernels().latent_gather(cache, slots, out, _st(cache))
    return out


def latent_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, kr: torch.Tensor, gate: Optional[torch.Tensor],
                     cu_q: torch.Tensor, cu_k: torch.Tensor, max_q: int, heads: int, window: Optional[int],
                     scale: float, simt: bool = False) -> torch.Tensor:
    """Attention of packed portions over reconstructed keys / values: q [Tq, heads * (dim + rot)] rotated,
    k [Tk, heads * dim], v [Tk, heads * vdim], kr [Tk, rot] rotated and shared by the heads.  The last query of a
    sequence sits at its last key; a query sees itself and the ``window - 1`` keys before it (None: all before it).
    ``gate`` [Tq, heads]: logits of a sigmoid on every head's output."""
    if not q.is_cuda:
        return ref.latent_attention(q, k, v, kr, gate, cu_q, cu_k, heads, window, scale)
    o = torch.empty(q.shape[0], v.shape[1], dtype=q.dtype, device=q.device)
    kernels().latent_attn(q, k, v, kr, gate, o, cu_q, cu_k, max_q, heads, window or 0, scale, simt, _st(q))
    return o


def decode_splits(batch: int, heads: int, table_width: int, block: int, window: Optional[int], row: int = 576) -> int:
    """Key ranges per sequence of the latent decode kernel.  It depends on shapes only (so that a captured step can be
    replayed): the count that minimises the waves of CTAs times the pages of one CTA, with two pages' time for a CTA's
    start and end.  A small row lets two CTAs share an SM."""
    pages = table_width if not window else min(table_width, -(-window // block) + 1)
    ctas, room = batch * -(-heads // 64), 148 * (2 if row <= 192 else 1)
    best = min(range(1, min(32, max(pages, 1)) + 1), key=lambda s: (-(-ctas * s // room) * (-(-pages // s) + 2), s))
    return best


def latent_decode(q_lat: torch.Tensor, cache: torch.Tensor, kv_rank: int, block_table: torch.Tensor,
                  seq_lens: torch.Tensor, window: Optional[int], scale: float, simt: bool = False,
                  splits: int = 0) -> torch.Tensor:
    """Weighted sums of the cached latents for one query token per sequence: q_lat [heads, R, kv_rank + rot] ->
    [heads, R, kv_rank] (rows past the batch are padding)."""
    heads, R, _ = q_lat.shape
    B = seq_lens.numel()
    if not q_lat.is_cuda:
        return ref.latent_decode(q_lat, cache, kv_rank, block_table, seq_lens, window, scale)
    out = torch.empty(heads, R, kv_rank, dtype=q_lat.dtype, device=q_lat.device)
    if splits <= 0:
        splits = decode_splits(B, heads, block_table.shape[1], cache.shape[1], window, cache.shape[2])
    po = pml = None
    if splits > 1:
        po = torch.empty(B * heads * splits * kv_rank, dtype=torch.float32, device=q_lat.device)
        pml = torch.empty(B * heads * splits * 2, dtype=torch.float32, device=q_lat.device)
    kernels().latent_decode(q_lat, cache, block_table, seq_lens, out, po, pml, splits, window or 0, scale, simt,
                            _st(q_lat))
    return out


def latent_values(o_lat: torch.Tensor, w_uv: torch.Tensor, gate: Optional[torch.Tensor], batch: int) -> torch.Tensor:
    """The value map of every head on its weighted latent, gated: o_lat [heads, R, kv_rank], w_uv [heads, vdim,
    kv_rank], gate logits [B, heads] -> [B, heads * vdim]."""
    heads, R, _ = o_lat.shape
    vdim = w_uv.shape[1]
    v = torch.empty(heads, R, vdim, dtype=o_lat.dtype, device=o_lat.device)
    project_heads(o_lat, w_uv, v, batch)
    if not o_lat.is_cuda:
        o = v[:, :batch].transpose(0, 1)
        if gate is not None:
            o = o * torch.sigmoid(gate.float()).to(o.dtype).unsqueeze(-1)
        return o.reshape(batch, heads * vdim)
    out = torch.empty(batch, heads * vdim, dtype=o_lat.dtype, device=o_lat.device)
    kernels().head_gate(v, gate, out)
    return out
