"""Latent attention of the ragged serving step (``csrc/latent_attn.cu``, ``linear_heads.cu``): the
cache holds one row ``[latent | rotated key part]`` per token for all heads.

Prompts: the rows a piece of queries sees are expanded to every head's keys and values by one product
and go through the tcgen05 kernel.  Decoding: the queries are brought into the latent space and read
the cached rows as they are.

CPU tensors take a PyTorch restatement of the same math; CUDA tensors always run the kernels.
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from . import _lib
from .decode import PAGE
from .ragged import AttnPlan, RaggedBatch, _cells, _p

_F = ctypes.c_float


def head_pitch(dim: int, vdim: int) -> int:
    """Distance of the heads in the queries and in the expanded keys and values."""
    return max(64, (max(dim, vdim) + 63) // 64 * 64)


def pieces_allowed(dim: int, vdim: int, scale: float) -> bool:
    """Whether the tcgen05 kernel takes heads of this size (``dim``: with the rotated part)."""
    return head_pitch(dim, vdim) <= 128 and scale > 0


def latent_prep(raw: torch.Tensor, doff: int, heads: int, dim: int, rot: int, rank: int,
                norm: torch.Tensor, eps: float, rope: torch.Tensor, pitch: int, batch: RaggedBatch,
                cache: torch.Tensor, page_table: torch.Tensor,
                rows_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Behind the projections ``raw`` (queries ``[heads, dim + rot]`` at column 0, the latent and the
    shared key part at ``doff``): RMS norm of the latent, rotation of neighbouring pairs of the
    rotated parts by ``rope [rows, rot / 2, 2]``, the write of the rows into the cache pages
    ``[pages, PAGE, 1, row]`` (and into the first rows of ``rows_out``).  Returns the queries
    ``[rows, heads, pitch]``, zeros behind ``dim + rot``."""
    T, row_p = raw.shape[0], cache.shape[-1]
    q = torch.empty((T, heads, pitch), dtype=raw.dtype, device=raw.device)
    if not raw.is_cuda:
        def rot_pairs(x):                                  # [rows, n, rot]
            c, s = rope[:, None, :, 0], rope[:, None, :, 1]
            a, b = x[..., 0::2], x[..., 1::2]
            return torch.stack([a * c - b * s, b * c + a * s], -1).flatten(-2)
        x = raw[:, :heads * (dim + rot)].float().view(T, heads, dim + rot)
        q.zero_()
        q[..., :dim + rot] = torch.cat([x[..., :dim], rot_pairs(x[..., dim:])], -1).to(q.dtype)
        d = raw[:, doff:doff + rank + rot].float()
        c = d[:, :rank]
        c = c * torch.rsqrt((c * c).mean(-1, keepdim=True) + eps) * norm
        rows = torch.cat([c, rot_pairs(d[:, None, rank:])[:, 0]], 1).to(raw.dtype)
        page, at = _cells(page_table, batch)
        cache[page, at, 0, :rank + rot] = rows
        if rows_out is not None:
            rows_out[:T, :rank + rot] = rows
            rows_out[:T, rank + rot:] = 0
        return q
    rc = _lib.serving_lib().cb_latent_prep(
        _p(raw), raw.stride(0), 0, doff, heads, dim, rot, rank, _p(norm), _F(eps), _p(rope), _p(q),
        pitch, _p(cache), row_p, _p(rows_out), _p(page_table), page_table.shape[1], cache.shape[0],
        _p(batch.row_slot), _p(batch.pos), T, int(raw.dtype == torch.float32),
        _p(_lib.status_buffer(raw.device)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_latent_prep")
    return q


def linear_heads(x: torch.Tensor, w: torch.Tensor, y: torch.Tensor, y_head: int, *,
                 x_rows: Optional[torch.Tensor] = None, y_rows: Optional[torch.Tensor] = None,
                 gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``y[i, h] = w[h] @ x[i, h]`` with ``x [.., heads, K']`` (its first ``K = w.shape[2]`` numbers),
    ``w [heads, N, K]``, ``y`` a ``[.., cols]`` view whose head ``h`` starts at ``h * y_head``.
    ``x_rows`` / ``y_rows`` pick the rows of ``x`` / ``y``; ``gate``, a view like ``y``, multiplies by its
    sigmoid."""
    heads, N, K = w.shape
    n = x_rows.shape[0] if x_rows is not None else (y_rows.shape[0] if y_rows is not None else x.shape[0])
    if n == 0:
        return y
    if not x.is_cuda:
        xi = (x if x_rows is None else x[x_rows.long()])[:n, :, :K].float()
        v = torch.einsum("ihk,hnk->ihn", xi, w.float())
        idx = torch.arange(n) if y_rows is None else y_rows.long()
        for h in range(heads):
            col = slice(h * y_head, h * y_head + N)
            g = 1.0 if gate is None else torch.sigmoid(gate[idx][:, col].float())
            y[idx, col] = (v[:, h] * g).to(y.dtype)
        return y
    rc = _lib.serving_lib().cb_linear_heads(
        _p(x), x.stride(0), x.stride(1), _p(x_rows), _p(w), w.stride(1), _p(y), y.stride(0), y_head,
        _p(y_rows), _p(gate), gate.stride(0) if gate is not None else 0, heads, n, N, K,
        int(x.dtype == torch.float32), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_linear_heads")
    return y


def latent_attention(q: torch.Tensor, cache: torch.Tensor, page_table: torch.Tensor,
                     batch: RaggedBatch, rows: torch.Tensor, rank: int, rot: int, scale: float,
                     window: Optional[int], max_ctx: Optional[int] = None) -> torch.Tensor:
    """Queries ``q [n, heads, row]`` in the latent space, for the batch's ``rows [n]``, over the
    cached rows of their sequences: the softmax-weighted mean of the rows' first ``rank`` numbers,
    ``[n, heads, rank rounded up to 8]``.  A position sees itself and the ``window - 1`` before it."""
    n, heads, row_p = q.shape
    rank_p = (rank + 7) // 8 * 8
    out = (torch.empty if rank_p == rank else torch.zeros)((n, heads, rank_p), dtype=q.dtype,
                                                           device=q.device)
    if n == 0:
        return out
    if not q.is_cuda:
        for i, r in enumerate(rows.tolist()):
            pos, slot = int(batch.pos[r]), int(batch.row_slot[r])
            lo = max(0, pos + 1 - window) if window else 0
            t = torch.arange(lo, pos + 1)
            k = cache[page_table[slot, t // PAGE].long(), t % PAGE, 0, :rank + rot].float()
            s = q[i, :, :rank + rot].float() @ k.t() * scale
            out[i, :, :rank] = (torch.softmax(s, -1) @ k[:, :rank]).to(out.dtype)
        return out
    f32 = q.dtype == torch.float32
    splits, part_o, part_ml = 1, None, None
    if not f32:
        ctas, ctx = n * ((heads + 15) // 16), max_ctx or batch.max_ctx
        ctx = min(ctx, window) if window else ctx
        splits = max(1, min(16, (148 + ctas // 2) // ctas, (ctx + 127) // 128))
    if splits > 1:
        part_o = torch.empty((n, heads, splits, rank), dtype=torch.float32, device=q.device)
        part_ml = torch.empty((n, heads, splits, 2), dtype=torch.float32, device=q.device)
    rc = _lib.serving_lib().cb_latent_attn(
        _p(q), _p(cache), _p(page_table), page_table.shape[1], cache.shape[0], heads, rank + rot, row_p,
        rank, rank_p, window or 0, _F(scale), _p(out), _p(rows), _p(batch.row_slot), _p(batch.pos), n,
        splits, _p(part_o), _p(part_ml), int(f32), _p(_lib.status_buffer(q.device)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_latent_attn", launches=2 if splits > 1 else 1)
    return out


def gather_rows(cache: torch.Tensor, page_table: torch.Tensor, where: torch.Tensor, n: int,
                out: torch.Tensor) -> None:
    """``n`` cached rows, the ``i``-th that of slot ``where[2 i]`` at position ``where[2 i + 1]``."""
    row_p = cache.shape[-1]
    rc = _lib.serving_lib().cb_kv_gather(
        _p(cache), _p(cache), 1, 1, row_p, row_p, _p(page_table), page_table.shape[1], cache.shape[0],
        _p(where), n, _p(out), None, row_p, row_p, _p(_lib.status_buffer(out.device)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_kv_gather")


def piece_attention(q: torch.Tensor, kv: torch.Tensor, batch: RaggedBatch, plan: AttnPlan, vdim: int,
                    scale: float, gate: Optional[torch.Tensor], out: torch.Tensor) -> None:
    """The pieces of ``plan`` through the tcgen05 kernel: ``q [rows, heads, P]``, ``kv [key rows,
    2 heads P]`` (keys, then values), ``gate`` a view like ``out [rows, heads * vdim]``."""
    n_pieces, longest, pieces = batch.plan(plan)[1], batch.plan(plan)[2], batch.plan(plan)[4]
    if not n_pieces:
        return
    T, heads, P = q.shape
    rc = _lib.serving_lib().cb_attn_fwd_pieces(
        _p(q), _p(kv), _p(kv[:, heads * P:]), _p(out), T, kv.shape[0], _p(pieces), n_pieces, longest,
        heads, heads, P, P, vdim, q.stride(0), kv.stride(0), kv.stride(0), out.stride(0), _F(scale), None,
        _p(gate), gate.stride(0) if gate is not None else 0, 1, plan.window or 0, 0, _F(0.0), _F(0.0), 1, None, _F(1.0),
        _F(0.0), _p(_lib.status_buffer(q.device)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_attn_fwd_pieces")
