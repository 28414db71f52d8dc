"""Ops of the ragged serving step (``csrc/ragged_rows.cu``, ``residual.cu``, ``shortconv.cu``,
``delta_scan.cu``, ``ragged_attn.cu``; latent attention and further recurrences have modules of their
own): one batch holds portions of prompts beside single decoded tokens, each at its
own position of its own sequence, and recurrent and cached state is addressed by slot.

CPU tensors take a PyTorch restatement of the same math; CUDA tensors always run the kernels, in
bf16 or (for a model held in fp32) in full fp32.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import numpy as np
import torch

from . import _lib
from .decode import PAGE

CONV_TILE = 16        # tokens per block of the convolution kernels
ATTN_TILE = 64        # query rows per block of the tensor-core attention kernel
ROWS_MAX = 4          # entries of at most this many tokens take the row kernel
MIN_PIECE = 64        # chunks from this size on are worth a piece of their own
WINDOW_PIECE = 256    # query rows of a piece under a sliding window
_F = ctypes.c_float


def _p(t):
    return _lib.ptr(t)


@dataclass
class Entry:
    """The next ``tokens`` of the sequence in ``slot``, which already holds ``pos0`` tokens;
    ``want`` lists the places among them whose logits are asked for."""

    slot: int
    pos0: int
    tokens: Sequence[int]
    want: Sequence[int] = ()


@dataclass(frozen=True)
class AttnPlan:
    """How the long entries of a batch go through attention under one mask.  The rows of an entry
    that lie in one chunk form a piece for the tcgen05 kernel.  A piece that starts at its chunk's
    start (or at position 0) needs only this step's keys and values; one that continues a chunk
    also needs the cached ones, which are gathered into rows for it.  A continued chunk of few
    rows is not worth that and goes in tiles of ``ATTN_TILE`` rows that read the cache.

    Under a sliding ``window`` a piece is a run of at most ``WINDOW_PIECE`` rows together with the
    keys its first row sees before it; an entry that continues a sequence gathers its own keys and
    those of the window before it.  The first ``keep`` positions that the window has passed are a run of
    keys of their own.  Without ``tiles``, what is no piece goes row by row."""

    chunk: Optional[int]
    pieces: bool              # whether the layer's sizes allow the piece kernel
    window: Optional[int] = None
    tiles: bool = True
    keep: int = 0


SCAN_MIN = 16         # entries of more tokens than this take the chunked recurrence
SCAN_SEGMENT = 256    # and are cut into segments of at least this many
SCAN_BLOCKS = 2 * 148


@dataclass(frozen=True)
class ScanPlan:
    """How the entries of a batch go through a recurrence of ``blocks`` independent parts per entry
    (heads): short ones token by token, long ones 64 tokens at a time, cut into segments where
    there are fewer parts than the GPU has room for."""

    blocks: int
    chunks: bool              # whether the layer's sizes allow the chunked kernel


def _segments(plan: ScanPlan, long: List[int], lens: List[int]):
    """``([(entry, offset, tokens, 0)], [(entry, first segment, segments, 0)])``."""
    want = SCAN_BLOCKS // max(1, plan.blocks * len(long))
    segs, runs = [], []
    for i in long:
        n = max(1, min(want, lens[i] // SCAN_SEGMENT))
        size = -(-lens[i] // (64 * n)) * 64
        cut = [(i, o, min(size, lens[i] - o), 0) for o in range(0, lens[i], size)]
        runs.append((i, len(segs), len(cut), 0))
        segs += cut
    return segs, runs


def head_prep(raw: torch.Tensor, koff: int, voff: int, heads: int, kv_heads: int, dim: int, vdim: int,
              batch: "RaggedBatch", rope: Optional[torch.Tensor], k_cache: torch.Tensor,
              v_cache: torch.Tensor, page_table: torch.Tensor, *, interleaved: bool = False,
              unit_eps: Optional[float] = None, q_head: Optional[int] = None,
              k_rows: Optional[torch.Tensor] = None, v_rows: Optional[torch.Tensor] = None,
              eps: float = 0.0, q_norm: Optional[torch.Tensor] = None, k_norm: Optional[torch.Tensor] = None,
              unit_v: bool = False, q_factor: Optional[torch.Tensor] = None) -> torch.Tensor:
    """What stands between the projections ``raw`` (queries at column 0, keys at ``koff``, values at
    ``voff``) and the scores: rotation of the first ``2 * rope.shape[1]`` entries of the q and k heads (pairs
    half a rotation apart, or with ``interleaved`` neighbours), division of q and k by their root mean
    square over ``dim`` (``unit_eps`` inside the root; None: not), the write of k and v into the cache pages
    (and row by row into the first rows of ``k_rows [.., kv_heads, P]`` and ``v_rows``, zeros behind a
    head).  Returns ``q [rows, heads, q_head]``, zeros behind ``dim``.  ``heads`` and ``kv_heads`` count the
    heads of q and k; v has ``v_cache.shape[2]``.  ``kv_heads`` 0: queries alone, the cache is left alone.

    With ``q_norm [heads * dim]`` (and ``k_norm``) q and k are RMS-normed over all heads at once in front of
    the rotation; ``unit_v`` divides each head of v by its root mean square (both with ``eps``); ``q_factor
    [heads]`` multiplies the queries of a head at the end."""
    T, v_heads = raw.shape[0], v_cache.shape[2] if kv_heads else 0
    half = rope.shape[1] if rope is not None else 0
    Q = q_head or (dim + 7) // 8 * 8
    q = torch.empty((T, heads, Q), dtype=raw.dtype, device=raw.device)
    if not raw.is_cuda:
        def rotated(x):
            if half:
                c, s = rope[:, None, :, 0], rope[:, None, :, 1]
                a, b = (x[..., 0:2 * half:2], x[..., 1:2 * half:2]) if interleaved else \
                    (x[..., :half], x[..., half:2 * half])
                y = (a * c - b * s, b * c + a * s)
                y = torch.stack(y, -1).flatten(-2) if interleaved else torch.cat(y, -1)
                x = torch.cat([y, x[..., 2 * half:]], -1)
            if unit_eps is not None:
                x = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + unit_eps)
            return x
        def unit(x):
            return x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps)

        def heads_of(at, n, gain):
            x = raw[:, at:at + n * dim].float()
            x = x if gain is None else unit(x) * gain
            return rotated(x.view(T, n, dim))
        q.zero_()
        x = heads_of(0, heads, q_norm)
        q[..., :dim] = (x if q_factor is None else x * q_factor[:, None]).to(q.dtype)
        if kv_heads:
            page, at = _cells(page_table, batch)
            k_cache[page, at, :, :dim] = heads_of(koff, kv_heads, k_norm).to(k_cache.dtype)
            v = raw[:, voff:voff + v_heads * vdim].float().view(T, v_heads, vdim)
            v_cache[page, at, :, :vdim] = (unit(v) if unit_v else v).to(v_cache.dtype)
        return q
    rc = _lib.serving_lib().cb_head_prep(
        _p(raw), raw.stride(0), koff, voff, heads, kv_heads, v_heads, dim, vdim, half, _p(rope),
        int(interleaved), int(unit_eps is not None), _F(eps if unit_eps is None else unit_eps), _p(q_norm),
        _p(k_norm), int(unit_v), _p(q_factor), _p(q), Q, _p(k_cache),
        _p(v_cache), k_cache.shape[-1], v_cache.shape[-1], _p(k_rows), _p(v_rows),
        k_rows.shape[2] if k_rows is not None else 0, v_rows.shape[2] if v_rows is not None else 0,
        _p(page_table), page_table.shape[1], k_cache.shape[0], _p(batch.row_slot), _p(batch.pos), T,
        int(raw.dtype == torch.float32), _p(_lib.status_buffer(raw.device)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_head_prep")
    return q


def pieces_allowed(dim: int, vdim: int, chunk: Optional[int], scale: float) -> bool:
    return max(dim, vdim) <= 128 and scale > 0 and (chunk is None or chunk >= MIN_PIECE)


def row_head(dim: int, vdim: int) -> int:
    """Distance of the heads in the row-wise q, k and v of the piece kernel."""
    return 64 if max(dim, vdim) <= 64 else 128


def row_heads(dim: int, vdim: int, maps: int) -> Tuple[int, int]:
    """Distance of the heads in q and k, and in v, of the piece kernel without a convolution: with one
    map they are the same."""
    p = row_head(dim, vdim)
    return (p, p) if maps == 1 else (row_head(dim, 0), p)


def _cut(plan: AttnPlan, pos0: int, n: int):
    """``(rows that continue a chunk, positions of that chunk before them, [(offset, rows), ...])``
    of an entry of ``n`` tokens."""
    if plan.chunk is None:
        return (n, pos0, []) if pos0 else (0, 0, [(0, n)])
    head = min(n, -pos0 % plan.chunk)
    return head, pos0 % plan.chunk, [(o, min(plan.chunk, n - o))
                                     for o in range(head, n, plan.chunk)]


class RaggedBatch:
    """Index arrays of one step, in one int32 buffer (one host-to-device copy).  ``tile_rows``
    says whether long entries may take the tensor-core attention kernels (bf16 models on CUDA);
    otherwise every row is listed for the row kernel.  ``plans`` are the attention and
    recurrence plans the model's layers will ask for."""

    def __init__(self, entries: List[Entry], device, tile_rows: bool = True,
                 into: Optional["RaggedBatch"] = None,
                 plans: Sequence = (AttnPlan(None, False),)) -> None:
        n = len(entries)
        lens = [len(e.tokens) for e in entries]
        if not n or min(lens) < 1:
            raise ValueError("a step needs entries of at least one token")
        self.n, self.T, self.lens = n, sum(lens), lens
        self.kept: dict = {}         # what a layer leaves for later layers of the same step
        self.pos0_host = [e.pos0 for e in entries]
        self.slots_host = [e.slot for e in entries]
        self.max_ctx = max(e.pos0 + m for e, m in zip(entries, lens))
        row0 = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
        tokens = np.concatenate([np.asarray(e.tokens, dtype=np.int32) for e in entries])
        pos = np.concatenate([np.arange(e.pos0, e.pos0 + m, dtype=np.int32)
                              for e, m in zip(entries, lens)])
        row_slot = np.repeat(np.asarray([e.slot for e in entries], dtype=np.int32), lens)
        ct = [(i, o) for i, m in enumerate(lens) for o in range(0, m, CONV_TILE)]
        big = [i for i, m in enumerate(lens) if tile_rows and m > ROWS_MAX]
        small = [i for i in range(n) if i not in set(big)]
        rows = np.concatenate([np.arange(row0[i], row0[i + 1], dtype=np.int32) for i in small]) \
            if small else np.zeros(0, np.int32)
        want = np.asarray([row0[i] + k for i, e in enumerate(entries) for k in e.want],
                          dtype=np.int32)
        parts = [pos, np.asarray(self.pos0_host, np.int32), tokens, row_slot,
                 np.asarray(self.slots_host, np.int32), row0[:n], np.asarray(lens, np.int32),
                 np.asarray([c[0] for c in ct], np.int32), np.asarray([c[1] for c in ct], np.int32),
                 rows, want, np.arange(self.T, dtype=np.int32)]
        self.plans, cols = {}, len(parts)
        def align():                                               # read four at a time
            parts.append(np.zeros(-sum(len(x) for x in parts) % 4, np.int32))
        for plan in dict.fromkeys(plans):
            if isinstance(plan, ScanPlan):
                long = [i for i, m in enumerate(lens) if tile_rows and plan.chunks and m > SCAN_MIN]
                segs, runs = _segments(plan, long, lens)
                align()
                self.plans[plan] = (n - len(long), len(segs), len(runs), len(parts))
                parts += [np.asarray(segs, np.int32).reshape(-1), np.asarray(runs, np.int32).reshape(-1),
                          np.asarray([i for i in range(n) if i not in set(long)], np.int32)]
                continue
            tiles, pieces, where = [], [], []
            extra = 0
            for i in big:
                p0, r0 = entries[i].pos0, int(row0[i])
                if plan.window is not None:
                    if not plan.pieces:
                        if plan.tiles:
                            tiles += [(i, o, min(ATTN_TILE, lens[i] - o)) for o in range(0, lens[i], ATTN_TILE)]
                        continue
                    ahead = min(p0, plan.window - 1)
                    first = r0                             # key row of the entry's first token
                    kept = min(plan.keep, p0 + lens[i])    # positions 0 .. kept - 1 from this key row on
                    kept0 = r0
                    if p0:
                        keys = np.arange(p0 - ahead, p0 + lens[i], dtype=np.int32)
                        if p0 > ahead:
                            keys = np.concatenate([np.arange(min(kept, p0 - ahead), dtype=np.int32), keys])
                        where.append(np.stack([np.full_like(keys, entries[i].slot), keys], 1))
                        kept0 = self.T + extra
                        extra += len(keys)
                        first = self.T + extra - lens[i]
                    for o in range(0, lens[i], WINDOW_PIECE):
                        before = min(ahead + o, plan.window - 1)
                        size, unseen = min(WINDOW_PIECE, lens[i] - o), p0 + o - before
                        pieces.append((r0 + o, size, first + o - before, before, kept0,
                                       kept if unseen + before + size > plan.window else 0, unseen, 0))
                    continue
                head, ahead, ps = _cut(plan, p0, lens[i]) if plan.pieces else (lens[i], 0, [])
                if plan.pieces and head > MIN_PIECE:
                    keys = np.arange(p0 - ahead, p0 + head, dtype=np.int32)
                    where.append(np.stack([np.full_like(keys, entries[i].slot), keys], 1))
                    pieces.append((r0, head, self.T + extra, ahead, 0, 0, 0, 0))
                    extra += len(keys)
                elif plan.tiles:
                    tiles += [(i, o, min(ATTN_TILE, head - o)) for o in range(0, head, ATTN_TILE)]
                pieces += [(r0 + o, m, r0 + o, 0, 0, 0, 0, 0) for o, m in ps]
            tiles.sort(key=lambda t: -(entries[t[0]].pos0 + t[1]))     # the most keys first
            pieces.sort(key=lambda t: -t[1] * (t[1] + 2 * t[3]))
            if pieces:
                align()
            self.plans[plan] = (len(tiles), len(pieces), max([t[1] for t in pieces], default=0),
                                extra, len(parts))
            parts += [np.asarray(pieces, np.int32).reshape(-1),
                      np.concatenate(where).reshape(-1) if where else np.zeros(0, np.int32),
                      *np.asarray(tiles, np.int32).reshape(-1, 3).T]
        host = torch.from_numpy(np.concatenate(parts).astype(np.int32, copy=False))
        if into is None:
            self.buf = host.to(device)
        else:
            if into.buf.numel() != host.numel():
                raise ValueError("the batch does not fit the captured one")
            self.buf = into.buf
            self.buf.copy_(host)
        views, o = [], 0
        for part in parts:
            views.append(self.buf[o:o + len(part)])
            o += len(part)
        (self.pos, self.pos0, self.tokens, self.row_slot, self.slot, self.row0, self.len,
         self.conv_entry, self.conv_off, self.rows, self.want, self.every_row) = views[:cols]
        self._views = views
        self.positions = self.buf[:self.T + n]       # pos and pos0: what a decode step advances
        self.n_conv, self.n_rows, self.n_want = len(ct), len(rows), len(want)
        self.n_big = len(big)

    def plan(self, plan: AttnPlan):
        """``(tiles, pieces, longest piece, gathered rows, piece array, (slot, position) of the
        gathered rows, tile entries, offsets, lengths)``."""
        n_tiles, n_pieces, longest, extra, at = self.plans[plan]
        return (n_tiles, n_pieces, longest, extra, *self._views[at:at + 5])

    def scan(self, plan: ScanPlan):
        """``(short entries, segments, entries in segments, segment array, run array, short array)``."""
        n_short, n_segs, n_runs, at = self.plans[plan]
        return (n_short, n_segs, n_runs, *self._views[at:at + 3])

    def kv_rows(self, plan: AttnPlan) -> int:
        """Rows of the ``k_rows`` / ``v_rows`` buffers under ``plan``: this step's, then gathered
        ones (0: no piece, no buffers)."""
        _, n_pieces, _, extra, _ = self.plans[plan]
        return self.T + extra if n_pieces else 0

    def entry_args(self):
        return _p(self.slot), _p(self.row0), _p(self.len), _p(self.pos0)


def embed_norm(tokens: torch.Tensor, embed: torch.Tensor, weight: Optional[torch.Tensor],
               width: int, eps: float, out: torch.Tensor, scale: float = 1.0) -> torch.Tensor:
    """Rows of ``embed`` (RMS-normalised with ``weight`` when given) times ``scale`` as the fp32 residual
    stream; columns ``width ..`` of ``out`` are zero."""
    if not out.is_cuda:
        x = embed[tokens.long(), :width].float()
        if weight is not None:
            x = x * torch.rsqrt((x * x).mean(-1, keepdim=True) + eps) * weight[:width]
        out.zero_()
        out[:, :width] = x * scale
        return out
    rc = _lib.serving_lib().cb_embed_norm(
        _p(tokens), _p(embed), embed.stride(0), embed.shape[0], _p(weight), _p(out), out.stride(0),
        out.shape[0], width, _F(eps), _F(scale), int(embed.dtype == torch.float32),
        _p(_lib.status_buffer(out.device)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_embed_norm")
    return out


def rms_rows(x: torch.Tensor, w1: torch.Tensor, width: int, eps: float, dtype: torch.dtype,
             w2: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None
             ) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """RMS norm of the fp32 stream (of its ``rows`` only, when given) in the activation type,
    with one weight or, in the same pass, with two."""
    n = x.shape[0] if rows is None else rows.shape[0]
    if not x.is_cuda:
        v = x if rows is None else x[rows.long()]
        r = v * torch.rsqrt((v[:, :width] ** 2).mean(-1, keepdim=True) + eps)
        return (r * w1).to(dtype), None if w2 is None else (r * w2).to(dtype)
    y1 = torch.empty((n, x.shape[1]), dtype=dtype, device=x.device)
    y2 = torch.empty_like(y1) if w2 is not None else None
    rc = _lib.serving_lib().cb_rms_rows(
        _p(x), x.stride(0), _p(rows), _p(w1), _p(y1), _p(w2), _p(y2), y1.stride(0), n, width,
        _F(eps), int(dtype == torch.float32), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_rms_rows")
    return y1, y2


@dataclass
class Spread:
    """A sublayer's result in pieces: row ``t`` is the sum over ``k`` of ``weight[t, k] * rows[slot[t, k]]``
    (``slot`` int32 and ``weight`` fp32 ``[tokens, top]``, ``rows`` in the activation type); where the slot is
    negative, row ``t`` of ``own`` stands for it."""

    rows: torch.Tensor
    slot: torch.Tensor
    weight: torch.Tensor
    own: Optional[torch.Tensor] = None

    def sum(self) -> torch.Tensor:
        v = 0
        for k in range(self.weight.shape[1]):
            r = self.rows[self.slot[:, k].clamp_min(0).long()].float()
            if self.own is not None:
                r = torch.where(self.slot[:, k, None] < 0, self.own.float(), r)
            v = v + r * self.weight[:, k, None]
        return v


def add_norm(x: Optional[torch.Tensor], width: int, eps: float, dtype: torch.dtype, *,
             y: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None,
             post: Optional[torch.Tensor] = None, gain: Optional[torch.Tensor] = None,
             shift: Optional[torch.Tensor] = None, before: Optional[torch.Tensor] = None,
             batch: Optional["RaggedBatch"] = None, rows: Optional[torch.Tensor] = None,
             keep: bool = True, casts: Sequence[torch.Tensor] = (),
             spread: Optional["Spread"] = None, y_weight: Optional[torch.Tensor] = None,
             scale: Optional[torch.Tensor] = None, center: Optional[torch.Tensor] = None,
             taps: Optional[torch.Tensor] = None
             ) -> Tuple[Optional[torch.Tensor], Optional[torch.Tensor]]:
    """One pass between two sublayers, ``(x', h)``: ``v = y + bias`` (plus the weighted rows of ``spread``,
    which may also stand alone), RMS-normed with gain ``post`` when
    given; ``x' = x + v`` in fp32 (``v`` alone without ``x``, ``x`` itself without ``y``); ``h`` the RMS
    norm of ``x'`` with ``gain`` in the activation type, shifted by ``h + (h_before - h) * shift`` with
    the previous token's h (``before [slots, ld]`` at an entry's start, which is advanced).  Gains are
    one number or a vector.  ``y_weight [rows]`` multiplies a row of y before anything is added to it,
    ``scale`` (a vector) multiplies v; with ``center`` the norm of ``x'`` is a layer norm and this vector is
    added to it.  With ``taps [n, ld]`` h becomes ``h + conv(h)``, the causal convolution over time of every
    channel (the last tap for the token itself), whose earlier inputs at an entry's start are ``before
    [slots, n - 1, ld]`` (advanced too).  ``rows`` restricts the pass to some rows (``x'`` is not returned then),
    ``keep=False`` drops ``x'``; ``casts`` are up to two views that get ``x'`` in the activation type."""
    src = x if x is not None else y
    added = y is not None or spread is not None
    ld, n = src.shape[1], src.shape[0] if rows is None else rows.shape[0]
    if rows is not None:
        keep = False
    if not src.is_cuda:
        pick = (lambda t: t) if rows is None else (lambda t: t[rows.long()])

        def norm(v, g, c=None):
            if c is not None:
                v = v - v[:, :width].mean(-1, keepdim=True)
            v = v * torch.rsqrt((v[:, :width] ** 2).mean(-1, keepdim=True) + eps) * g
            return v if c is None else v + c
        out = None if x is None else pick(x)
        if added:
            v = pick(y).float() if y is not None else torch.zeros_like(out)
            v = v if y_weight is None else v * pick(y_weight)[:, None]
            v = v if spread is None else v + pick(spread.sum())
            v = v if bias is None else v + bias
            v = v if post is None else norm(v, post)
            v = v if scale is None else v * scale
            out = v if out is None else out + v
        for c in casts:
            c.copy_(out.to(c.dtype))
        h = None
        if gain is not None:
            h = norm(out, gain, center)
            if taps is not None:
                h = h + _conv_ref(h, taps, before, batch)
            if shift is not None:
                prev, r = torch.zeros_like(h), 0
                prev[1:] = h[:-1]
                for i, m in enumerate(batch.lens):
                    s = batch.slots_host[i]
                    prev[r] = before[s] if int(batch.pos0[i]) > 0 else 0.0
                    before[s] = h[r + m - 1]
                    r += m
                h = h + (prev - h) * shift
            h = h.to(dtype)
        return (out if keep else None), h
    x_out = torch.empty((n, ld), dtype=torch.float32, device=src.device) \
        if keep and (added or x is None) else None
    h = torch.empty((n, ld), dtype=dtype, device=src.device) if gain is not None else None
    shifted = shift is not None or taps is not None
    none = (None,) * 6
    tiles = shifted and not (taps is not None and batch.T == batch.n)      # else every entry is one token
    ents = none if not shifted else (*batch.entry_args(), *((_p(batch.conv_entry), _p(batch.conv_off)) if tiles
                                                            else (None, None)))
    stats = torch.empty((n, 2), dtype=torch.float32, device=src.device) if tiles and taps is not None else None
    cast = list(casts) + [None] * (2 - len(casts))
    sp = (None, 0, None, None, 0, None, 0) if spread is None else (
        _p(spread.rows), spread.rows.stride(0), _p(spread.slot), _p(spread.weight), spread.slot.shape[1],
        _p(spread.own), spread.own.stride(0) if spread.own is not None else 0)
    rc = _lib.serving_lib().cb_add_norm(
        _p(x), _p(y), _p(bias), _p(post), int(post is not None and post.numel() > 1), _p(x_out), ld,
        y.stride(0) if y is not None else 0, _p(gain), int(gain is not None and gain.numel() > 1), _p(h),
        ld, _p(cast[0]), _p(cast[1]), casts[0].stride(0) if casts else 0, _p(shift), _p(before),
        _p(rows), *ents, batch.n_conv if tiles else n, width, _F(eps), int(dtype == torch.float32),
        int(y is not None and y.dtype == torch.float32), *sp, _p(y_weight), _p(scale), _p(center), _p(taps),
        taps.shape[0] if taps is not None else 0, _p(stats), n, _lib.stream_ptr())
    _lib.check_rc(rc, "cb_add_norm", launches=1 if stats is None else 2)
    return (x_out if x_out is not None else (x if keep else None)), h


def rope_table(pos: torch.Tensor, inv_freq: torch.Tensor) -> torch.Tensor:
    """``[rows, half, 2]`` fp32 (cos, sin) of ``pos * inv_freq``."""
    n, half = pos.shape[0], inv_freq.shape[0]
    if not pos.is_cuda:
        a = pos.float()[:, None] * inv_freq[None]
        return torch.stack([a.cos(), a.sin()], -1)
    out = torch.empty((n, half, 2), dtype=torch.float32, device=pos.device)
    rc = _lib.serving_lib().cb_rope_table(_p(pos), _p(inv_freq), n, half, _p(out),
                                          _lib.stream_ptr())
    _lib.check_rc(rc, "cb_rope_table")
    return out


def _conv_ref(raw: torch.Tensor, taps_w: torch.Tensor, state: torch.Tensor, batch: RaggedBatch
              ) -> torch.Tensor:
    """Convolution of ``raw [rows, C]`` entry by entry; advances ``state [slots, taps-1, C]``."""
    n1 = taps_w.shape[0] - 1
    out = torch.empty(raw.shape, dtype=torch.float32)
    r = 0
    for i, m in enumerate(batch.lens):
        s = batch.slots_host[i]
        prev = state[s].float() if int(batch.pos0[i]) > 0 else torch.zeros(n1, raw.shape[1])
        u = torch.cat([prev, raw[r:r + m].float()])
        out[r:r + m] = sum(u[j:j + m] * taps_w[j] for j in range(n1 + 1))
        if n1:
            state[s] = u[-n1:].to(state.dtype)
        r += m
    return out


def _cells(page_table: torch.Tensor, batch: RaggedBatch):
    pos, slot = batch.pos.long(), batch.row_slot.long()
    return page_table[slot, pos // PAGE].long(), pos % PAGE


def shortconv_attn(raw: torch.Tensor, koff: int, voff: int, taps_w: torch.Tensor,
                   state: torch.Tensor, heads: int, kv_heads: int, dim: int, vdim: int,
                   batch: RaggedBatch, rope: Optional[torch.Tensor], k_cache: torch.Tensor,
                   v_cache: torch.Tensor, page_table: torch.Tensor,
                   v_first: Optional[torch.Tensor] = None, mix: Optional[torch.Tensor] = None,
                   write_first: bool = False, k_rows: Optional[torch.Tensor] = None,
                   v_rows: Optional[torch.Tensor] = None, q: Optional[torch.Tensor] = None
                   ) -> torch.Tensor:
    """What stands between the projections and the scores of an attention layer: a causal
    convolution over time on every channel of q, k and v (``taps_w [taps, channels]``), rotary
    embedding of the first ``2 * rope.shape[1]`` entries of the q and k heads in the rotate-half
    layout, value mixing ``v <- (1 - mix) v + mix v_first`` (or, with ``write_first``, keeping v as
    ``v_first``), and the write of k and v into the cache pages (and, when given, row by row into
    the first rows of ``k_rows [.., kv_heads, P]`` and ``v_rows``).  Returns ``q [rows, heads, dim]``, or
    fills the ``q [rows, heads, Q >= dim]`` it is given; padding is left alone."""
    T = raw.shape[0]
    half = rope.shape[1] if rope is not None else 0
    mode = 1 if write_first else (2 if mix is not None else 0)
    qc, kc, vc = heads * dim, kv_heads * dim, kv_heads * vdim
    if not raw.is_cuda:
        u = torch.cat([raw[:, :qc], raw[:, koff:koff + kc], raw[:, voff:voff + vc]], 1)
        y = _conv_ref(u, taps_w, state, batch)
        q, k = y[:, :qc].view(T, heads, dim), y[:, qc:qc + kc].view(T, kv_heads, dim)
        v = y[:, qc + kc:].view(T, kv_heads, vdim)
        if half:
            c, s = rope[:, None, :, 0], rope[:, None, :, 1]

            def rot(x):
                a, b = x[..., :half], x[..., half:2 * half]
                return torch.cat([a * c - b * s, b * c + a * s, x[..., 2 * half:]], -1)
            q, k = rot(q), rot(k)
        if mode == 1:
            v_first.copy_(v.reshape(T, -1))
        elif mode == 2:
            v = (1 - mix) * v + mix * v_first.float().view(T, kv_heads, vdim)
        page, at = _cells(page_table, batch)
        k_cache[page, at, :, :dim] = k.to(k_cache.dtype)
        v_cache[page, at, :, :vdim] = v.to(v_cache.dtype)
        return q.to(raw.dtype)
    if q is None:
        q = torch.empty((T, heads, dim), dtype=raw.dtype, device=raw.device)
    rc = _lib.serving_lib().cb_shortconv_attn(
        _p(raw), raw.stride(0), koff, voff, _p(taps_w), taps_w.shape[0], _p(state), heads, kv_heads,
        dim, vdim, *batch.entry_args(), _p(batch.conv_entry), _p(batch.conv_off), batch.n_conv, half,
        _p(rope), _p(q), q.shape[2], _p(k_cache), _p(v_cache), k_cache.shape[-1], v_cache.shape[-1],
        _p(page_table), page_table.shape[1], k_cache.shape[0], _p(v_first), _p(mix), mode,
        _p(k_rows), _p(v_rows), k_rows.shape[2] if k_rows is not None else dim, int(raw.dtype == torch.float32), _p(_lib.status_buffer(raw.device)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_shortconv_attn")
    return q


def shortconv_delta(raw: torch.Tensor, koff: int, voff: int, boff: int, taps_w: torch.Tensor,
                    state: torch.Tensor, heads: int, kv_heads: int, dim: int, vdim: int,
                    batch: RaggedBatch, a: torch.Tensor, A_log: torch.Tensor,
                    dt_bias: torch.Tensor):
    """Inputs of the gated delta recurrence, fp32: convolution and SiLU of q, k and v, unit norm of
    q and k (q also times ``dim ** -0.5``), the decay ``exp(-exp(A_log) softplus(a + dt_bias))`` of
    every key channel, the step size ``sigmoid(raw[:, boff + h])``.  Returns
    ``(q [kv_heads, rows, P], k, kq [kv_heads, rows], v [rows, heads, vdim], g [heads, rows, P],
    beta [heads, rows])``, the channels of q, k and g padded with zeros to a multiple of 32."""
    T = raw.shape[0]
    P = (dim + 31) // 32 * 32
    qc, vc = kv_heads * dim, heads * vdim
    f32 = dict(dtype=torch.float32, device=raw.device)
    alloc = torch.zeros if not raw.is_cuda else torch.empty
    q, k = alloc((kv_heads, T, P), **f32), alloc((kv_heads, T, P), **f32)
    kq, v = alloc((kv_heads, T), **f32), alloc((T, heads, vdim), **f32)
    g, beta = alloc((heads, T, P), **f32), alloc((heads, T), **f32)
    if not raw.is_cuda:
        u = torch.cat([raw[:, :qc], raw[:, koff:koff + qc], raw[:, voff:voff + vc]], 1)
        y = torch.nn.functional.silu(_conv_ref(u, taps_w, state, batch))

        def unit(x):
            return x * torch.rsqrt((x * x).sum(-1, keepdim=True) + 1e-6)
        q[..., :dim] = (unit(y[:, :qc].view(T, kv_heads, dim)) * dim ** -0.5).transpose(0, 1)
        k[..., :dim] = unit(y[:, qc:2 * qc].view(T, kv_heads, dim)).transpose(0, 1)
        kq.copy_((q * k).sum(-1))
        v.copy_(y[:, 2 * qc:].view(T, heads, vdim))
        z = torch.nn.functional.softplus(a[:, :heads * dim].float() + dt_bias, threshold=100.0)
        g[..., :dim] = torch.exp(-torch.exp(A_log)[:, None, None]
                                 * z.view(T, heads, dim).transpose(0, 1))
        beta.copy_(torch.sigmoid(raw[:, boff:boff + heads].float()).t())
        return q, k, kq, v, g, beta
    rc = _lib.serving_lib().cb_shortconv_delta(
        _p(raw), raw.stride(0), koff, voff, boff, _p(taps_w), taps_w.shape[0], _p(state), heads,
        kv_heads, dim, vdim, *batch.entry_args(), _p(batch.conv_entry), _p(batch.conv_off),
        batch.n_conv, _p(a), a.stride(0), _p(A_log), _p(dt_bias), _p(q), _p(k), _p(kq), _p(v), _p(g),
        _p(beta), T, P, int(raw.dtype == torch.float32), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_shortconv_delta")
    return q, k, kq, v, g, beta


def delta_scan(q: torch.Tensor, k: torch.Tensor, kq: torch.Tensor, v: torch.Tensor,
               g: torch.Tensor, beta: torch.Tensor, state: torch.Tensor, batch: RaggedBatch
               ) -> torch.Tensor:
    """The gated delta rule over every entry, from and into ``state [slots, heads, dim, vdim]``
    (fp32).  Returns the read-outs ``[rows, heads, vdim]``, fp32."""
    T, heads, vdim = v.shape
    kv_heads, dim, P = q.shape[0], state.shape[2], q.shape[2]
    o = torch.empty_like(v)
    if not v.is_cuda:
        per, r = heads // kv_heads, 0
        for i, m in enumerate(batch.lens):
            s = batch.slots_host[i]
            S = state[s].clone() if int(batch.pos0[i]) > 0 else torch.zeros_like(state[s])
            for t in range(r, r + m):
                kk, qq = (x[:, t, :dim].repeat_interleave(per, 0) for x in (k, q))
                S = S * g[:, t, :dim, None]
                w = beta[:, t, None] * (v[t] - torch.einsum("hdv,hd->hv", S, kk))
                S = S + kk[:, :, None] * w[:, None, :]
                o[t] = torch.einsum("hdv,hd->hv", S, qq)
            state[s] = S
            r += m
        return o
    rc = _lib.serving_lib().cb_delta_scan(
        _p(q), _p(k), _p(kq), _p(v), _p(g), _p(beta), _p(state), _p(o), T, heads, kv_heads, dim,
        P, vdim, *batch.entry_args(), batch.n, _lib.stream_ptr())
    _lib.check_rc(rc, "cb_delta_scan")
    return o


def gated_head_norm(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, eps: float,
                    out: torch.Tensor) -> torch.Tensor:
    """``out = o / rms(o) * weight * sigmoid(gate)`` per head; ``o [rows, heads, vdim]`` fp32,
    ``gate`` and ``out`` ``[rows, heads * vdim]`` views."""
    T, heads, vdim = o.shape
    if not o.is_cuda:
        y = o * torch.rsqrt((o * o).mean(-1, keepdim=True) + eps) * weight
        y = y * torch.sigmoid(gate[:, :heads * vdim].float()).view(T, heads, vdim)
        return out.copy_(y.reshape(T, -1).to(out.dtype))
    rc = _lib.serving_lib().cb_gated_head_norm(
        _p(o), _p(gate), gate.stride(0), _p(weight), _p(out), out.stride(0), T, heads, vdim, _F(eps),
        int(out.dtype == torch.float32), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_gated_head_norm")
    return out


def ragged_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                     page_table: torch.Tensor, batch: RaggedBatch, heads: int, kv_heads: int,
                     dim: int, vdim: int, scale: float, out: torch.Tensor, *,
                     chunk: Optional[int] = None, window: Optional[int] = None, keep: int = 0,
                     softcap: Optional[float] = None, score_max: float = 0.0, maps: int = 1,
                     map_weight: Optional[torch.Tensor] = None, map_factor: float = 1.0,
                     eps: float = 0.0, sink: Optional[torch.Tensor] = None,
                     gate: Optional[torch.Tensor] = None, gate_wide: bool = False,
                     max_ctx: Optional[int] = None,
                     k_rows: Optional[torch.Tensor] = None,
                     v_rows: Optional[torch.Tensor] = None,
                     plan: Optional[AttnPlan] = None, gathered: bool = False) -> torch.Tensor:
    """Causal attention of every query row over the cached keys of its own sequence, restricted to
    the row's chunk (positions with the same ``pos // chunk``) when ``chunk`` is given, or to itself and
    the ``window - 1`` positions before it (and the sequence's first ``keep`` positions).  Scores ``s`` become ``softcap * tanh(s / softcap)``
    (``score_max`` bounds ``|s|``, 0 where no bound is known).  ``sink``
    (fp32 ``[heads]``) is a logit that enters the softmax denominator only; ``gate`` multiplies by its
    sigmoid: a view whose column ``h`` belongs to head ``h``, or (``gate_wide``) a view like ``out``.  Query
    head ``h`` reads key/value head ``h // (heads // kv_heads)``.  ``q`` is ``[rows, heads, Q >= dim]``,
    ``out`` a ``[rows, heads * vdim]``
    view; ``max_ctx`` bounds the keys of any row (it only chooses how many CTAs share a row).  With
    row-wise ``k_rows`` and ``v_rows`` at hand (:meth:`RaggedBatch.kv_rows` rows of ``[kv_heads, P]``,
    this step's filled in; q then has the keys' head distance), the pieces of ``plan`` go through
    the tcgen05 kernel; the default plan has pieces when the buffers are given (``gathered``: so are the
    cached rows behind this step's).

    With two ``maps`` a head has two queries and its key head two keys (``q [rows, heads * 2, Q]``,
    ``k_cache [pages, PAGE, kv_heads * 2, dim_p]``, map 0 first) over the same values; with their outputs
    ``a0`` and ``a1`` the head's output is ``a0 - map_weight * a1`` (``map_weight`` one fp32 number on the
    device) divided by its root mean square (``eps`` inside the root), times ``map_factor``."""
    T = q.shape[0]
    if not q.is_cuda:
        per = heads // kv_heads
        r = 0
        for i, m in enumerate(batch.lens):
            pos = batch.pos[r:r + m].long()
            n = int(pos[-1]) + 1
            pages = page_table[batch.slots_host[i], :(n + PAGE - 1) // PAGE].long()
            K = k_cache[pages].reshape(-1, kv_heads, maps, k_cache.shape[-1])[:n, ..., :dim].float()
            V = v_cache[pages].reshape(-1, kv_heads, v_cache.shape[-1])[:n, :, :vdim].float()
            K, V = K.repeat_interleave(per, 1).flatten(1, 2), V.repeat_interleave(per * maps, 1)
            s = torch.einsum("thd,nhd->htn", q[r:r + m, :, :dim].float(), K) * scale
            if softcap is not None:
                s = softcap * torch.tanh(s / softcap)
            j = torch.arange(n)
            lo = pos // chunk * chunk if chunk else torch.zeros_like(pos)
            lo = torch.clamp(pos + 1 - window, min=0) if window else lo
            ok = (j[None] <= pos[:, None]) & ((j[None] >= lo[:, None]) | (j[None] < keep))
            s = s.masked_fill(~ok, float("-inf"))
            top = s.amax(-1, keepdim=True)
            if sink is not None:
                top = torch.maximum(top, sink.view(-1, 1, 1))
            w = torch.exp(s - top)
            den = w.sum(-1, keepdim=True)
            if sink is not None:
                den = den + torch.exp(sink.view(-1, 1, 1) - top)
            o = torch.einsum("htn,nhd->thd", w / den, V)
            if maps == 2:
                o = o[:, 0::2] - map_weight * o[:, 1::2]
                o = o * torch.rsqrt((o * o).mean(-1, keepdim=True) + eps) * map_factor
            if gate is not None:
                g = torch.sigmoid(gate[r:r + m].float())
                o = o * (g[:, :heads * vdim].view(m, heads, vdim) if gate_wide else g[:, :heads, None])
            out[r:r + m] = o.reshape(m, -1).to(out.dtype)
            r += m
        return out
    st = _p(_lib.status_buffer(q.device))
    lib = _lib.serving_lib()
    spec = _AttnSpec(heads, kv_heads, dim, vdim, k_cache.shape[-1], v_cache.shape[-1], chunk or 0,
                     window or 0, keep, maps, int(gate_wide), scale, softcap or 0.0, map_factor, eps)
    common = (_p(q), q.shape[2], _p(k_cache), _p(v_cache), _p(page_table), page_table.shape[1],
              k_cache.shape[0], ctypes.byref(spec), _p(sink), _p(gate),
              gate.stride(0) if gate is not None else 0, _p(map_weight), _p(out), out.stride(0))
    n, rows = batch.n_rows, batch.rows
    if batch.n_big:
        n_tiles, n_pieces, longest, extra, pieces, where, t_entry, t_off, t_len = batch.plan(
            plan or AttnPlan(chunk, k_rows is not None, window, keep=keep))
        if not n_tiles and not n_pieces:       # sizes that neither kernel takes
            n, rows = T, batch.every_row
        if n_tiles:
            rc = lib.cb_ragged_attn_tiles(*common, *batch.entry_args(), _p(t_entry), _p(t_off),
                                          _p(t_len), n_tiles, st, _lib.stream_ptr())
            _lib.check_rc(rc, "cb_ragged_attn_tiles")
        if extra and not gathered:
            rc = lib.cb_kv_gather(_p(k_cache), _p(v_cache), kv_heads * maps, kv_heads, k_cache.shape[-1],
                                  v_cache.shape[-1], _p(page_table), page_table.shape[1],
                                  k_cache.shape[0], _p(where), extra, _p(k_rows[T:]), _p(v_rows[T:]),
                                  k_rows.shape[2], v_rows.shape[2], st, _lib.stream_ptr())
            _lib.check_rc(rc, "cb_kv_gather")
        if n_pieces:
            rc = lib.cb_attn_fwd_pieces(
                _p(q), _p(k_rows), _p(v_rows), _p(out), T, k_rows.shape[0], _p(pieces), n_pieces,
                longest, heads, kv_heads, k_rows.shape[2], v_rows.shape[2], vdim, q.stride(0),
                k_rows.stride(0), v_rows.stride(0), out.stride(0), _F(scale), _p(sink), _p(gate),
                gate.stride(0) if gate is not None else 0, int(gate_wide), window or 0, keep,
                _F(softcap or 0.0), _F(score_max), maps, _p(map_weight), _F(map_factor), _F(eps), st, _lib.stream_ptr())
            _lib.check_rc(rc, "cb_attn_fwd_pieces")
    if n:
        per = heads // kv_heads * maps
        ctas = n * kv_heads * ((per + 15) // 16)
        ctx = max_ctx or batch.max_ctx
        ctx = min([ctx] + [c + keep for c in (chunk, window) if c])
        # a CTA takes 128 keys at a time
        splits = max(1, min(16, (2 * 148 + ctas - 1) // ctas, (ctx + 127) // 128))
        part_o = part_ml = None
        if splits > 1 or maps > 1:
            part_o = torch.empty((n, heads * maps, splits, vdim), dtype=torch.float32, device=q.device)
            part_ml = torch.empty((n, heads * maps, splits, 2), dtype=torch.float32, device=q.device)
        rc = lib.cb_ragged_attn_rows(*common, _p(rows), _p(batch.row_slot), _p(batch.pos), n,
                                     splits, _p(part_o), _p(part_ml), int(q.dtype == torch.float32),
                                     st, _lib.stream_ptr())
        _lib.check_rc(rc, "cb_ragged_attn_rows", launches=2 if part_o is not None else 1)
    return out


class _AttnSpec(ctypes.Structure):
    """``RaggedSpec`` of ``csrc/ragged_attn.cu``."""

    _fields_ = [(n, ctypes.c_int) for n in ("heads", "kv_heads", "dim", "vdim", "dim_p", "vdim_p", "chunk",
                                            "window", "keep", "maps", "gate_wide")] + \
               [(n, ctypes.c_float) for n in ("scale", "softcap", "map_factor", "eps")]
