"""Mixture of experts of the serving step (``csrc/experts.cu``): routing by sigmoid or softmax scores among
the best groups, without a capacity (every chosen expert runs), experts with a gated unit, and identity
experts, whose result is their input.

Few rows stream the weights of the chosen experts (:func:`experts_few`).  Larger batches are sorted by
expert into a buffer whose experts start at multiples of a block of rows, and the experts' products are one
grouped launch each (:func:`route`, :func:`sort_rows`, :func:`grouped_linear`); the results leave through
:class:`coeus_b200.ops.ragged.Spread`.

CPU tensors take a PyTorch restatement of the same math; CUDA tensors always run the kernels.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import _lib
from .gemm import clamped_glu

BLOCKS = (128, 256)   # rows of one expert's tile: 256 where experts have many
FEW = 16              # rows up to which the experts' weights are streamed
ROUTE_FEW = 128       # rows up to which the router's product and the choice are one launch
ROUTE_TOKENS = 32     # tokens per block of the choice otherwise
_F = ctypes.c_float


def _p(t):
    return _lib.ptr(t)


@dataclass(frozen=True)
class Routing:
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    identity: int = 0         # experts ``experts ..`` that pass their input on
    softmax: bool = False     # scores: softmax over all of them, else sigmoids
    group_best: int = 2       # a group counts the sum of its one or two largest scores
    normalise: bool = True    # weights are divided by their sum
    shared_gate: bool = False   # the router's next output is the logit of the shared expert's gate

    @property
    def outputs(self) -> int:
        return self.experts + self.identity


@dataclass
class Choice:
    """``expert`` (int32) and ``weight`` (fp32) ``[tokens, top]``, ``shared`` (fp32 ``[tokens]``) the shared
    expert's weight where it has one; on the GPU also what sorting needs: the tokens of a block, the rank of
    a pair among its block's of the same expert, the blocks' counts."""

    expert: torch.Tensor
    weight: torch.Tensor
    shared: Optional[torch.Tensor] = None
    per_block: int = 0
    rank: Optional[torch.Tensor] = None
    counts: Optional[torch.Tensor] = None


def choose(z: torch.Tensor, r: Routing, correction: Optional[torch.Tensor] = None
           ) -> Tuple[torch.Tensor, torch.Tensor]:
    """The choice in PyTorch, from the router's logits ``z [tokens, outputs]``; ties go to the lower index.
    ``correction`` is added to the scores that are compared, not to the weights."""
    s = torch.softmax(z.float(), -1) if r.softmax else torch.sigmoid(z.float())
    rated = s if correction is None else s + correction
    T, n = s.shape[0], r.outputs // r.groups
    value = rated.view(T, r.groups, n).topk(min(r.group_best, n), -1).values.sum(-1)
    kept = torch.sort(value, dim=-1, descending=True, stable=True).indices[:, :r.keep]
    ok = torch.zeros(T, r.groups, dtype=torch.bool, device=z.device).scatter_(1, kept, True)
    masked = rated.masked_fill(~ok.repeat_interleave(n, 1), float("-inf"))
    expert = torch.sort(masked, dim=-1, descending=True, stable=True).indices[:, :r.top]
    w = s.gather(1, expert)
    return expert.to(torch.int32), (w / (w.sum(-1, keepdim=True) + 1e-20) if r.normalise else w) * r.scale


def route(h: torch.Tensor, router: torch.Tensor, r: Routing, correction: Optional[torch.Tensor] = None) -> Choice:
    """The experts of every row of ``h [tokens, W]`` by the logits ``h @ router^T`` (``router [outputs, and
    the shared expert's gate, rounded up to 8, W]``), which are fp32."""
    T, W = h.shape
    if not h.is_cuda:
        z = h.float() @ router.float().t()
        return Choice(*choose(z[:, :r.outputs], r, correction),
                      torch.sigmoid(z[:, r.outputs]) if r.shared_gate else None)
    from .gemm import linear
    few, dev = T <= ROUTE_FEW, h.device
    logits = None
    if not few:
        logits = linear(h, router, torch.empty((T, router.shape[0]), dtype=torch.float32, device=dev))
    per = 1 if few else ROUTE_TOKENS
    blocks = (T + per - 1) // per
    expert, rank = (torch.empty((T, r.top), dtype=torch.int32, device=dev) for _ in range(2))
    weight = torch.empty((T, r.top), dtype=torch.float32, device=dev)
    counts = torch.empty((r.outputs, blocks), dtype=torch.int32, device=dev)
    shared = torch.empty(T, dtype=torch.float32, device=dev) if r.shared_gate else None
    rc = _lib.serving_lib().cb_moe_choose(
        _p(logits), logits.stride(0) if logits is not None else 0, _p(h), h.stride(0), _p(router),
        router.stride(0), W, T, r.outputs, r.top, r.groups, r.keep, _F(r.scale), int(r.softmax), r.group_best,
        int(r.normalise), _p(correction), _p(shared), _p(expert), _p(weight),
        _p(rank), _p(counts), int(h.dtype == torch.float32), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_moe_choose")
    return Choice(expert, weight, shared, per, rank, counts)


@dataclass
class Sorted:
    """``rows [blocks * 128 or 256, W]``: every token's row once per expert it uses, sorted by expert;
    ``slot [tokens, top]`` says where (-1: nowhere, an identity expert); ``block_expert [blocks]`` is the expert
    of a block of rows, -1 behind the last one."""

    rows: torch.Tensor
    slot: torch.Tensor
    block_expert: torch.Tensor


def sort_rows(h: torch.Tensor, c: Choice, r: Routing) -> Sorted:
    T, W = h.shape
    pairs = T * r.top
    block = BLOCKS[1] if pairs >= 1024 * r.experts else BLOCKS[0]
    blocks = pairs // block + min(r.experts, pairs)
    dev = h.device
    rows = torch.empty((blocks * block, W), dtype=h.dtype, device=dev)
    if not h.is_cuda:
        rows.zero_()
        slot = torch.full((T, r.top), -1, dtype=torch.int32)
        block_expert, at = [], 0
        for e in range(r.experts):
            t, k = (c.expert == e).nonzero(as_tuple=True)
            if len(t):
                slot[t, k] = torch.arange(at, at + len(t), dtype=torch.int32)
                rows[at:at + len(t)] = h[t]
                n = (len(t) + block - 1) // block
                block_expert += [e] * n
                at += n * block
        block_expert += [-1] * (blocks - len(block_expert))
        return Sorted(rows, slot, torch.tensor(block_expert, dtype=torch.int32))
    slot = torch.empty((T, r.top), dtype=torch.int32, device=dev)
    block_expert = torch.empty(blocks, dtype=torch.int32, device=dev)
    base = torch.empty_like(c.counts)
    rc = _lib.serving_lib().cb_moe_sort(
        _p(h), h.stride(0), _p(c.expert), _p(c.rank), _p(c.counts), T, r.experts, r.top, c.per_block,
        c.counts.shape[1], _p(base), _p(slot), _p(block_expert), blocks, block, _p(rows), W,
        int(h.dtype == torch.float32), _p(_lib.status_buffer(dev)), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_moe_sort", launches=2)
    return Sorted(rows, slot, block_expert)


def grouped_linear(x: torch.Tensor, w: torch.Tensor, block_expert: torch.Tensor, out: torch.Tensor, *,
                   glu: Optional[Tuple[float, float, float]] = None) -> torch.Tensor:
    """``out[block] = x[block] @ w[block_expert[block]]^T`` for every block of rows (``w [experts, N, K]``, as
    many blocks as ``block_expert`` has entries, of 128 or 256 rows); blocks of no expert are left alone.  ``glu = (slope, limit, shift)``: see :func:`coeus_b200.ops.gemm.linear`."""
    E, N, K = w.shape
    M = x.shape[0]
    block = M // block_expert.shape[0]
    if x.shape[1] != K or block not in BLOCKS or M != block_expert.shape[0] * block or out.shape != (M, N // 2 if glu else N):
        raise ValueError(f"grouped_linear: shapes {tuple(x.shape)} {tuple(w.shape)} {tuple(out.shape)}")
    if not x.is_cuda:
        for b, e in enumerate(block_expert.tolist()):
            if e >= 0:
                s = slice(b * block, (b + 1) * block)
                z = x[s].float() @ w[e].float().t()
                out[s] = (clamped_glu(z, *glu) if glu else z).to(out.dtype)
        return out
    slope, limit, shift = glu or (0.0, 0.0, 0.0)
    lib, st = _lib.serving_lib(), _p(_lib.status_buffer(x.device))
    if x.dtype == torch.float32:
        rc = lib.cb_linear_f32_grouped(
            _p(x), x.stride(0), _p(w), w.stride(1), None, _p(block_expert), block, _p(out), out.stride(0), M, N, K,
            int(glu is not None), _F(slope), _F(limit), _F(shift), _lib.stream_ptr())
        _lib.check_rc(rc, "cb_linear_f32_grouped")
        return out
    rc = lib.cb_gemm_bf16_blocks(
        _p(x), _p(w), None, _p(out), M, N, K, E, x.stride(0), w.stride(1), out.stride(0), _p(block_expert), block,
        int(glu is not None), _F(slope), _F(limit), _F(shift), st, _lib.stream_ptr())
    _lib.check_rc(rc, "cb_gemm_bf16_blocks")
    return out


def experts_few(h: torch.Tensor, c: Choice, r: Routing, w_in: torch.Tensor, w_down: torch.Tensor,
                limit: float, s_in: Optional[torch.Tensor], s_down: Optional[torch.Tensor],
                s_limit: float, slope: float, shift: float = 1.0) -> torch.Tensor:
    """All experts of up to ``FEW`` bf16 rows and the shared one: fp32 ``[tokens, W]``."""
    T, W = h.shape
    n, ns = w_down.shape[2], s_down.shape[1] if s_down is not None else 0
    live = min(r.experts, T * r.top)
    act = torch.empty((T, live * n + ns), dtype=h.dtype, device=h.device)
    y = torch.empty((T, W), dtype=torch.float32, device=h.device)
    rc = _lib.serving_lib().cb_moe_few(
        _p(h), h.stride(0), T, W, r.experts, r.top, _p(c.expert), _p(c.weight), _p(c.shared),
        _p(w_in), _p(w_down), n, _F(limit), _p(s_in), _p(s_down), ns, _F(s_limit), _F(slope), _F(shift), _p(act), act.stride(0), _p(y),
        y.stride(0), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_moe_few", launches=2)
    return y
