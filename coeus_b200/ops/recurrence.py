"""Recurrences of the ragged serving step: the Mamba-2 state-space layer (``csrc/shortconv.cu``,
``ssd.cu``) and the minGRU (``mingru.cu``).  State is addressed by slot and lives in fp32.

CPU tensors take a PyTorch restatement of the same math; CUDA tensors always run the kernels.
"""
from __future__ import annotations

import ctypes

import torch
import torch.nn.functional as F

from . import _lib
from .ragged import RaggedBatch, ScanPlan, _conv_ref, _p

_F = ctypes.c_float


SCAN_COLS = 64       # columns of a head per block
CHUNK_STATE = 128    # largest state the chunked kernel takes


def ssd_plan(heads: int, vdim: int, N: int) -> ScanPlan:
    return ScanPlan(heads * ((vdim + SCAN_COLS - 1) // SCAN_COLS), N <= CHUNK_STATE)


def shortconv_act(raw: torch.Tensor, off: int, taps_w: torch.Tensor, bias: torch.Tensor,
                  state: torch.Tensor, batch: RaggedBatch) -> torch.Tensor:
    """Causal convolution over time with bias and SiLU of the channels ``raw[:, off:off + C]``
    (``taps_w [taps, C]``, ``C`` a multiple of eight), advancing ``state [slots, taps - 1, C]``."""
    T, C = raw.shape[0], taps_w.shape[1]
    if not raw.is_cuda:
        return F.silu(_conv_ref(raw[:, off:off + C], taps_w, state, batch) + bias).to(raw.dtype)
    out = torch.empty((T, C), dtype=raw.dtype, device=raw.device)
    rc = _lib.serving_lib().cb_shortconv_act(
        _p(raw), raw.stride(0), off, _p(taps_w), _p(bias), taps_w.shape[0], C, _p(state), _p(out),
        *batch.entry_args(), _p(batch.conv_entry), _p(batch.conv_off), batch.n_conv,
        int(raw.dtype == torch.float32), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_shortconv_act")
    return out


def ssd_scan(u: torch.Tensor, boff: int, coff: int, dt: torch.Tensor, dt_bias: torch.Tensor,
             A_log: torch.Tensor, D: torch.Tensor, state: torch.Tensor, groups: int, vdim: int,
             batch: RaggedBatch, y: torch.Tensor) -> torch.Tensor:
    """The state-space recurrence: ``u [rows, ..]`` holds ``x [heads, vdim]`` at column 0 and ``B``,
    ``C [groups, N]`` at ``boff``, ``coff``; ``dt`` is a view whose column ``h`` is head ``h``'s raw step
    size.  Per head ``S <- exp(-exp(A_log) dt) S + dt B x^T``, ``y = S^T C + D x`` with
    ``dt <- softplus(dt + dt_bias)``, from and into ``state [slots, heads, N, >= vdim]``."""
    heads, N = state.shape[1], state.shape[2]
    if not u.is_cuda:
        per, r = heads // groups, 0
        for i, m in enumerate(batch.lens):
            s = batch.slots_host[i]
            S = state[s, :, :, :vdim].clone() if int(batch.pos0[i]) > 0 else \
                torch.zeros_like(state[s, :, :, :vdim])
            for t in range(r, r + m):
                x = u[t, :heads * vdim].float().view(heads, vdim)
                B, C = (u[t, o:o + groups * N].float().view(groups, N).repeat_interleave(per, 0)
                        for o in (boff, coff))
                d = F.softplus(dt[t, :heads].float() + dt_bias, threshold=100.0)
                S = S * torch.exp(-torch.exp(A_log) * d)[:, None, None] \
                    + (d[:, None] * B)[:, :, None] * x[:, None, :]
                out = torch.einsum("hnp,hn->hp", S, C) + D[:, None] * x
                y[t, :heads * vdim] = out.reshape(-1).to(y.dtype)
            state[s, :, :, :vdim] = S
            r += m
        return y
    lib, f32 = _lib.serving_lib(), u.dtype == torch.float32
    common = (_p(u), u.stride(0), boff, coff, _p(dt), dt.stride(0), _p(dt_bias), _p(A_log), _p(D),
              _p(state), _p(y), y.stride(0), heads, groups, N, vdim, state.shape[3],
              *batch.entry_args())
    n_short, n_segs, n_runs, segs, runs, short = batch.scan(ssd_plan(heads, vdim, N))
    if n_short:
        rc = lib.cb_ssd_step(*common, _p(short), n_short, int(f32), _lib.stream_ptr())
        _lib.check_rc(rc, "cb_ssd_step")
    if n_segs:
        kept = decay = None
        if n_segs > n_runs:
            kept = torch.empty((n_segs, *state.shape[1:]), dtype=torch.float32, device=u.device)
            decay = torch.empty((n_segs, heads), dtype=torch.float32, device=u.device)
        rc = lib.cb_ssd_chunk(*common, _p(segs), n_segs, _p(runs), n_runs, _p(kept), _p(decay),
                              _lib.stream_ptr())
        _lib.check_rc(rc, "cb_ssd_chunk", launches=1 if kept is None else 3)
    return y


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, parts: int, eps: float,
                     out: torch.Tensor) -> torch.Tensor:
    """``y silu(z)`` in ``parts`` equal parts, each divided by its root mean square, times ``weight``;
    ``y``, ``z`` and ``out`` are ``[rows, inner]`` views."""
    T, inner = y.shape[0], weight.shape[0]
    if not y.is_cuda:
        v = (y[:, :inner].float() * F.silu(z[:, :inner].float())).view(T, parts, -1)
        v = v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps)
        return out.copy_((v.view(T, inner) * weight).to(out.dtype))
    rc = _lib.serving_lib().cb_gated_group_norm(
        _p(y), y.stride(0), _p(z), z.stride(0), _p(weight), _p(out), out.stride(0), T, inner, parts,
        _F(eps), int(y.dtype == torch.float32), _lib.stream_ptr())
    _lib.check_rc(rc, "cb_gated_group_norm")
    return out


def mingru_scan(raw: torch.Tensor, zoff: int, uoff: int, goff: int, state: torch.Tensor,
           batch: RaggedBatch, out: torch.Tensor) -> torch.Tensor:
    """``S <- (1 - z) S + z c`` element by element, ``z`` the sigmoid of the columns at ``zoff``, ``c =
    u + 1/2`` for the columns ``u >= 0`` at ``uoff`` and ``sigmoid(u)`` otherwise, from and into
    ``state [slots, width]``; ``out = S silu(g)``, ``g`` the columns at ``goff``."""
    W = state.shape[1]
    if not raw.is_cuda:
        r = 0
        for i, m in enumerate(batch.lens):
            s = batch.slots_host[i]
            S = state[s].clone() if int(batch.pos0[i]) > 0 else torch.zeros_like(state[s])
            for t in range(r, r + m):
                z = torch.sigmoid(raw[t, zoff:zoff + W].float())
                u, g = raw[t, uoff:uoff + W].float(), raw[t, goff:goff + W].float()
                S = (1 - z) * S + z * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
                out[t, :W] = (S * F.silu(g)).to(out.dtype)
            state[s] = S
            r += m
        return out
    rc = _lib.serving_lib().cb_mingru(
        _p(raw), raw.stride(0), zoff, uoff, goff, _p(state), _p(out), out.stride(0), W,
        *batch.entry_args(), batch.n, max(batch.lens), int(raw.dtype == torch.float32),
        _lib.stream_ptr())
    _lib.check_rc(rc, "cb_mingru")
    return out
