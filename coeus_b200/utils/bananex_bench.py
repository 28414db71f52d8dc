"""Sizes of the Bananex serving benchmark and its kernels one by one against the roofline (see
:mod:`coeus_b200.utils.serving_bench`).

As many runs of layers as the closest model has layers: latent attention, Mamba-2 and minGRU in turn,
the middle third of the stack a loop of two passes."""
from __future__ import annotations

from typing import Dict, List

import torch

from ..models import hybrid as H

DIM, ROT, VDIM, RANK, WINDOW = 96, 32, 128, 512, 1024
STATE, COLS = 128, 64        # Mamba-2: state per head, columns per head


def config(width: int, layers: int, heads: int, kv_heads: int) -> H.HybridConfig:
    from .serving_bench import VOCAB
    mixers = (H.LatentAttentionSpec(heads, DIM, ROT, VDIM, RANK, (DIM + ROT) ** -0.5, WINDOW, 1e6),
              H.Mamba2Spec(2 * width // COLS, COLS, STATE, 1, 4, 1), H.MinGruSpec(width))
    loop = H.LoopSpec(layers // 6, layers // 3, 3) if layers < 12 else H.LoopSpec(3, 6, 2)
    stored = layers - (loop.stop - loop.start) * (loop.times - 1)
    return H.HybridConfig(VOCAB, width, tuple(
        H.LayerSpec(mixers[i % 3], H.MlpSpec(4 * width)) for i in range(stored)), 1e-5,
        architecture="Bananex", logit_scale=0.5, loop=loop)


def kernel_table(size: str = "1b-layers", only: str = "", iters: int = 10) -> List[Dict]:
    """Every kernel of the design and the like kernels of the closest model on the shapes of ``size``: a
    prompt batch of 8 x 2048 tokens and a decode step of 64 sequences."""
    from ..infer.engine import make_engine
    from ..infer.kv_cache import PagedKVCache
    from ..ops import gemm as G
    from ..ops import latent as L
    from ..ops import ragged as R
    from ..ops import recurrence as RC
    from .serving_bench import CONTEXT, HEAD, SIZES, closest_kernels, recorder
    W, _, nh, kv = SIZES[size]
    dev, bf = "cuda", torch.bfloat16
    rows: List[Dict] = []
    rec = recorder(rows, only, iters)

    def t(*shape, dtype=bf):
        return torch.randn(shape, device=dev, dtype=torch.float32).to(dtype)
    lm = H.HybridLM.random(config(W, 12, nh, kv))
    la, lm2, lg = lm.layers[:3]
    for phase, B, S, at in (("prefill 8x2048", 8, 2048, 0), ("decode 64", 64, 1, CONTEXT)):
        T = B * S
        eng = make_engine(lm, max_batch=B)
        eng.open_slots(B, at + S + 64)
        for b in range(B):
            eng.cache.reserve(b, at + S)
        batch = eng._batch([R.Entry(b, at, [0] * S) for b in range(B)])
        prompt = S > 1

        def product(name, x, w, **kw):
            n, k = w.shape
            bound = dict(flops=2 * T * n * k) if prompt else dict(bytes_=n * k * 2)
            out = torch.empty((T, n), dtype=bf, device=dev)
            rec(name, phase, lambda: G.linear(x, w, out, **kw), **bound)

        def added(name, x, w):
            n, k = w.shape
            rec(name, phase, lambda: eng._product(x, w),
                **(dict(flops=2 * T * n * k) if prompt else dict(bytes_=n * k * 2)))
        x, h = t(T, W, dtype=torch.float32), t(T, W)
        y = eng._product(t(T, W), lg.w_out)
        norm = T * W * (8 + 2 + y.element_size())
        rec("add_norm with token shift", phase, lambda: R.add_norm(
            x, W, 1e-5, bf, y=y, bias=la.b_down, post=la.norm2b, gain=la.norm1, shift=la.shift,
            before=eng.state[0, "before"], batch=batch), bytes_=norm + (0 if prompt else T * W * 8))
        rec("add_norm", phase, lambda: R.add_norm(x, W, 1e-5, bf, y=y, post=la.norm1b, gain=la.norm2),
            bytes_=norm)
        both = t(T, 2 * W)
        added("linear loop (x, x0)", both, lm.loop_in)
        product("linear up, bias, gelu", h, la.w_up, epi="gelu_erf", bias=la.b_up)
        added("linear down", t(T, 4 * W), la.w_down)
        # ---- latent attention
        product("linear latent in", h, la.w_in)
        raw = t(T, la.w_in.shape[0])
        rope = R.rope_table(batch.pos, lm.inv_freq[la.rope_key])
        s, cache, table = la.spec.mixer, eng.cache.k[0], eng.cache.page_table
        P, row_p, gate = la.w_kv.shape[2], cache.shape[-1], raw[:, la.seg["g"]:]
        plan = eng._plan(s)
        lat = t(max(T, batch.kv_rows(plan)), row_p) if prompt else None
        prep = lambda: L.latent_prep(raw, la.seg["dkv"], nh, DIM, ROT, RANK, la.latent_norm, 1e-5, rope,  # noqa: E731
                                     P, batch, cache, table, rows_out=lat)
        rec("latent_prep", phase, prep,
            bytes_=T * 2 * (2 * nh * P + (3 if prompt else 2) * row_p))
        q, out = prep(), torch.empty((T, nh * VDIM), dtype=bf, device=dev)
        if prompt:
            product("linear latent to keys and values", lat, la.w_kv.view(2 * nh * P, row_p))
            key_val = t(T, 2 * nh * P)
            pairs = B * (WINDOW * WINDOW / 2 + (S - WINDOW) * WINDOW)
            rec("attention (window pieces)", phase, lambda: L.piece_attention(
                q, key_val, batch, plan, VDIM, s.scale, gate, out), flops=4 * pairs * nh * P)
        else:
            ql = torch.empty((T, nh, row_p), dtype=bf, device=dev)
            rec("linear_heads absorb", phase, lambda: L.linear_heads(
                q, la.w_absorb, ql.view(T, -1), row_p, x_rows=batch.rows),
                bytes_=la.w_absorb.numel() * 2 + T * nh * (P + row_p) * 2)
            ctx = lambda: L.latent_attention(ql, cache, table, batch, batch.rows, RANK, ROT, s.scale,  # noqa: E731
                                             WINDOW, at + 1)
            rec("latent_attention (decode)", phase, ctx, bytes_=B * WINDOW * row_p * 2 + T * nh * (row_p + RANK) * 2,
                flops=2 * B * WINDOW * nh * (row_p + RANK))
            o = ctx()
            rec("linear_heads value, gate", phase, lambda: L.linear_heads(
                o, la.w_value[:, :, :RANK], out, VDIM, y_rows=batch.rows, gate=gate),
                bytes_=nh * VDIM * RANK * 2 + T * nh * (RANK + 2 * VDIM) * 2)
        added("linear latent out", out, la.w_out)
        # ---- Mamba-2
        m, st = lm2.spec.mixer, eng.state
        product("linear mamba2 in", h, lm2.w_in)
        raw = t(T, lm2.w_in.shape[0])
        conv = lambda: RC.shortconv_act(raw, lm2.seg["x"], lm2.conv, lm2.conv_b, st[1, "conv"], batch)  # noqa: E731
        rec("shortconv_act", phase, conv, bytes_=T * lm2.channels * (4 + (0 if prompt else 12)))
        u, y2 = conv(), t(T, m.out_dim)
        scan = lambda: RC.ssd_scan(u, lm2.boff, lm2.coff, raw[:, lm2.seg["dt"]:], lm2.dt_bias, lm2.A_log,  # noqa: E731
                                   lm2.D, st[1, "ssd"], m.groups, m.vdim, batch, y2)
        io = T * (lm2.channels + m.out_dim) * 2
        if prompt:      # as a recurrence on the FMA units: decay, outer product, read-out
            rec("ssd_scan (chunks)", phase, scan, bytes_=io, fma=3 * T * m.heads * m.vdim * m.state)
        else:
            rec("ssd_scan (step)", phase, scan, bytes_=io + T * m.heads * m.vdim * m.state * 8)
        out2 = torch.empty_like(y2)
        rec("gated_group_norm", phase, lambda: RC.gated_group_norm(
            y2, raw[:, lm2.seg["z"]:], lm2.out_norm, 1, 1e-5, out2), bytes_=T * m.out_dim * 6)
        added("linear mamba2 out", out2, lm2.w_out)
        # ---- minGRU
        product("linear mingru in, bias", h, lg.w_in, bias=lg.b_in)
        raw, out3 = t(T, lg.w_in.shape[0]), torch.empty((T, W), dtype=bf, device=dev)
        rec("mingru_scan", phase, lambda: RC.mingru_scan(
            raw, lg.seg["z"], lg.seg["x"], lg.seg["g"], st[2, "gru"], batch, out3),
            bytes_=T * W * 8 + (0 if prompt else T * W * 8))
        pages = (at + S + 63) // 64
        c = PagedKVCache(1, kv, HEAD, B * pages, B, pages, dev)
        for b in range(B):
            c.reserve(b, at + S)
        closest_kernels(rec, phase, B, S, at, W, nh, kv, c)
        del eng, c
    return rows
