"""Sizes of the Rupasun serving benchmark and its kernels one by one against the roofline (see
:mod:`coeus_b200.utils.serving_bench`).

Two layers of differential attention, then one of capped attention under a window, and so on; the first
feed-forward is dense, the others choose 4 of 32 experts beside a shared one, with as many numbers in use
per token as the dense one has."""
from __future__ import annotations

from typing import Dict, List

import torch

from ..models import hybrid as H

MAP, HEAD, WINDOW, CAP = 64, 128, 1024, 30.0     # size of a map's keys, of values and capped heads
EXPERTS, TOP, GROUPS, KEEP = 32, 4, 4, 2


def config(width: int, layers: int, heads: int, kv_heads: int) -> H.HybridConfig:
    from .serving_bench import VOCAB
    diff = H.DiffAttentionSpec(heads, kv_heads, MAP, HEAD, MAP ** -0.5, MAP, 1e6, diff=0.4)
    capped = H.CappedAttentionSpec(heads, kv_heads, HEAD, HEAD, HEAD ** -0.5, HEAD, 1e4, WINDOW, CAP)
    shared = (2 * width // 3 + 127) // 128 * 128
    moe = H.MoeSpec(EXPERTS, TOP, H.GluSpec(width // 2, 7.0), 2.0, GROUPS, KEEP, H.GluSpec(shared, 7.0))
    return H.HybridConfig(VOCAB, width, tuple(
        H.LayerSpec(capped if i % 3 == 2 else diff, moe if i else H.MlpSpec(4 * width))
        for i in range(layers)), 1e-5, architecture="Rupasun")


def kernel_table(size: str = "1b-layers", only: str = "", iters: int = 10) -> List[Dict]:
    """Every kernel of the design and the like kernels of the closest models on the shapes of ``size``: a
    prompt batch of 8 x 2048 tokens, decode steps of 64 and 16 sequences."""
    from ..infer.engine import make_engine
    from ..infer.kv_cache import PagedKVCache
    from ..ops import experts as X
    from ..ops import gemm as G
    from ..ops import moe as M
    from ..ops import ragged as R
    from .serving_bench import CONTEXT, SIZES, closest_kernels, recorder
    W, _, nh, kv = SIZES[size]
    dev, bf, eps = "cuda", torch.bfloat16, 1e-5
    rows: List[Dict] = []
    rec = recorder(rows, only, iters)

    def t(*shape, dtype=bf):
        return torch.randn(shape, device=dev, dtype=torch.float32).to(dtype)
    lm = H.HybridLM.random(config(W, 3, nh, kv))
    dense, lc = lm.layers[0], lm.layers[2]
    ex, moe = lc.experts, lc.experts.spec
    r = ex.routing
    ff, fs = moe.expert.ff, moe.shared.ff
    for phase, B, S, at in (("prefill 8x2048", 8, 2048, 0), ("decode 64", 64, 1, CONTEXT),
                            ("decode 16", 16, 1, CONTEXT)):
        T = B * S
        eng = make_engine(lm, max_batch=B)
        eng.open_slots(B, at + S + 64)
        for b in range(B):
            eng.cache.reserve(b, at + S)
        batch = eng._batch([R.Entry(b, at, [0] * S) for b in range(B)])
        prompt = S > 1

        def bound(n, k):
            return dict(flops=2 * T * n * k) if prompt else dict(bytes_=n * k * 2)

        def product(name, x, w, **kw):
            n, k = w.shape
            out = torch.empty((T, n // 2 if "glu" in kw else n), dtype=bf, device=dev)
            rec(name, phase, lambda: G.linear(x, w, out, **kw), **bound(n, k))

        def added(name, x, w):
            rec(name, phase, lambda: eng._product(x, w), **bound(*w.shape))
        x, h = t(T, W, dtype=torch.float32), t(T, W)
        y = eng._product(t(T, W), lc.w_out)
        io = T * W * (8 + 2 + y.element_size())
        rec("add_norm", phase, lambda: R.add_norm(x, W, eps, bf, y=y, post=lc.norm1b, gain=lc.norm2), bytes_=io)
        product("linear dense up, squared relu", h, dense.w_up, epi="relu2")
        added("linear dense down", t(T, 4 * W), dense.w_down)
        # ---- attention
        for name, n, layer in (("diff", 0, dense), ("capped", 2, lc)):
            s, kh = layer.spec.mixer, kv * layer.spec.mixer.maps
            product(f"linear {name} in", h, layer.w_in)
            raw = t(T, layer.w_in.shape[0])
            rope = R.rope_table(batch.pos, lm.inv_freq[layer.rope_key])
            c, i, plan = eng.cache, eng._cache_index[n], eng._plan(s)
            qh, vh = R.row_heads(s.dim, s.vdim, s.maps)
            k_rows = t(T, kh, qh) if prompt else None
            v_rows = t(T, kv, vh) if prompt else None
            prep = lambda: R.head_prep(                                              # noqa: E731
                raw, layer.seg["k"], layer.seg["v"], nh * s.maps, kh, s.dim, s.vdim, batch, rope, c.k[i], c.v[i],
                c.page_table, interleaved=s.interleaved, unit_eps=eps if s.unit_qk else None,
                q_head=qh if prompt else None, k_rows=k_rows, v_rows=v_rows)
            qk, v = (nh + kv) * s.maps * s.dim, kv * s.vdim
            rec(f"head_prep {name}", phase, prep, bytes_=T * 2 * (2 * (qk + v) + (kh * s.dim + v if prompt else 0)))
            q, out = prep(), torch.empty((T, nh * s.vdim), dtype=bf, device=dev)
            attn = lambda: R.ragged_attention(                                       # noqa: E731
                q, c.k[i], c.v[i], c.page_table, batch, nh, kv, s.dim, s.vdim, s.scale, out, window=s.window,
                softcap=s.softcap, score_max=s.score_max, maps=s.maps, map_weight=layer.map_weight,
                map_factor=1.0 - s.diff if s.maps == 2 else 1.0, eps=eps,
                gate=raw[:, layer.seg["g"]:] if s.gated else None, gate_wide=True, k_rows=k_rows, v_rows=v_rows,
                plan=plan)
            seen = min(s.window or at + S, at + S)
            if prompt:
                pairs = B * (seen * seen / 2 + (S - seen) * seen)
                rec(f"attention {name} (pieces)", phase, attn, flops=2 * pairs * nh * s.maps * (s.dim + s.vdim))
                if name == "diff":
                    for b in range(B):
                        eng.cache.reserve(b, 1024)
                    part = eng._batch([R.Entry(b, 512, [0] * 512) for b in range(B)])
                    k2, v2 = t(part.kv_rows(plan), kh, qh), t(part.kv_rows(plan), kv, vh)
                    pairs = B * (512 * 512 + 512 * 512 / 2)
                    rec("attention diff (continued, cached keys)", phase, lambda: R.ragged_attention(
                        q[:B * 512], c.k[i], c.v[i], c.page_table, part, nh, kv, s.dim, s.vdim, s.scale,
                        out[:B * 512], maps=2, map_weight=layer.map_weight, map_factor=0.6, eps=eps, k_rows=k2,
                        v_rows=v2, plan=plan), flops=2 * pairs * nh * s.maps * (s.dim + s.vdim))
            else:
                rec(f"attention {name} (decode)", phase, attn, bytes_=B * seen * (kh * s.dim + kv * s.vdim) * 2)
            added(f"linear {name} out", out, layer.w_out)
        # ---- experts
        c = X.route(h, ex.router, r)
        used = len(torch.unique(c.expert))
        route_bytes = T * W * 2 if prompt else EXPERTS * W * 2
        rec("route", phase, lambda: X.route(h, ex.router, r), bytes_=route_bytes)
        weights = used * 3 * ff * W * 2
        if T <= X.FEW:
            rec("experts and shared (few rows)", phase, lambda: X.experts_few(
                h, c, r, ex.w_in, ex.w_down, moe.expert.limit, ex.s_in, ex.s_down, moe.shared.limit, ex.slope),
                bytes_=weights + 3 * fs * W * 2)
        else:
            s = X.sort_rows(h, c, r)
            rec("sort_rows", phase, lambda: X.sort_rows(h, c, r), bytes_=T * W * 2 * (1 + TOP))
            n = s.rows.shape[0]
            act, res = t(n, ff), t(n, W)
            pairs = T * TOP
            rec("experts in, gated unit", phase, lambda: X.grouped_linear(
                s.rows, ex.w_in, s.block_expert, act, glu=(ex.slope, moe.expert.limit)),
                **(dict(flops=4 * pairs * ff * W) if prompt else dict(bytes_=weights * 2 / 3)))
            rec("experts down", phase, lambda: X.grouped_linear(act, ex.w_down, s.block_expert, res),
                **(dict(flops=2 * pairs * ff * W) if prompt else dict(bytes_=weights / 3)))
            product("linear shared in, gated unit", h, ex.s_in, glu=(ex.slope, moe.shared.limit))
            added("linear shared down", t(T, fs), ex.s_down)
            ys = eng._product(t(T, fs), ex.s_down)
            spread = R.Spread(res, s.slot, c.weight)
            rec("add_norm with spread", phase, lambda: R.add_norm(
                x, W, eps, bf, y=ys, post=lc.norm1b, gain=lc.norm2, spread=spread),
                bytes_=T * W * (8 + 2 + ys.element_size() + 2 * TOP))
            del s, act, res, spread
        del eng, batch
        if B == 16:
            continue
        pages = (at + S + 63) // 64
        cache = PagedKVCache(1, kv, HEAD, B * pages, B, pages, dev)
        for b in range(B):
            cache.reserve(b, at + S)
        closest_kernels(rec, phase, B, S, at, W, nh, kv, cache)
        del cache
        # the mixture of experts of the training stack: equal capacities, softmax routing
        cap = max(128, T * TOP // EXPERTS)
        logits = t(T, EXPERTS, dtype=torch.float32)
        expert, w, _, slot, _ = M.route(logits, TOP, cap)
        rec("closest: moe route", phase, lambda: M.route(logits, TOP, cap), bytes_=T * EXPERTS * 8)
        send = t(EXPERTS * cap, W)
        rec("closest: moe gather", phase, lambda: M.gather_rows(h, expert, slot, send, cap),
            bytes_=T * W * 2 * (1 + TOP))
        xg = send.view(EXPERTS, cap, W)
        wg, wd = t(EXPERTS, W, 2 * ff), t(EXPERTS, ff, W)
        grouped = (lambda f: dict(flops=f * EXPERTS * cap)) if prompt else \
            (lambda f: dict(bytes_=f * EXPERTS))                                     # noqa: E731
        rec("closest: grouped gate and up", phase, lambda: G.gemm_grouped(xg, wg, b_mn=True), **grouped(4 * ff * W))
        ag = t(EXPERTS, cap, ff)
        rec("closest: grouped down", phase, lambda: G.gemm_grouped(ag, wd, b_mn=True), **grouped(2 * ff * W))
        rec("closest: moe combine", phase, lambda: M.combine_rows(send, expert, slot, cap, w, h),
            bytes_=T * W * 2 * (2 + TOP))
        del send, xg, wg, wd, ag
    return rows
