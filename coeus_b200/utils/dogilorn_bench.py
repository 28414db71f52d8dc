"""Sizes of the Dogilorn serving benchmark and its kernels one by one against the roofline (see
:mod:`coeus_b200.utils.serving_bench`).

Every layer has attention under a window that keeps the first tokens; every third one uses the keys and
values of the layer before it.  The first feed-forward is dense, the others choose 4 of 32 experts, four of
which are identities, beside a shared one.  The closest model is a Rupasun decoder with capped attention
under the same window in every layer and experts of the same sizes; :func:`closest_config`."""
from __future__ import annotations

from typing import Dict, List

import torch

from ..models import hybrid as H

HEAD, WINDOW, KEEP_FIRST = 128, 1024, 4
EXPERTS, IDENTITY, TOP, GROUPS, KEEP = 28, 4, 4, 4, 2


def _shared(width: int) -> int:
    return (2 * width // 3 + 127) // 128 * 128


def config(width: int, layers: int, heads: int, kv_heads: int) -> H.HybridConfig:
    from .serving_bench import VOCAB

    def attention(i: int) -> H.KeptWindowAttentionSpec:
        return H.KeptWindowAttentionSpec(heads, kv_heads, HEAD, HEAD, HEAD ** -0.5, HEAD, 5e5, WINDOW,
                                         keep_first=KEEP_FIRST, kv_from=i - 1 if i % 3 == 2 else None)
    moe = H.SoftmaxMoeSpec(EXPERTS, TOP, H.GluSpec(width // 2), groups=GROUPS, keep=KEEP,
                           shared=H.GluSpec(_shared(width)), identity=IDENTITY)
    dense = H.GluMlpSpec((8 * width // 3 + 127) // 128 * 128, 7.0)
    return H.HybridConfig(VOCAB, width, tuple(H.LayerSpec(attention(i), moe if i else dense) for i in range(layers)),
                          1e-5, architecture="Dogilorn", embed_scale=width ** 0.5, conv_taps=4)


def closest_config(width: int, layers: int, heads: int, kv_heads: int) -> H.HybridConfig:
    from .serving_bench import VOCAB
    capped = H.CappedAttentionSpec(heads, kv_heads, HEAD, HEAD, HEAD ** -0.5, HEAD, 5e5, WINDOW, 30.0)
    moe = H.MoeSpec(EXPERTS + IDENTITY, TOP, H.GluSpec(width // 2, 7.0), 2.0, GROUPS, KEEP,
                    H.GluSpec(_shared(width), 7.0))
    return H.HybridConfig(VOCAB, width, tuple(
        H.LayerSpec(capped, moe if i else H.MlpSpec(4 * width)) for i in range(layers)), 1e-5,
        architecture="Rupasun")


def _kernels(rec, lm: H.HybridLM, label: str, phase: str, B: int, S: int, at: int, W: int, nh: int, kv: int) -> None:
    """The kernels of one model on a batch of ``B`` entries of ``S`` tokens at position ``at``."""
    from ..infer.engine import make_engine
    from ..ops import experts as X
    from ..ops import gemm as G
    from ..ops import ragged as R
    dev, bf, eps, T, prompt = "cuda", torch.bfloat16, 1e-5, B * S, S > 1

    def t(*shape, dtype=bf):
        return torch.randn(shape, device=dev, dtype=torch.float32).to(dtype)
    eng = make_engine(lm, max_batch=B)
    eng.open_slots(B, at + S + 64)
    for b in range(B):
        eng.cache.reserve(b, at + S)
    batch = eng._batch([R.Entry(b, at, [0] * S) for b in range(B)])

    def r(name, fn, **kw):
        rec(label + name, phase, fn, **kw)

    def bound(n, k):
        return dict(flops=2 * T * n * k) if prompt else dict(bytes_=n * k * 2)

    def product(name, x, w, **kw):
        out = torch.empty((T, w.shape[0] // (2 if kw.get("glu") else 1)), dtype=bf, device=dev)
        r(name, lambda: G.linear(x, w, out, **kw), **bound(*w.shape))

    def added(name, x, w):
        r(name, lambda: eng._product(x, w), **bound(*w.shape))
    dense, layer = lm.layers[0], lm.layers[1]
    x, h = t(T, W, dtype=torch.float32), t(T, W)
    y = eng._product(t(T, W), layer.w_out)
    io = T * W * (8 + 2 + y.element_size())
    tail = dict(post=layer.norm1b, scale=layer.scale1, y=y)
    r("add_norm", lambda: R.add_norm(x, W, eps, bf, gain=layer.norm2, center=layer.center2, **tail), bytes_=io)
    if layer.taps is not None:
        state = eng.state[1, "before"]
        r("add_norm with the input convolution", lambda: R.add_norm(
            x, W, eps, bf, gain=layer.norm1, center=layer.center1, taps=layer.taps, before=state, batch=batch, **tail),
            bytes_=io + (0 if prompt else 2 * state[:1].numel() * 4 * B))
    product("linear dense up", h, dense.w_up, epi=lm.cfg.design.act, bias=dense.b_up, glu=dense.glu)
    added("linear dense down", t(T, dense.ff_padded), dense.w_down)
    # ---- attention: with keys of its own, then with those of another layer
    for n, part in ((1, layer), (2, lm.layers[2])):
        s = part.spec.mixer
        own = s.kv_from is None
        if n == 2 and own:
            continue
        name = "" if own else " (shared keys)"
        product(f"linear in{name}", h, part.w_in)
        raw, out = t(T, part.w_in.shape[0]), torch.empty((T, nh * HEAD), dtype=bf, device=dev)
        rope = {k: R.rope_table(batch.pos, f) for k, f in lm.inv_freq.items()}
        table, c, i, plan = rope[part.rope_key], eng.cache, eng._cache_index[n], eng._plan(s)
        rows = batch.kv_rows(plan)
        k_rows, v_rows = (t(rows, kv, HEAD), t(rows, kv, HEAD)) if rows else (None, None)
        heads = nh + (2 * kv if own else 0)
        prep = lambda: R.head_prep(                                              # noqa: E731
            raw, part.seg.get("k", 0), part.seg.get("v", 0), nh, kv if own else 0, HEAD, HEAD, batch, table, c.k[i],
            c.v[i], c.page_table, interleaved=True, unit_eps=eps if s.unit_qk else None,
            q_head=HEAD if rows else None, k_rows=k_rows if own else None, v_rows=v_rows if own else None, eps=eps,
            q_norm=part.q_norm, k_norm=part.k_norm, unit_v=s.unit_v, q_factor=part.temp)
        r(f"head_prep{name}", prep, bytes_=T * HEAD * 2 * (2 * heads + (2 * kv if rows and own else 0)))
        q = prep()

        def attn(q, b, out, k, v):
            return R.ragged_attention(
                q, c.k[i], c.v[i], c.page_table, b, nh, kv, HEAD, HEAD, s.scale, out, window=s.window,
                keep=s.keep_first, softcap=s.softcap, score_max=s.score_max, sink=part.sink,
                gate=raw[:out.shape[0], part.seg["g"]:] if s.gated else None, gate_wide=True, k_rows=k, v_rows=v,
                plan=plan)
        seen = min(WINDOW, at + S)
        if prompt and own:
            pairs = B * (seen * seen / 2 + (S - seen) * seen)
            r("attention (pieces)", lambda: attn(q, batch, out, k_rows, v_rows), flops=4 * pairs * nh * HEAD)
            for b in range(B):
                c.reserve(b, 2048)
            cont = eng._batch([R.Entry(b, 1536, [0] * 512) for b in range(B)])
            k2, v2 = t(cont.kv_rows(plan), kv, HEAD), t(cont.kv_rows(plan), kv, HEAD)
            r("attention (continued, cached keys)", lambda: attn(q[:B * 512], cont, out[:B * 512], k2, v2),
              flops=4 * B * 512 * WINDOW * nh * HEAD)
        elif own:
            r("attention (decode)", lambda: attn(q, batch, out, None, None), bytes_=B * seen * kv * HEAD * 4)
        if own:
            added("linear out", out, part.w_out)
    # ---- experts
    ex, moe = layer.experts, layer.experts.spec
    ff, fs, route = moe.expert.ff, moe.shared.ff, ex.routing
    chosen = X.route(h, ex.router, route, ex.correction)
    real = int((chosen.expert < moe.experts).sum())
    used = len(torch.unique(chosen.expert.clamp_max(moe.experts - 1)))
    r("route", lambda: X.route(h, ex.router, route, ex.correction),
      bytes_=T * W * 2 if prompt else ex.router.numel() * 2)
    weights = used * 3 * ff * W * 2
    if T <= X.FEW:
        r("experts and shared (few rows)", lambda: X.experts_few(
            h, chosen, route, ex.w_in, ex.w_down, moe.expert.limit, ex.s_in, ex.s_down, moe.shared.limit, ex.slope,
            ex.shift), bytes_=weights + 3 * fs * W * 2)
        return
    s = X.sort_rows(h, chosen, route)
    r("sort_rows", lambda: X.sort_rows(h, chosen, route), bytes_=T * W * 2 + real * W * 2)
    n = s.rows.shape[0]
    act, res = t(n, ff), t(n, W)
    unit = (ex.slope, moe.expert.limit, ex.shift)
    r("experts in, gated unit", lambda: X.grouped_linear(s.rows, ex.w_in, s.block_expert, act, glu=unit),
      **(dict(flops=4 * real * ff * W) if prompt else dict(bytes_=weights * 2 / 3)))
    r("experts down", lambda: X.grouped_linear(act, ex.w_down, s.block_expert, res),
      **(dict(flops=2 * real * ff * W) if prompt else dict(bytes_=weights / 3)))
    product("linear shared in, gated unit", h, ex.s_in, glu=unit)
    added("linear shared down", t(T, fs), ex.s_down)
    ys = eng._product(t(T, fs), ex.s_down)
    spread = R.Spread(res, s.slot, chosen.weight, h if moe.identity else None)
    tail.update(y=ys, y_weight=chosen.shared, spread=spread, post=layer.norm2b, scale=layer.scale2)
    nbytes = T * W * (8 + 2 + ys.element_size() + 2 * TOP)
    if layer.taps is None:
        r("add_norm with spread", lambda: R.add_norm(x, W, eps, bf, gain=layer.norm1, **tail), bytes_=nbytes)
    else:
        r("add_norm with spread and the input convolution", lambda: R.add_norm(
            x, W, eps, bf, gain=layer.norm1, center=layer.center1, taps=layer.taps, before=state, batch=batch, **tail),
            bytes_=nbytes + (0 if prompt else 2 * state[:1].numel() * 4 * B))


def kernel_table(size: str = "1b-layers", only: str = "", iters: int = 10) -> List[Dict]:
    """Every kernel of the design and the like kernels of the closest models on the shapes of ``size``: a
    prompt batch of 8 x 2048 tokens, decode steps of 64 and 16 sequences."""
    from ..infer.kv_cache import PagedKVCache
    from .serving_bench import CONTEXT, SIZES, closest_kernels, recorder
    W, _, nh, kv = SIZES[size]
    rows: List[Dict] = []
    rec = recorder(rows, only, iters)
    models = [(H.HybridLM.random(config(W, 3, nh, kv)), ""),
              (H.HybridLM.random(closest_config(W, 2, nh, kv)), "closest: ")]
    models[1][0].layers.append(models[1][0].layers[1])
    for phase, B, S, at in (("prefill 8x2048", 8, 2048, 0), ("decode 64", 64, 1, CONTEXT),
                            ("decode 16", 16, 1, CONTEXT)):
        for lm, label in models:
            _kernels(rec, lm, label, phase, B, S, at, W, nh, kv)
        if B == 16:
            continue
        pages = (at + S + 63) // 64
        cache = PagedKVCache(1, kv, HEAD, B * pages, B, pages, "cuda")
        for b in range(B):
            cache.reserve(b, at + S)
        closest_kernels(rec, phase, B, S, at, W, nh, kv, cache, "decoder: ")
        del cache
    return rows
