"""Serving throughput of a design of mixed layers beside the framework's closest model at equal size,
and its kernels one by one against the roofline (``python bench.py --serving
sapasun|bananex|rupasun|dogilorn [--kernels]``; designs behind the first are in :mod:`coeus_b200.utils.bananex_bench`,
:mod:`coeus_b200.utils.rupasun_bench` and :mod:`coeus_b200.utils.dogilorn_bench`).

The closest model is the RMSNorm / SwiGLU / rotary decoder with grouped-query attention: same
width, depth, heads and vocabulary, the feed-forward as wide as gives the same parameters per
layer (three matrices of 8/3 width against two of 4 width; for a mixture of experts: per token).  Dogilorn
also runs beside a Rupasun model of the same window and experts.  Weights are random.  Times are CUDA
events around whole engine calls (prompt batches, decode steps), after warm-up; every call streams
weights and caches far above the L2 cache.  The kernel table flushes L2 between launches.
"""
from __future__ import annotations

import json
import time
from typing import Callable, Dict, List

import torch

from ..models import hybrid as H
from ..models.config import DecoderConfig
from ..models.decoder import DecoderLM
from ..infer.engine import make_engine

VOCAB = 32000
SIZES = {   # width, layers, heads, key/value heads
    "1b-layers": (2048, 12, 16, 4),
    "7b-layers": (4096, 6, 32, 8),
}
HEAD = 128
CHUNK = 1024
PROMPTS = ((1, 4096), (8, 2048))
DECODE = (1, 16, 64)
CONTEXT = 2560       # in the middle of a chunk


def sapasun_config(width: int, layers: int, heads: int, kv_heads: int) -> H.HybridConfig:
    """Two attention layers, then a recurrent one, and so on."""
    attn = H.AttentionSpec(heads, kv_heads, HEAD, HEAD, 4, HEAD ** -0.5, CHUNK, HEAD // 2, 1e6, True)
    delta = H.ChannelDeltaSpec(heads, heads, HEAD, HEAD, 4, HEAD, HEAD)
    return H.HybridConfig(VOCAB, width, tuple(
        H.LayerSpec(delta if i % 3 == 2 else attn, H.MlpSpec(4 * width)) for i in range(layers)),
        1e-5, 30.0)


def closest_config(width: int, layers: int, heads: int, kv_heads: int) -> DecoderConfig:
    return DecoderConfig(hidden_dim=width, num_layers=layers, num_heads=heads, num_kv_heads=kv_heads,
                         intermediate_dim=(8 * width // 3 + 127) // 128 * 128, vocab_size=VOCAB,
                         max_seq_len=8192, use_bias=False, activation="swiglu", norm="rmsnorm",
                         pos="rope")


def timed(fn: Callable[[], object], n: int, warmup: int) -> float:
    """Milliseconds per call."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(n):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / n


def throughput(model, steps: int, warmup: int) -> List[Dict]:
    out = []
    g = torch.Generator(device="cuda").manual_seed(0)
    for B, S in PROMPTS:
        ids = torch.randint(0, VOCAB, (B, S), device="cuda", generator=g)
        eng = make_engine(model, max_batch=B)
        ms = timed(lambda: eng.prefill(ids, S + 64), max(3, steps // 4), warmup)
        out.append({"phase": "prefill", "batch": B, "tokens": S, "ms": ms,
                    "tokens_per_s": B * S / ms * 1e3})
    for B in DECODE:
        ids = torch.randint(0, VOCAB, (B, CONTEXT), device="cuda", generator=g)
        eng = make_engine(model, max_batch=B)
        eng.prefill(ids, CONTEXT + warmup + 2 * steps + 64, seq_chunk=8)
        tok = torch.zeros(B, dtype=torch.int64, device="cuda")
        ms = timed(lambda: eng.decode_step(tok), 2 * steps, warmup)
        out.append({"phase": "decode", "batch": B, "context": CONTEXT, "ms": ms,
                    "tokens_per_s": B / ms * 1e3})
        del eng
    return out


def recorder(rows: List[Dict], only: str, iters: int) -> Callable:
    """``rec(name, phase, fn, bytes_ | flops | fma)``: times ``fn`` with L2 flushed in between and adds a
    row; the bound is the largest of the times its bytes, bf16 operations and fp32 FMAs need."""
    from .kernel_bench import peaks, timeit
    hbm, tensor, source = peaks()
    fp32 = 148 * 128 * 1.965e9          # FMA issue slots per second

    def rec(name, phase, fn, bytes_=0, flops=0, fma=0):
        if only not in f"{name}, {phase}":
            return
        us = timeit(fn, min(3, iters), iters, True) * 1e3
        best, kind = max((bytes_ / hbm / 1e3, "bytes"), (flops / tensor / 1e6, "bf16"),
                         (fma / fp32 * 1e6, "fp32"))
        rows.append({"kernel": name, "phase": phase, "us": round(us, 1), "bound": kind,
                     "roofline_us": round(best, 1), "fraction": round(best / us, 3),
                     "peaks": source})
    return rec


def closest_kernels(rec, phase: str, B: int, S: int, at: int, W: int, nh: int, kv: int, c,
                    label: str = "closest: ") -> None:
    """The closest model's kernels at width ``W``; ``c`` is a cache of ``kv`` heads of ``HEAD``."""
    from ..ops import attention as A
    from ..ops import decode as D
    from ..ops import elementwise as E
    from ..ops import gemm as G
    from ..ops import norm as N
    T, d, dev = B * S, HEAD, "cuda"
    qkv = (nh + 2 * kv) * d

    def t(*shape):
        return torch.randn(shape, device=dev, dtype=torch.float32).to(torch.bfloat16)
    q = t(T, nh, d)
    hx, wn = t(T, W), t(W)
    rec(label + "norm_fwd", phase, lambda: N.norm_fwd(hx, wn, None, 1e-5, True), bytes_=T * W * 4)
    w1 = t(W, qkv)
    if S > 1:
        rec(label + "linear qkv", phase, lambda: G.linear_fwd(hx, w1), flops=2 * T * W * qkv)
        kk, vv = t(T, kv * d), t(T, kv * d)
        rec(label + "attention", phase, lambda: A.attention_fwd(q.view(T, -1), kk, vv, B, S, nh, d, causal=True),
            flops=4 * B * S * S / 2 * nh * d)
    else:
        rec(label + "linear qkv", phase, lambda: G.linear_fwd(hx, w1), bytes_=W * qkv * 2)
        ctx = torch.full((B,), CONTEXT, dtype=torch.int32, device=dev)
        pages = (CONTEXT + 63) // 64
        kc, vc = t(B * pages, 64, kv, d), t(B * pages, 64, kv, d)
        pt = torch.arange(B * pages, dtype=torch.int32, device=dev).view(B, pages)
        rec(label + "attention", phase, lambda: D.decode_attention(q.view(T, -1), kc, vc, pt, ctx, nh, d, nkv=kv),
            bytes_=B * CONTEXT * kv * d * 2 * 2)
    buf = t(T, qkv)
    pos = torch.full((B,), at, dtype=torch.int32, device=dev)
    rec(label + "rope", phase, lambda: E.rope_(buf, nh + kv, d, S, pos_dev=pos if S == 1 else None),
        bytes_=T * (nh + kv) * d * 4)
    rec(label + "kv_write", phase, lambda: D.kv_write(
        buf[:, nh * d:(nh + kv) * d], buf[:, (nh + kv) * d:], c.k[0], c.v[0], c.page_table, pos, S,
        kv, d), bytes_=T * kv * d * 2 * 4)
    gu = t(T, 2 * (8 * W // 3 // 128 * 128))
    rec(label + "swiglu", phase, lambda: E.swiglu_fwd(gu), bytes_=gu.numel() * 3)


def kernel_table(size: str = "1b-layers", only: str = "", iters: int = 10) -> List[Dict]:
    """Every kernel of the design and the like kernels of the closest model on the shapes of
    ``size``: a prompt batch of 8 x 2048 tokens and a decode step of 64 sequences.  ``bound`` names
    the roofline (measured copy bandwidth, measured bf16 throughput, or fp32 FMA issue at the
    maximum clock), ``fraction`` is algorithmic work / time / roofline."""
    from ..ops import gemm as G
    from ..ops import ragged as R
    W, _, nh, kv = SIZES[size]
    d, dev, bf = HEAD, "cuda", torch.bfloat16
    rows: List[Dict] = []
    rec = recorder(rows, only, iters)

    def t(*shape, dtype=bf):
        return torch.randn(shape, device=dev, dtype=torch.float32).to(dtype)
    cfg = sapasun_config(W, 3, nh, kv)
    lm = H.HybridLM.random(cfg)
    for phase, B, S, at in (("prefill 8x2048", 8, 2048, 0), ("decode 64", 64, 1, CONTEXT)):
        T = B * S
        eng = make_engine(lm, max_batch=B)
        eng.open_slots(B, at + S + 64)
        for b in range(B):
            eng.cache.reserve(b, at + S)
        batch = eng._batch([R.Entry(b, at, [0] * S) for b in range(B)])
        la, ld = lm.layers[0], lm.layers[2]
        x, wp = t(T, W, dtype=torch.float32), lm.layers[0].norm1
        out = torch.empty((T, la.w_out.shape[1]), dtype=bf, device=dev)
        rec("rms_rows (two norms)", phase, lambda: R.rms_rows(x, wp, W, 1e-5, bf, w2=wp),
            bytes_=T * W * 8)
        h = t(T, W)
        raw = t(T, la.w_in.shape[0])
        up = (h, la.w_up, out[:, la.act_off:], "relu2", None, False)
        n_in = la.w_in.shape[0] + la.w_up.shape[0]
        wb = lambda n, k: n * k * 2                                     # noqa: E731
        if S > 1:
            rec("linear in + up", phase, lambda: G.linear_pair((h, la.w_in, raw, "none", None, False), up),
                flops=2 * T * n_in * W)
            rec("linear out + down (added to the stream)", phase,
                lambda: G.linear(out, la.w_out, x, accumulate=True), flops=2 * T * W * la.w_out.shape[1])
        else:
            rec("linear in + up", phase, lambda: G.linear_pair((h, la.w_in, raw, "none", None, False), up),
                bytes_=wb(n_in, W))
            rec("linear out + down (added to the stream)", phase,
                lambda: G.linear(out, la.w_out, x, accumulate=True), bytes_=wb(W, la.w_out.shape[1]))
            h1 = t(1, W)
            raw1, out1 = raw[:1], out[:1]
            rec("linear in + up, 1 row", "decode 1", lambda: G.linear_pair(
                (h1, la.w_in, raw1, "none", None, False),
                (h1, la.w_up, out1[:, la.act_off:], "relu2", None, False)), bytes_=wb(n_in, W))
        rope = R.rope_table(batch.pos, lm.inv_freq[la.rope_key])
        st, c = eng.state, eng.cache
        kr = t(T, kv, d) if S > 1 else None
        vr = t(T, kv, d) if S > 1 else None
        vf = t(T, kv * d)
        qkv = (nh + 2 * kv) * d
        rec("shortconv_attn", phase, lambda: R.shortconv_attn(
            raw, la.seg["k"], la.seg["v"], la.conv, st[0, "conv"], nh, kv, d, d, batch, rope, c.k[0],
            c.v[0], c.page_table, v_first=vf, mix=la.mix, k_rows=kr, v_rows=vr),
            bytes_=T * (2 * qkv + 2 * kv * d * (2 if S > 1 else 0) + kv * d) * 2
            + (0 if S > 1 else T * 2 * 3 * qkv * 2))
        q = t(T, nh, d)
        gate = raw[:, la.seg["g"]:]
        attn = lambda: R.ragged_attention(                              # noqa: E731
            q, c.k[0], c.v[0], c.page_table, batch, nh, kv, d, d, d ** -0.5, out[:, :nh * d],
            chunk=CHUNK, sink=la.sink, gate=gate, k_rows=kr, v_rows=vr)
        if S > 1:
            pairs = B * sum(min(CHUNK, S - s) ** 2 / 2 for s in range(0, S, CHUNK))
            rec("attention (prompt pieces)", phase, attn, flops=4 * pairs * nh * d)
            for b in range(B):
                eng.cache.reserve(b, 1024)
            pairs = B * (512 * 512 + 512 * 512 / 2)      # half a chunk behind the cached other half
            part = eng._batch([R.Entry(b, 512, [0] * 512) for b in range(B)])
            k2, v2 = (t(part.kv_rows(R.AttnPlan(CHUNK, True)), kv, d) for _ in range(2))
            rec("attention (rest of a chunk, cached keys)", phase, lambda: R.ragged_attention(
                q[:B * 512], c.k[0], c.v[0], c.page_table, part, nh, kv, d, d, d ** -0.5,
                out[:B * 512, :nh * d], chunk=CHUNK, sink=la.sink, gate=gate[:B * 512],
                k_rows=k2, v_rows=v2), flops=4 * pairs * nh * d)
        else:
            rec("attention (decode)", phase, attn,
                bytes_=B * (at % CHUNK + 1) * kv * d * 2 * 2)
        raw_d = t(T, ld.w_in.shape[0])
        a = t(T, nh * d, dtype=torch.float32)
        conv = lambda: R.shortconv_delta(                               # noqa: E731
            raw_d, ld.seg["k"], ld.seg["v"], ld.seg["b"], ld.conv, st[2, "conv"], nh, nh, d, d, batch,
            a, ld.A_log, ld.dt_bias)
        rec("shortconv_delta", phase, conv, bytes_=T * nh * d * (3 * 2 + 5 * 4)
            + (0 if S > 1 else T * 2 * 3 * 3 * nh * d * 2))
        z = conv()
        scan = lambda: R.delta_scan(*z, st[2, "delta"], batch)          # noqa: E731
        if S > 1:
            rec("delta_scan", phase, scan, fma=4 * T * nh * d * d)
        else:
            rec("delta_scan", phase, scan, bytes_=B * nh * d * d * 8)
        o, g2 = t(T, nh, d, dtype=torch.float32), t(T, nh * d)
        rec("gated_head_norm", phase, lambda: R.gated_head_norm(o, g2, ld.head_norm, 1e-5,
                                                                out[:, :nh * d]),
            bytes_=T * nh * d * 8)
        closest_kernels(rec, phase, B, S, at, W, nh, kv, c)
        del eng, z
    return rows


DESIGNS = ("sapasun", "bananex", "rupasun", "dogilorn")


def bench_of(design: str):
    """``(config, kernel_table)`` of a design."""
    from . import bananex_bench, dogilorn_bench, rupasun_bench
    return {"sapasun": (sapasun_config, kernel_table),
            "bananex": (bananex_bench.config, bananex_bench.kernel_table),
            "rupasun": (rupasun_bench.config, rupasun_bench.kernel_table),
            "dogilorn": (dogilorn_bench.config, dogilorn_bench.kernel_table)}[design]


def run(design: str, steps: int = 20, warmup: int = 3, kernels: bool = False, sampler=None) -> None:
    """One JSON line per size and model, then (``kernels``) one per kernel."""
    from ..ops import _lib
    from .dogilorn_bench import closest_config as closest_hybrid
    config, table = bench_of(design)
    models = {design: lambda size: H.HybridLM.random(config(*size))}
    if design == "dogilorn":
        models["closest: rupasun"] = lambda size: H.HybridLM.random(closest_hybrid(*size))
    models["closest"] = lambda size: DecoderLM(closest_config(*size), "cuda", training=False)
    for name, size in SIZES.items():
        for which, make in models.items():
            model = make(size)
            s = sampler() if sampler is not None else None
            if s is not None:
                s.start()
            launches = _lib.launch_count
            t0 = time.perf_counter()
            rows = throughput(model, steps, max(warmup, 3))
            print(json.dumps({
                "metric": "serving tokens/sec (device-timed)", "size": name, "model": which,
                "config": {"width": size[0], "layers": size[1], "heads": size[2],
                           "kv_heads": size[3], "head_dim": HEAD, "vocab": VOCAB,
                           "l2": "no flush: every call streams more than L2"},
                "parameters": model.num_parameters(), "dtype": "bf16",
                "data": "synthetic (random weights and token ids)", "results": rows,
                "gpu_launches": _lib.launch_count - launches,
                "seconds": time.perf_counter() - t0,
                "clocks": s.stop() if s is not None else None}), flush=True)
            _lib.check_status(torch.device("cuda", torch.cuda.current_device()))
            del model
            torch.cuda.empty_cache()
    if kernels:
        for row in table():
            print(json.dumps(row), flush=True)


def main(argv=None) -> int:
    """``python -m coeus_b200.utils.serving_bench --kernel delta_scan``: a kernel table alone, or its
    rows whose ``name, phase`` contains the text (with ``--iters 1`` a small case for a profiler)."""
    import argparse
    ap = argparse.ArgumentParser()
    ap.add_argument("--design", default="sapasun", choices=DESIGNS)
    ap.add_argument("--size", default="1b-layers", choices=list(SIZES))
    ap.add_argument("--kernel", default="")
    ap.add_argument("--iters", type=int, default=10)
    a = ap.parse_args(argv)
    for row in bench_of(a.design)[1](a.size, a.kernel, a.iters):
        print(json.dumps(row), flush=True)
    return 0


if __name__ == "__main__":
    import sys
    sys.exit(main())
