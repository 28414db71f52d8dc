"""Serving engine of the hybrid decoders (:mod:`coeus_b200.models.hybrid`).

One step function runs everything: a step brings entries, each the next tokens of one sequence
(a whole prompt, a portion of one, or a single decoded token), and they go through the layers as
one ragged batch.  Keys and values live in the paged cache, convolution inputs and recurrent
states in slots.  A step whose entries are single tokens is replayed from a CUDA graph.

The generation, slot and serving interfaces of :class:`coeus_b200.infer.engine.InferenceEngine`
are kept on top of it.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import numpy as np
import torch

from ..foundation.error import ProcessingError
from ..models.hybrid import (CACHED, AttentionSpec, HeadAttentionSpec, HybridLM, LatentAttentionSpec,
                             Mamba2Spec)
from ..ops import experts as X
from ..ops import gemm as G
from ..ops import latent as L
from ..ops import ragged as R
from ..ops import recurrence as RC
from ..ops.decode import PAGE
from .engine import InferenceEngine
from .kv_cache import PagedKVCache, SequenceState

Entry = R.Entry


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class _KvRows:
    """Row-wise keys and values of a layer in one step: the step's rows, then cached ones gathered for the
    pieces of one plan."""

    k: Optional[torch.Tensor] = None
    v: Optional[torch.Tensor] = None
    gathered: Optional[R.AttnPlan] = None


class HybridEngine(InferenceEngine):
    ragged = True
    prefill_tokens = 16384       # rows of one step when a prompt batch is cut by generate()

    def __init__(self, model: HybridLM, max_batch: int = 64, max_len: Optional[int] = None,
                 use_graph: Optional[bool] = None) -> None:
        self.m = model
        self.cfg = model.cfg
        self.max_batch = max_batch
        self.max_len = max_len or self.cfg.max_seq_len
        self.cache: Optional[PagedKVCache] = None
        self.state: Optional[SequenceState] = None
        self.stats: Dict[str, float] = {}
        self.use_graph = (model.device.type == "cuda") if use_graph is None else use_graph
        self._graphs: Dict[int, tuple] = {}
        self._tiles = model.device.type == "cuda" and model.dtype == torch.bfloat16
        self._runs = self.cfg.runs()
        self._shared: Dict[int, List[int]] = {}     # layer -> the later layers that use its keys and values
        for i, layer in enumerate(self.cfg.layers):
            if getattr(layer.mixer, "kv_from", None) is not None:
                self._shared.setdefault(layer.mixer.kv_from, []).append(i)
        self._plans = [self._plan(layer.mixer) for layer in self.cfg.layers
                       if isinstance(layer.mixer, CACHED)]
        self._plans += [RC.ssd_plan(a.heads, a.vdim, a.state) for a in
                        (layer.mixer for layer in self.cfg.layers) if isinstance(a, Mamba2Spec)]

    def _plan(self, a) -> R.AttnPlan:
        if isinstance(a, AttentionSpec):
            return R.AttnPlan(a.chunk, self._tiles and R.pieces_allowed(a.dim, a.vdim, a.chunk, a.scale))
        if isinstance(a, HeadAttentionSpec):
            plain = a.maps == 1 or (a.softcap is None and not a.gated)
            plain &= not a.keep_first or (a.maps == 1 and a.softcap is None)
            return R.AttnPlan(None, self._tiles and plain and R.pieces_allowed(a.dim, a.vdim, None, a.scale),
                              a.window, tiles=a.maps * a.dim <= 256, keep=a.keep_first)
        return R.AttnPlan(None, self._tiles and L.pieces_allowed(a.dim + a.rot_dim, a.vdim, a.scale),
                          a.window or 1 << 30, tiles=False)

    def _batch(self, entries: List[Entry], into: Optional[R.RaggedBatch] = None) -> R.RaggedBatch:
        return R.RaggedBatch(entries, self.m.device, tile_rows=self._tiles, into=into,
                             plans=self._plans)

    # ------------------------------------------------------------------ cache and state
    def open_slots(self, max_seqs: int, max_len: int, num_pages: Optional[int] = None
                   ) -> PagedKVCache:
        """Cache and state for ``max_seqs`` sequences of up to ``max_len`` tokens.  ``num_pages``
        sizes the shared page pool (default: every slot can grow to ``max_len``).  Every run of a
        layer has a cache or state of its own."""
        m = self.m
        per_seq = max(1, (max_len + PAGE - 1) // PAGE)
        dims = []
        self._cache_index: Dict[int, int] = {}
        for n, run in enumerate(self._runs):
            a = m.layers[run.layer].spec.mixer
            if getattr(a, "kv_from", None) is not None:        # without a loop runs are layers
                self._cache_index[n] = self._cache_index[a.kv_from]
            elif isinstance(a, CACHED):
                self._cache_index[n] = len(dims)
                if isinstance(a, LatentAttentionSpec):
                    dims.append((1, _up8(a.latent), 0))
                else:
                    maps = getattr(a, "maps", 1)       # every map has a key of its own, values are shared
                    dims.append((a.kv_heads, _up8(a.dim), _up8(a.vdim), a.kv_heads * maps))
        self.cache = PagedKVCache(len(dims), 0, 0, num_pages or max_seqs * per_seq, max_seqs,
                                  per_seq, m.device, m.dtype, layer_dims=dims)
        self.state = SequenceState(max_seqs, m.device)
        for n, run in enumerate(self._runs):
            layer = m.layers[run.layer]
            s = layer.spec.mixer
            if hasattr(s, "conv"):
                self.state.add(n, "conv", (s.conv - 1, layer.channels), m.dtype)
            if s.kind == "channel_delta":
                self.state.add(n, "delta", (s.heads, s.dim, s.vdim), torch.float32)
            elif s.kind == "mamba2":
                self.state.add(n, "ssd", (s.heads, s.state, (s.vdim + 3) // 4 * 4), torch.float32)
            elif s.kind == "mingru":
                self.state.add(n, "gru", (_up8(s.width),), torch.float32)
            if layer.shift is not None:
                self.state.add(n, "before", (self.cfg.width_padded,), torch.float32)
            if layer.taps is not None:
                self.state.add(n, "before", (layer.taps.shape[0] - 1, self.cfg.width_padded), torch.float32)
        self._graphs.clear()
        return self.cache

    def release_slot(self, slot: int) -> None:
        self.cache.release(slot)

    # ------------------------------------------------------------------ one step
    def _mixer_in(self, layer, h1: torch.Tensor, h2: Optional[torch.Tensor]):
        """The stacked projections of the mixer and, in place in the ``[mixer | activation]``
        buffer, the feed-forward's activation."""
        T, m = h1.shape[0], self.m
        raw = torch.empty((T, layer.w_in.shape[0]), dtype=m.dtype, device=m.device)
        cat = torch.empty((T, layer.w_out.shape[1]), dtype=m.dtype, device=m.device)
        if layer.out_dim != layer.act_off:
            cat[:, layer.out_dim:layer.act_off].zero_()
        up = None
        if layer.w_up is not None:
            up = (h2, layer.w_up, cat[:, layer.act_off:], "relu2", None, False)
        G.linear_pair((h1, layer.w_in, raw, "none", None, False), up)
        return raw, cat

    def _attention(self, n: int, layer, raw: torch.Tensor, cat: torch.Tensor, b: R.RaggedBatch,
                   rope: dict, v_first: Optional[torch.Tensor], max_ctx: int):
        s, c, i = layer.spec.mixer, self.cache, self._cache_index[n]
        first = s.v_mix and v_first is None
        if first:
            v_first = torch.empty((b.T, s.kv_heads * s.vdim), dtype=raw.dtype, device=raw.device)
        q = k_rows = v_rows = None
        plan = self._plan(s)
        key_rows = b.kv_rows(plan)
        if key_rows:       # head sizes the kernel does not have are padded with zeros
            P = R.row_head(s.dim, s.vdim)
            new = torch.empty if s.dim == s.vdim == P else torch.zeros
            k_rows, v_rows = (new((key_rows, s.kv_heads, P), dtype=raw.dtype, device=raw.device)
                              for _ in range(2))
            q = new((b.T, s.heads, P), dtype=raw.dtype, device=raw.device)
        q = R.shortconv_attn(
            raw, layer.seg["k"], layer.seg["v"], layer.conv, self.state[n, "conv"], s.heads,
            s.kv_heads, s.dim, s.vdim, b, rope.get(layer.rope_key), c.k[i], c.v[i], c.page_table,
            v_first=v_first if s.v_mix else None, mix=layer.mix if s.v_mix and not first else None,
            write_first=first, k_rows=k_rows, v_rows=v_rows, q=q)
        R.ragged_attention(q, c.k[i], c.v[i], c.page_table, b, s.heads, s.kv_heads, s.dim, s.vdim,
                           s.scale, cat[:, :layer.out_dim], chunk=s.chunk, sink=layer.sink,
                           gate=raw[:, layer.seg["g"]:], max_ctx=max_ctx,
                           k_rows=k_rows, v_rows=v_rows, plan=plan)
        return v_first

    def _delta(self, n: int, layer, raw: torch.Tensor, cat: torch.Tensor, b: R.RaggedBatch) -> None:
        s, m, seg = layer.spec.mixer, self.m, layer.seg
        T = raw.shape[0]
        a = torch.empty((T, layer.w_a2.shape[0]), dtype=torch.float32, device=m.device)
        gate = torch.empty((T, layer.w_g2.shape[0]), dtype=m.dtype, device=m.device)
        a1, g1 = raw[:, seg["a1"]:], raw[:, seg["g1"]:]
        G.linear_pair((a1[:, :layer.w_a2.shape[1]], layer.w_a2, a, "none", None, False),
                      (g1[:, :layer.w_g2.shape[1]], layer.w_g2, gate, "none", None, False))
        qkvg = R.shortconv_delta(raw, seg["k"], seg["v"], seg["b"], layer.conv,
                                 self.state[n, "conv"], s.heads, s.kv_heads, s.dim, s.vdim, b, a,
                                 layer.A_log, layer.dt_bias)
        o = R.delta_scan(*qkvg, self.state[n, "delta"], b)
        R.gated_head_norm(o, gate, layer.head_norm, self.cfg.norm_eps, cat[:, :layer.out_dim])

    # the mixers of a sequential block fill ``out``, the columns in front of their output projection
    def _heads(self, n: int, layer, raw: torch.Tensor, out: torch.Tensor, b: R.RaggedBatch, rope: dict,
               max_ctx: int) -> None:
        s, c, i = layer.spec.mixer, self.cache, self._cache_index[n]
        eps, plan, kh = self.cfg.norm_eps, self._plan(s), s.kv_heads * s.maps
        own, rows = s.kv_from is None, _KvRows()
        if not own:
            rows = b.kept[s.kv_from]
        else:       # row-wise keys and values for the piece kernel, of this layer and those that use them too
            users = [plan] + [self._plan(self.cfg.layers[j].mixer) for j in self._shared.get(n, ())]
            size = max(b.kv_rows(p) for p in users)
            if size:        # heads at the distance that the piece kernel has
                q_head, v_head = R.row_heads(s.dim, s.vdim, s.maps)
                rows = _KvRows(*(torch.empty((size, h, p), dtype=raw.dtype, device=raw.device)
                                 for h, p in ((kh, q_head), (s.kv_heads, v_head))))
            if n in self._shared:
                b.kept[n] = rows
        pieces = b.kv_rows(plan)       # later rows of the buffers may hold nothing: they stay out of sight
        q = R.head_prep(raw, layer.seg.get("k", 0), layer.seg.get("v", 0), s.heads * s.maps, kh if own else 0,
                        s.dim, s.vdim, b, rope.get(layer.rope_key), c.k[i], c.v[i], c.page_table,
                        interleaved=s.interleaved, unit_eps=eps if s.unit_qk else None,
                        q_head=rows.k.shape[2] if pieces else None, k_rows=rows.k if own else None,
                        v_rows=rows.v if own else None, eps=eps, q_norm=layer.q_norm, k_norm=layer.k_norm,
                        unit_v=s.unit_v, q_factor=layer.temp)
        R.ragged_attention(
            q, c.k[i], c.v[i], c.page_table, b, s.heads, s.kv_heads, s.dim, s.vdim, s.scale,
            out[:, :layer.out_dim], window=s.window, keep=s.keep_first, softcap=s.softcap, score_max=s.score_max,
            maps=s.maps, map_weight=layer.map_weight, map_factor=1.0 - s.diff if s.maps == 2 else 1.0, eps=eps,
            sink=layer.sink, gate=raw[:, layer.seg["g"]:] if s.gated else None, gate_wide=True, max_ctx=max_ctx,
            k_rows=rows.k[:pieces] if pieces else None, v_rows=rows.v[:pieces] if pieces else None, plan=plan,
            gathered=rows.gathered == plan)
        if pieces:
            rows.gathered = plan

    def _experts(self, layer, h: torch.Tensor) -> dict:
        """The mixture of experts of ``h``, as what the next pass over the stream adds."""
        e, m = layer.experts, layer.experts.spec
        r = e.routing
        c = X.route(h, e.router, r, e.correction)
        shared = m.shared is not None
        if h.is_cuda and h.dtype == torch.bfloat16 and h.shape[0] <= X.FEW:
            return dict(y=X.experts_few(h, c, r, e.w_in, e.w_down, m.expert.limit, e.s_in, e.s_down,
                                        m.shared.limit if shared else 0.0, e.slope, e.shift))

        def rows(n, w):
            return torch.empty((n, w), dtype=h.dtype, device=h.device)
        s = X.sort_rows(h, c, r)
        n = s.rows.shape[0]
        act = X.grouped_linear(s.rows, e.w_in, s.block_expert, rows(n, e.w_in.shape[1] // 2),
                               glu=(e.slope, m.expert.limit, e.shift))
        res = X.grouped_linear(act, e.w_down, s.block_expert, rows(n, e.wp))
        add = dict(spread=R.Spread(res, s.slot, c.weight, h if m.identity else None))
        if shared:
            act = G.linear(h, e.s_in, rows(h.shape[0], e.s_in.shape[0] // 2),
                           glu=(e.slope, m.shared.limit, e.shift))
            add.update(y=self._product(act, e.s_down), y_weight=c.shared)
        return add

    def _latent(self, n: int, layer, raw: torch.Tensor, out: torch.Tensor, b: R.RaggedBatch,
                rope: dict, max_ctx: int) -> None:
        s, m, seg = layer.spec.mixer, self.m, layer.seg
        cache, table = self.cache.k[self._cache_index[n]], self.cache.page_table
        plan, H = self._plan(s), s.heads
        P, row_p = layer.w_kv.shape[2], cache.shape[-1]
        pieces = b.plans[plan][1]
        lat = None
        if pieces:
            lat = torch.empty((b.kv_rows(plan), row_p), dtype=raw.dtype, device=raw.device)
        q = L.latent_prep(raw, seg["dkv"], H, s.dim, s.rot_dim, s.kv_rank, layer.latent_norm,
                          self.cfg.norm_eps, rope[layer.rope_key], P, b, cache, table, rows_out=lat)
        gate = raw[:, seg["g"]:]
        if pieces:
            extra, where = b.plan(plan)[3], b.plan(plan)[5]
            if extra:
                L.gather_rows(cache, table, where, extra, lat[b.T:])
            kv = torch.empty((lat.shape[0], 2 * H * P), dtype=raw.dtype, device=raw.device)
            G.linear(lat, layer.w_kv.view(2 * H * P, row_p), kv)
            L.piece_attention(q, kv, b, plan, s.vdim, s.scale, gate, out)
        rows = b.rows if pieces or not b.n_big else b.every_row
        if rows.shape[0]:
            ql = torch.empty((rows.shape[0], H, row_p), dtype=raw.dtype, device=raw.device)
            L.linear_heads(q, layer.w_absorb, ql.view(-1, H * row_p), row_p, x_rows=rows)
            o = L.latent_attention(ql, cache, table, b, rows, s.kv_rank, s.rot_dim, s.scale, s.window,
                                   max_ctx)
            L.linear_heads(o, layer.w_value[:, :, :o.shape[2]], out, s.vdim, y_rows=rows, gate=gate)

    def _mamba2(self, n: int, layer, raw: torch.Tensor, out: torch.Tensor, b: R.RaggedBatch) -> None:
        s, seg = layer.spec.mixer, layer.seg
        u = RC.shortconv_act(raw, seg["x"], layer.conv, layer.conv_b, self.state[n, "conv"], b)
        y = torch.empty((b.T, _up8(s.out_dim)), dtype=raw.dtype, device=raw.device)
        RC.ssd_scan(u, layer.boff, layer.coff, raw[:, seg["dt"]:], layer.dt_bias, layer.A_log, layer.D,
                    self.state[n, "ssd"], s.groups, s.vdim, b, y)
        RC.gated_group_norm(y, raw[:, seg["z"]:], layer.out_norm, s.norm_groups, self.cfg.norm_eps,
                            out[:, :s.out_dim])

    def _mingru(self, n: int, layer, raw: torch.Tensor, out: torch.Tensor, b: R.RaggedBatch) -> None:
        seg = layer.seg
        RC.mingru_scan(raw, seg["z"], seg["x"], seg["g"], self.state[n, "gru"], b, out)

    def _product(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """``x @ w^T`` on its way into the residual stream: fp32 where that costs nothing or the
        contraction has to be cut to occupy the SMs, else in the working type."""
        M, N = x.shape[0], w.shape[0]
        if not x.is_cuda or x.dtype == torch.float32 or M <= G.SKINNY_MAX:
            return G.linear(x, w, torch.empty((M, N), dtype=torch.float32, device=x.device))
        if ((M + 127) // 128) * ((N + 127) // 128) <= 74:
            return G.linear(x, w, torch.zeros((M, N), dtype=torch.float32, device=x.device),
                            accumulate=True)
        return G.linear(x, w, torch.empty((M, N), dtype=x.dtype, device=x.device))

    def _forward(self, b: R.RaggedBatch, max_ctx: int, layer_out: Optional[list] = None
                 ) -> Optional[torch.Tensor]:
        """All layers over the batch; logits ``[wanted, vocab_padded]`` (fp32) of the wanted rows,
        None when there are none.  ``layer_out`` collects the residual stream after every layer."""
        m, cfg = self.m, self.cfg
        rope = {k: R.rope_table(b.pos, f) for k, f in m.inv_freq.items()}
        x = torch.empty((b.T, cfg.width_padded), dtype=torch.float32, device=m.device)
        R.embed_norm(b.tokens, m.embed, m.embed_norm, cfg.hidden_dim, cfg.norm_eps, x, cfg.embed_scale)
        blocks = self._parallel if cfg.design.parallel else self._sequential
        xf = blocks(x, b, rope, max_ctx, layer_out)
        if xf is None:
            return None
        logits = torch.empty((b.n_want, cfg.vocab_padded), dtype=torch.float32, device=m.device)
        return G.linear(xf, m.head, logits, softcap=cfg.logit_softcap)

    def _parallel(self, x: torch.Tensor, b: R.RaggedBatch, rope: dict, max_ctx: int,
                  layer_out: Optional[list]) -> Optional[torch.Tensor]:
        """Blocks whose mixer and feed-forward read the same stream."""
        m, W, eps = self.m, self.cfg.hidden_dim, self.cfg.norm_eps
        v_first = None
        for n, run in enumerate(self._runs):
            layer = m.layers[run.layer]
            h1, h2 = R.rms_rows(x, layer.norm1, W, eps, m.dtype, w2=layer.norm2)
            raw, cat = self._mixer_in(layer, h1, h2)
            if isinstance(layer.spec.mixer, AttentionSpec):
                v_first = self._attention(n, layer, raw, cat, b, rope, v_first, max_ctx)
            else:
                self._delta(n, layer, raw, cat, b)
            G.linear(cat, layer.w_out, x, accumulate=True)
            if layer_out is not None:
                layer_out.append(x[:, :W].clone())
        if not b.n_want:
            return None
        return R.rms_rows(x, m.final_gain, W, eps, m.dtype, rows=b.want)[0]

    def _sequential(self, x: torch.Tensor, b: R.RaggedBatch, rope: dict, max_ctx: int,
                    layer_out: Optional[list]) -> Optional[torch.Tensor]:
        """Blocks of one sublayer after the other, norms before and after each.  A sublayer's result
        stays pending (``add``) until the pass in front of the next one."""
        m, cfg = self.m, self.cfg
        W, wp, eps, dt = cfg.hidden_dim, cfg.width_padded, cfg.norm_eps, m.dtype
        add: dict = {}
        both = None
        if cfg.loop is not None:           # operand [x | x0] of the product in front of every pass
            both = torch.empty((b.T, 2 * wp), dtype=dt, device=m.device)
            R.add_norm(x, W, eps, dt, casts=[both[:, wp:]])
        for n, run in enumerate(self._runs):
            layer = m.layers[run.layer]
            if run.starts is not None:
                R.add_norm(x, W, eps, dt, casts=[both[:, :wp]], keep=False, **add)
                x, add = None, dict(y=self._product(both, m.loop_in), bias=m.loop_step[run.starts])
            back = {}                      # what the mixer reads of earlier tokens' h
            if layer.shift is not None or layer.taps is not None:
                back = dict(shift=layer.shift, taps=layer.taps, before=self.state[n, "before"], batch=b)
            x, h = R.add_norm(x, W, eps, dt, gain=layer.norm1, center=layer.center1, **back, **add)
            raw = torch.empty((b.T, layer.w_in.shape[0]), dtype=dt, device=m.device)
            G.linear(h, layer.w_in, raw, bias=layer.b_in)
            out = torch.empty((b.T, layer.act_off), dtype=dt, device=m.device)
            if layer.out_dim != layer.act_off:
                out[:, layer.out_dim:].zero_()
            if isinstance(layer.spec.mixer, (HeadAttentionSpec, LatentAttentionSpec)):
                mix = self._heads if isinstance(layer.spec.mixer, HeadAttentionSpec) else self._latent
                mix(n, layer, raw, out, b, rope, max_ctx)
            else:
                {"mamba2": self._mamba2, "mingru": self._mingru}[layer.spec.mixer.kind](n, layer, raw, out, b)
            add = dict(y=self._product(out, layer.w_out), post=layer.norm1b, scale=layer.scale1)
            if layer.norm2 is not None:
                x, h = R.add_norm(x, W, eps, dt, gain=layer.norm2, center=layer.center2, **add)
            if layer.experts is not None:
                add = dict(post=layer.norm2b, scale=layer.scale2, **self._experts(layer, h))
            elif layer.w_up is not None:
                act = torch.empty((b.T, layer.ff_padded), dtype=dt, device=m.device)
                G.linear(h, layer.w_up, act, epi=cfg.design.act, bias=layer.b_up, glu=layer.glu)
                add = dict(y=self._product(act, layer.w_down), bias=layer.b_down, post=layer.norm2b,
                           scale=layer.scale2)
            if layer_out is not None:
                x, add = R.add_norm(x, W, eps, dt, **add)[0], {}
                layer_out.append(x[:, :W].clone())
        if not b.n_want:
            return None
        return R.add_norm(x, W, eps, dt, gain=m.final_gain, center=m.final_center, rows=b.want, **add)[1]

    def step(self, entries: List[Entry], layer_out: Optional[list] = None
             ) -> Optional[torch.Tensor]:
        """Runs the entries as one batch and returns the logits of their wanted places, in order,
        ``[wanted, vocab_padded]`` fp32 (None when nothing is wanted).  Pages are reserved here;
        an entry's ``pos0`` must be the number of tokens its slot already holds."""
        c = self.cache
        seen = set()
        for e in entries:
            if e.slot in seen:
                raise ProcessingError.invalid_input(f"slot {e.slot} has two entries in one step")
            seen.add(e.slot)
            if e.pos0 != c.length(e.slot):
                raise ProcessingError.invalid_input(
                    f"slot {e.slot} holds {c.length(e.slot)} tokens, the entry starts at {e.pos0}")
            ids = np.asarray(e.tokens)
            if ids.min() < 0 or ids.max() >= self.cfg.vocab_size:
                raise ProcessingError.invalid_input(
                    f"token ids must lie in [0, {self.cfg.vocab_size})")
        for e in entries:
            c.reserve(e.slot, e.pos0 + len(e.tokens))
        if self.use_graph and layer_out is None and \
                all(len(e.tokens) == 1 and len(e.want) == 1 and e.pos0 > 0 for e in entries):
            out = self._decode_graph(entries)
        else:
            b = self._batch(entries)
            out = self._forward(b, b.max_ctx, layer_out)
        for e in entries:
            c.set_length(e.slot, e.pos0 + len(e.tokens))
        return out

    def _capture(self, entries: List[Entry]):
        """Graph of a step of ``len(entries)`` single tokens.  The warm-up and the capture run on
        the entries themselves: they write the same cache cells and would advance the recurrent
        state, which is put back."""
        n = len(entries)
        b = self._batch(entries)
        ctx = self.cache.page_table.shape[1] * PAGE
        idx = b.slot.long()
        keep = {k: t[idx].clone() for k, t in self.state.tensors.items()}
        side = torch.cuda.Stream(self.m.device)
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            self._forward(b, ctx)
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize(self.m.device)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            out = self._forward(b, ctx)
        for k, t in keep.items():
            self.state.tensors[k][idx] = t
        self._graphs[n] = (graph, b, out)
        return self._graphs[n]

    def _decode_graph(self, entries: List[Entry]) -> torch.Tensor:
        g = self._graphs.get(len(entries))
        if g is None:
            g = self._capture(entries)
        else:
            self._batch(entries, into=g[1])
            g[1].slots_host = [e.slot for e in entries]
        self._graph_pos = None
        g[0].replay()
        return g[2]

    # ------------------------------------------------------------------ generation interface
    def prefill(self, ids: torch.Tensor, total_len: int, seq_chunk: Optional[int] = None,
                token_chunk: Optional[int] = None) -> torch.Tensor:
        """Prompts ``ids [B, S]`` into slots ``0 .. B-1``; the last position's logits ``[B, V]``.
        ``seq_chunk`` sequences and ``token_chunk`` positions are taken at a time (any sizes)."""
        B, S = ids.shape
        if B > self.max_batch:
            raise ProcessingError.limit_exceeded("batch size", self.max_batch, B)
        c = self.cache
        need = (total_len + PAGE - 1) // PAGE
        if c is None or c.page_table.shape[0] < B or c.page_table.shape[1] < need:
            c = self.open_slots(B, total_len)
        for b in list(c.owned):
            c.release(b)
        for b in range(B):
            c.reserve(b, total_len)
        rows = ids.cpu().numpy()
        nb = max(1, min(B, int(seq_chunk or B)))
        step = max(1, min(S, int(token_chunk or S), max(1, self.prefill_tokens // nb)))
        out: List[torch.Tensor] = []
        for b0 in range(0, B, nb):
            group = range(b0, min(B, b0 + nb))
            for s0 in range(0, S, step):
                s1 = min(S, s0 + step)
                want = [s1 - s0 - 1] if s1 == S else []
                got = self.step([Entry(b, s0, rows[b][s0:s1], want) for b in group])
            out.append(got.clone())
        return torch.cat(out)

    def decode_step(self, tokens: torch.Tensor) -> torch.Tensor:
        """One token per sequence (``[B]`` int64) at the next position; ``[B, V]`` logits.  With a
        captured graph the tokens stay on the device and the positions advance there."""
        B = tokens.shape[0]
        c = self.cache
        pos = [c.length(b) for b in range(B)]
        g = self._graphs.get(B) if self.use_graph else None
        if g is not None and g[1].slots_host == list(range(B)) and \
                getattr(self, "_graph_pos", None) == (id(g[0]), pos):
            for b in range(B):
                c.reserve(b, pos[b] + 1)
            g[1].tokens.copy_(tokens)
            g[1].positions.add_(1)
            g[0].replay()
            out = g[2]
            for b in range(B):
                c.set_length(b, pos[b] + 1)
        else:
            out = self.step([Entry(b, pos[b], [t], [0]) for b, t in enumerate(tokens.tolist())])
            g = self._graphs.get(B) if self.use_graph else None
        self._graph_pos = (id(g[0]), [p + 1 for p in pos]) if g is not None else None
        return out

    # ------------------------------------------------------------------ slot interface (serving)
    def prefill_slot(self, slot: int, ids: torch.Tensor, total_len: int,
                     token_chunk: Optional[int] = None) -> torch.Tensor:
        c = self.cache
        c.reserve(slot, total_len)
        toks = ids.tolist()
        n = int(token_chunk or len(toks))
        for s0 in range(0, len(toks), n):
            part = toks[s0:s0 + n]
            last = s0 + n >= len(toks)
            got = self.step([Entry(slot, s0, part, [len(part) - 1] if last else [])])
        return got[0].clone()

    def decode_slots(self, slots: torch.Tensor, tokens: torch.Tensor, positions: torch.Tensor
                     ) -> torch.Tensor:
        return self.step([Entry(s, p, [t], [0]) for s, t, p in
                          zip(slots.tolist(), tokens.tolist(), positions.tolist())])

    def prefill_slot_paged(self, slot, ids, total_len, prefix_pages):
        raise ProcessingError.unsupported("a prompt on cached prefix pages",
                                          "the layers' state at that point is not in the pages")
