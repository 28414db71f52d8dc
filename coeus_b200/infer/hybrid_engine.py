"""Serving engine of the hybrid decoders (:mod:`coeus_b200.models.hybrid`).

One step function runs everything: a step brings entries, each the next tokens of one sequence
(a whole prompt, a portion of one, or a single decoded token), and they go through the layers as
one ragged batch.  Keys and values live in the paged cache, convolution inputs and recurrent
states in slots.  A step whose entries are single tokens is replayed from a CUDA graph.

The generation, slot and serving interfaces of :class:`coeus_b200.infer.engine.InferenceEngine`
are kept on top of it.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import numpy as np
import torch

from ..foundation.error import ProcessingError
from ..models.hybrid import AttentionSpec, HybridLM
from ..ops import gemm as G
from ..ops import ragged as R
from ..ops.decode import PAGE
from .engine import InferenceEngine
from .kv_cache import PagedKVCache, SequenceState

Entry = R.Entry


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


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
        mixers = [self.cfg.layers[l].mixer for l in self.cfg.attention_layers()]
        self._plans = [R.AttnPlan(a.chunk, self._pieces(a)) for a in mixers]

    def _pieces(self, a: AttentionSpec) -> bool:
        return self._tiles and R.pieces_allowed(a.dim, a.vdim, a.chunk, a.scale)

    def _batch(self, entries: List[Entry], into: Optional[R.RaggedBatch] = None) -> R.RaggedBatch:
        return R.RaggedBatch(entries, self.m.device, tile_rows=self._tiles, into=into,
                             plans=self._plans)

    # ------------------------------------------------------------------ cache and state
    def open_slots(self, max_seqs: int, max_len: int, num_pages: Optional[int] = None
                   ) -> PagedKVCache:
        """Cache and state for ``max_seqs`` sequences of up to ``max_len`` tokens.  ``num_pages``
        sizes the shared page pool (default: every slot can grow to ``max_len``)."""
        cfg, m = self.cfg, self.m
        per_seq = max(1, (max_len + PAGE - 1) // PAGE)
        dims = []
        self._cache_index: Dict[int, int] = {}
        for l in cfg.attention_layers():
            a = cfg.layers[l].mixer
            self._cache_index[l] = len(dims)
            dims.append((a.kv_heads, _up8(a.dim), _up8(a.vdim)))
        self.cache = PagedKVCache(len(dims), 0, 0, num_pages or max_seqs * per_seq, max_seqs,
                                  per_seq, m.device, m.dtype, layer_dims=dims)
        self.state = SequenceState(max_seqs, m.device)
        for l, layer in enumerate(m.layers):
            s = layer.spec.mixer
            self.state.add(l, "conv", (s.conv - 1, layer.channels), m.dtype)
            if not isinstance(s, AttentionSpec):
                self.state.add(l, "delta", (s.heads, s.dim, s.vdim), torch.float32)
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

    def _attention(self, l: int, layer, raw: torch.Tensor, cat: torch.Tensor, b: R.RaggedBatch,
                   rope: dict, v_first: Optional[torch.Tensor], max_ctx: int):
        s, c, i = layer.spec.mixer, self.cache, self._cache_index[l]
        first = s.v_mix and v_first is None
        if first:
            v_first = torch.empty((b.T, s.kv_heads * s.vdim), dtype=raw.dtype, device=raw.device)
        q = k_rows = v_rows = None
        plan = R.AttnPlan(s.chunk, self._pieces(s))
        n = b.kv_rows(plan)
        if n:       # head sizes the kernel does not have are padded with zeros
            P = R.row_head(s.dim, s.vdim)
            new = torch.empty if s.dim == s.vdim == P else torch.zeros
            k_rows, v_rows = (new((n, s.kv_heads, P), dtype=raw.dtype, device=raw.device)
                              for _ in range(2))
            q = new((b.T, s.heads, P), dtype=raw.dtype, device=raw.device)
        q = R.shortconv_attn(
            raw, layer.seg["k"], layer.seg["v"], layer.conv, self.state[l, "conv"], s.heads,
            s.kv_heads, s.dim, s.vdim, b, rope.get(layer.rope_key), c.k[i], c.v[i], c.page_table,
            v_first=v_first if s.v_mix else None, mix=layer.mix if s.v_mix and not first else None,
            write_first=first, k_rows=k_rows, v_rows=v_rows, q=q)
        R.ragged_attention(q, c.k[i], c.v[i], c.page_table, b, s.heads, s.kv_heads, s.dim, s.vdim,
                           s.scale, cat[:, :layer.out_dim], chunk=s.chunk, sink=layer.sink,
                           gate=raw[:, layer.seg["g"]:], max_ctx=max_ctx,
                           k_rows=k_rows, v_rows=v_rows, plan=plan)
        return v_first

    def _delta(self, l: int, layer, raw: torch.Tensor, cat: torch.Tensor, b: R.RaggedBatch) -> None:
        s, m, seg = layer.spec.mixer, self.m, layer.seg
        T = raw.shape[0]
        a = torch.empty((T, layer.w_a2.shape[0]), dtype=torch.float32, device=m.device)
        gate = torch.empty((T, layer.w_g2.shape[0]), dtype=m.dtype, device=m.device)
        a1, g1 = raw[:, seg["a1"]:], raw[:, seg["g1"]:]
        G.linear_pair((a1[:, :layer.w_a2.shape[1]], layer.w_a2, a, "none", None, False),
                      (g1[:, :layer.w_g2.shape[1]], layer.w_g2, gate, "none", None, False))
        qkvg = R.shortconv_delta(raw, seg["k"], seg["v"], seg["b"], layer.conv,
                                 self.state[l, "conv"], s.heads, s.kv_heads, s.dim, s.vdim, b, a,
                                 layer.A_log, layer.dt_bias)
        o = R.delta_scan(*qkvg, self.state[l, "delta"], b)
        R.gated_head_norm(o, gate, layer.head_norm, self.cfg.norm_eps, cat[:, :layer.out_dim])

    def _forward(self, b: R.RaggedBatch, max_ctx: int, layer_out: Optional[list] = None
                 ) -> Optional[torch.Tensor]:
        """All layers over the batch; logits ``[wanted, vocab_padded]`` (fp32) of the wanted rows,
        None when there are none.  ``layer_out`` collects the residual stream after every layer."""
        m, cfg = self.m, self.cfg
        W, eps = cfg.hidden_dim, cfg.norm_eps
        x = torch.empty((b.T, cfg.width_padded), dtype=torch.float32, device=m.device)
        R.embed_norm(b.tokens, m.embed, m.embed_norm, W, eps, x)
        rope = {k: R.rope_table(b.pos, f) for k, f in m.inv_freq.items()}
        v_first = None
        for l, layer in enumerate(m.layers):
            h1, h2 = R.rms_rows(x, layer.norm1, W, eps, m.dtype, w2=layer.norm2)
            raw, cat = self._mixer_in(layer, h1, h2)
            if isinstance(layer.spec.mixer, AttentionSpec):
                v_first = self._attention(l, layer, raw, cat, b, rope, v_first, max_ctx)
            else:
                self._delta(l, layer, raw, cat, b)
            G.linear(cat, layer.w_out, x, accumulate=True)
            if layer_out is not None:
                layer_out.append(x[:, :W].clone())
        if not b.n_want:
            return None
        xf, _ = R.rms_rows(x, m.final_norm, W, eps, m.dtype, rows=b.want)
        logits = torch.empty((b.n_want, cfg.vocab_padded), dtype=torch.float32, device=m.device)
        return G.linear(xf, m.head, logits, softcap=cfg.logit_softcap)

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
