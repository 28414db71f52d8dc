"""Checks of a decoder of mixed layers, whatever its design: the serving path (step, cache, state,
engine, scheduler) against the design's plain implementation, and what the checks of single mechanisms
share."""
import torch

from coeus_b200.infer.engine import make_engine
from coeus_b200.infer.scheduler import ContinuousBatcher
from coeus_b200.models import hybrid as H
from coeus_b200.ops import ragged as R
from coeus_b200.ops.decode import PAGE

_memo = {}


def rel(got, want):
    got, want = got.double().cpu(), want.double()
    return float((got - want).abs().max() / want.abs().max().clamp_min(1e-30))


def rnd(shape, seed, device, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(shape, generator=g).to(dtype).to(device)


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist()


class Bench:
    """One model on one device, its weights, its oracle (``forward(cfg, weights, ids)``: the logits of
    every position) and its tolerance."""

    def __init__(self, cfg, weights, forward, device, dtype, tol=None):
        self.cfg, self.w, self.forward = cfg, weights, forward
        self.device, self.dtype = torch.device(device), dtype
        self.lm = H.HybridLM(cfg, weights, device, dtype)
        self.tol = tol or (2e-5 if dtype == torch.float32 else 0.05)

    def oracle(self, ids):
        """The oracle's logits, kept between tests."""
        key = (self.cfg, self.forward, tuple(ids))
        if key not in _memo:
            _memo[key] = self.forward(self.cfg, self.w, list(ids))
        return _memo[key]

    def engine(self, slots=4, max_len=512, num_pages=None, **kw):
        eng = make_engine(self.lm, max_batch=slots, **kw)
        eng.open_slots(slots, max_len, num_pages=num_pages)
        return eng

    def close(self, got, want, tol=None):
        """Root-mean-square difference over the vocabulary, relative to the oracle's spread."""
        got = got[..., :self.cfg.vocab_size].double().cpu()
        err = (got - want).square().mean(-1).sqrt() / want.std()
        assert torch.isfinite(got).all()
        assert float(err.max()) < (tol or self.tol), (float(err.max()), int(err.argmax()))

    def whole(self, ids, eng=None):
        eng = eng or self.engine(1)
        return eng.step([R.Entry(0, 0, ids, range(len(ids)))]).clone()


def feed(eng, slot, ids, cuts):
    """Feeds ``ids`` in portions of the sizes ``cuts`` (repeated); all logits."""
    out, at, i = [], 0, 0
    while at < len(ids):
        n = min(cuts[i % len(cuts)], len(ids) - at)
        out.append(eng.step([R.Entry(slot, at, ids[at:at + n], range(n))]).clone())
        at, i = at + n, i + 1
    return torch.cat(out)


# ------------------------------------------------------------------------------- model checks
def check_whole_prompt(b):
    for n, s in ((1, 2), (2, 3), (7, 4), (140, 5)):
        ids = tokens(b.cfg, n, s)
        b.close(b.whole(ids), b.oracle(ids))


def check_token_by_token(b):
    ids = tokens(b.cfg, 140, 5)
    b.close(feed(b.engine(1), 0, ids, [1]), b.oracle(ids))


def check_portions(b):
    ids = tokens(b.cfg, 140, 5)
    want = b.oracle(ids)
    for cuts in ([2], [3, 2], [63, 2, 1], [64], [17, 5, 31]):
        b.close(feed(b.engine(1), 0, ids, cuts), want)


def check_mixed_batches(b):
    """Four unequal requests advance together, portions beside single tokens, one of them left out
    of some steps; each gets what it gets alone."""
    seqs = [tokens(b.cfg, n, 5 if n == 140 else n) for n in (140, 33, 90, 5)]
    want = [b.oracle(s) for s in seqs]
    eng, at = b.engine(4), [0] * 4
    plan = [(40, 3, 1, 2), (0, 1, 64, 1), (1, 1, 1, 1), (2, 0, 3, 0), (30, 28, 0, 1), (1, 1, 21, 1)]
    k = 0
    while any(a < len(s) for a, s in zip(at, seqs)):
        takes = plan[k] if k < len(plan) else (7, 1, 1, 1)
        k += 1
        entries = []
        for i, n in enumerate(takes):
            part = seqs[i][at[i]:at[i] + n]
            if part:
                entries.append((i, R.Entry(i, at[i], part, range(len(part)))))
        if not entries:
            continue
        out, r = eng.step([e for _, e in entries]), 0
        for i, e in entries:
            n = len(e.tokens)
            b.close(out[r:r + n], want[i][at[i]:at[i] + n])
            r, at[i] = r + n, at[i] + n


def check_reuse(b):
    """A pool of few pages and two slots: requests come and go, every page and slot changes hands,
    in another order each time."""
    eng = b.engine(2, max_len=192, num_pages=5)
    seqs = [tokens(b.cfg, n, s) for n, s in ((140, 5), (33, 33), (70, 8), (140, 5), (90, 90), (1, 2))]
    waiting, live, used = list(range(len(seqs))), {}, set()
    free = [0, 1]
    while waiting or live:
        while waiting and free and (len(eng.cache.free) >= -(-len(seqs[waiting[0]]) // PAGE)):
            i = waiting.pop(0)
            slot = free.pop()
            eng.cache.reserve(slot, len(seqs[i]))
            used |= set(eng.cache.owned[slot])
            live[i] = slot
        entries = []
        for i, slot in live.items():
            at = eng.cache.length(slot)
            entries.append((i, R.Entry(slot, at, seqs[i][at:at + 29 + 7 * i],
                                       [len(seqs[i][at:at + 29 + 7 * i]) - 1])))
        out = eng.step([e for _, e in entries]).clone()
        for r, (i, e) in enumerate(entries):
            end = e.pos0 + len(e.tokens)
            b.close(out[r], b.oracle(seqs[i])[end - 1])
            if end == len(seqs[i]):
                eng.release_slot(live[i])
                free.append(live.pop(i))
    assert len(used) == 5 and eng.cache.pages_in_use() == 0


def check_long_decode(b):
    ids = tokens(b.cfg, 330, 9)
    want = b.oracle(ids)
    eng = b.engine(3)
    first = eng.step([R.Entry(1, 0, ids[:10], range(10))])
    b.close(first, want[:10])
    got = torch.cat([eng.step([R.Entry(1, p, [ids[p]], [0])]).clone() for p in range(10, 330)])
    b.close(got, want[10:])


def agrees(b, prompt, got):
    """Greedy tokens: each is the oracle's arg-max after the tokens before it, up to the error the
    logits may have."""
    z = b.forward(b.cfg, b.w, list(prompt) + list(got))
    for i, t in enumerate(got):
        row = z[len(prompt) - 1 + i]
        assert float(row.max() - row[t]) <= 3 * b.tol * float(z.std()), (i, t)


def check_generate(b):
    prompts = torch.tensor([tokens(b.cfg, 21, 11), tokens(b.cfg, 21, 12)], device=b.device)
    eng = make_engine(b.lm, max_batch=2)
    out = eng.generate(prompts, 12)
    for row, p in zip(out.tolist(), prompts.tolist()):
        assert row[:21] == p
        agrees(b, p, row[21:])
    again = eng.generate(prompts, 12, token_chunk=5, seq_chunk=1)     # other cuts, used slots
    for row, p in zip(again.tolist(), prompts.tolist()):
        agrees(b, p, row[21:])


def check_batcher(b):
    """More requests than slots through the scheduler, prompts read in portions beside decoding."""
    cb = ContinuousBatcher(make_engine(b.lm, max_batch=3), max_seqs=3, max_len=128, token_chunk=9,
                           step_tokens=16)
    reqs = [(tokens(b.cfg, n, 20 + n), k) for n, k in ((5, 7), (40, 3), (1, 9), (23, 1), (17, 6))]
    ids = {cb.submit(p, k): (p, k) for p, k in reqs}
    out = cb.run()
    for rid, (p, k) in ids.items():
        assert len(out[rid]) == k
        agrees(b, p, out[rid])
    assert cb.engine.cache.pages_in_use() == 0 and cb.stats["prefills"] == len(reqs)


MODEL_CHECKS = [check_whole_prompt, check_token_by_token, check_portions, check_mixed_batches,
                check_reuse, check_long_decode, check_generate, check_batcher]


# ----------------------------------------------------------------------- one mixer on its own
CUTS = (((1, 40), (2, 1), (1, 1), (70, 2), (127, 1), (9, 165)), ((3, 130), (5, 6), (202, 74)))


def single_mixer(spec, architecture, device, dtype, seed, **kw):
    """A model of one layer with this mixer alone, and the mixer's weights."""
    cfg = H.HybridConfig(16, 16, (H.LayerSpec(spec, None),), 1e-4, architecture=architecture, **kw)
    w = H.random_state(cfg, seed, dtype=torch.float32)
    w = {n: t.bfloat16().float() for n, t in w.items()}
    lm = H.HybridLM(cfg, w, device, dtype)
    return lm, {n[7:]: t.double() for n, t in w.items() if n.startswith("l0.mix.")}


def drive(lm, raws, cuts, run):
    """Two sequences through ``run(engine, layer, raw, out, batch, rope)``, cut at several places, in slots
    whose state holds something else; the mixer's outputs of each."""
    eng = lm.make_engine(max_batch=3)
    eng.open_slots(3, 512)
    for t in eng.state.tensors.values():
        t.fill_(9.0)
    layer, outs, at = lm.layers[0], [[], []], [0, 0]
    for s in (1, 2, 0, 2, 1):         # pages in an order that is not ascending
        eng.cache.reserve(s, min(eng.cache.page_table.shape[1], len(eng.cache.owned.get(s, [])) + 3) * PAGE)
    for s, raw in ((2, raws[0]), (0, raws[1])):
        eng.cache.reserve(s, raw.shape[0])
    for cut in cuts:
        b = eng._batch([R.Entry(slot, at[s], [0] * cut[s]) for s, slot in ((0, 2), (1, 0))])
        raw = torch.cat([raws[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
        out = torch.full((b.T, layer.act_off), 5.0, dtype=lm.dtype, device=lm.device)
        rope = {k: R.rope_table(b.pos, f) for k, f in lm.inv_freq.items()}
        run(eng, layer, raw, out, b, rope)
        outs[0].append(out[:cut[0]])
        outs[1].append(out[cut[0]:])
        at = [at[0] + cut[0], at[1] + cut[1]]
    return [torch.cat(o)[:, :layer.out_dim] for o in outs], eng
