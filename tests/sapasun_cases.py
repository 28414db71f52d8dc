"""Small Sapasun configurations, weights and checks shared by the CPU and the GPU tests.  The
oracle is :mod:`plain_sapasun`; the configurations are chosen so that sizes differ from one
another (heads, key and value widths, taps, chunks, ranks), with and without each option."""
import torch

import hybrid_checks
import plain_sapasun as plain
from hybrid_checks import MODEL_CHECKS, agrees, rel, rnd, tokens  # noqa: F401
from coeus_b200.models import hybrid as H
from coeus_b200.ops import gemm as G
from coeus_b200.ops import ragged as R
from coeus_b200.ops.decode import PAGE

A, D, M, L = H.AttentionSpec, H.ChannelDeltaSpec, H.MlpSpec, H.LayerSpec


def config(kind):
    if kind == "odd":         # nothing is a multiple of eight
        return H.HybridConfig(
            vocab_size=83, hidden_dim=44, norm_eps=2e-5, logit_softcap=9.0, layers=(
                L(D(6, 3, 10, 7, 2, 5, 3), M(50)),
                L(A(6, 3, 12, 5, 5, 0.4, 9, 6, 300.0, False), None),
                L(A(2, 1, 10, 6, 2, 0.3, 31, 10, 5000.0, True), M(21)),
                L(D(2, 2, 5, 9, 1, 4, 6), None),
                L(A(4, 1, 14, 6, 1, 0.2, 70, 4, 70.0, True), M(36)),
            ))
    if kind == "wide":        # vectorised paths, several pages per chunk, groups of 1, 3 and 8
        return H.HybridConfig(
            vocab_size=264, hidden_dim=96, norm_eps=1e-6, logit_softcap=20.0, layers=(
                L(A(8, 1, 80, 40, 4, 0.11, 150, 48, 1e4, True), M(128)),
                L(A(3, 1, 128, 40, 2, 0.09, 77, 64, 1e5, True), M(64)),
                L(D(4, 2, 72, 40, 3, 16, 8), M(64)),
                L(A(2, 2, 24, 136, 3, 0.2, 64, 16, 50.0, False), M(72)),
                L(D(1, 1, 130, 16, 4, 8, 24), M(40)),
            ))
    if kind == "square":      # key and value heads of one size: prompts in pieces
        return H.HybridConfig(
            vocab_size=120, hidden_dim=72, norm_eps=1e-5, logit_softcap=15.0, layers=(
                L(A(4, 2, 64, 64, 4, 0.15, 96, 32, 1e4, True), M(96)),
                L(D(2, 1, 32, 48, 4, 8, 8), M(40)),
                L(A(2, 2, 64, 64, 3, 0.12, 64, 64, 1e3, True), M(96)),
                L(A(1, 1, 128, 128, 2, 0.1, None, 128, 1e5, False), None),
            ))
    if kind == "delta":       # recurrence only
        return H.HybridConfig(
            vocab_size=40, hidden_dim=24, norm_eps=1e-5, logit_softcap=5.0, layers=(
                L(D(3, 1, 16, 8, 3, 4, 4), M(24)), L(D(2, 2, 8, 12, 2, 3, 5), M(16))))
    return H.HybridConfig(    # "attn": attention only, without rotation, mask or cap
        vocab_size=40, hidden_dim=32, norm_eps=1e-5, logit_softcap=None, layers=(
            L(A(4, 2, 8, 8, 3, 0.35, None, 0, 1.0, True), M(24)),
            L(A(6, 2, 6, 8, 2, 0.5, 16, 2, 10.0, True), M(24))))


def weights(cfg, seed=0):
    """Random weights under which old tokens matter: peaked attention, slow decay, sinks of some
    weight, mixing far from 0 and 1."""
    w = H.random_state(cfg, seed, dtype=torch.float32)
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}.mix."
        if isinstance(layer.mixer, A):
            w[p + "q"] *= 2.5
            if p + "vmix" in w:
                w[p + "vmix"] = torch.tensor(0.35 + 0.1 * i)
            w[p + "sink"] += 1.0
        else:
            w[p + "dt_bias"] -= 3.0
    return {n: t.bfloat16() for n, t in w.items()}


def plain_config(cfg):
    d = H.config_to_json(cfg)
    for layer in d["layers"]:
        if layer["type"] == "attention":
            layer["mixer"].setdefault("mask", {"size": 1 << 30})
            layer["mixer"].setdefault("rot", {"dims": 0, "base": 1.0})
    if d["logit_softcap"] is None:
        d["logit_softcap"] = 1e9
    return d


_made = {}


def make_weights(cfg, seed=1):
    if (cfg, seed) not in _made:
        _made[cfg, seed] = weights(cfg, seed)
    return _made[cfg, seed]


def forward(cfg, w, ids):
    return plain.forward(plain_config(cfg), w, ids)


def Bench(kind, device, dtype):
    cfg = config(kind)
    return hybrid_checks.Bench(cfg, make_weights(cfg), forward, device, dtype)


# --------------------------------------------------------------------------- mechanism checks
def batch_of(entries, device, tiles, chunk=None):
    return R.RaggedBatch([R.Entry(s, p, [0] * n) for s, p, n in entries], device, tile_rows=tiles,
                         plans=[R.AttnPlan(chunk, x) for x in (False, True)])


def check_norms(device, dtype, tol):
    x = rnd((5, 56), 1, device)
    x[:, 50:] = 0
    w1, w2 = (torch.nn.functional.pad(1 + rnd((50,), s, device), (0, 6)) for s in (2, 3))
    y1, y2 = R.rms_rows(x, w1, 50, 3e-4, dtype, w2=w2)
    xd = x[:, :50].cpu().double()
    for y, w in ((y1, w1), (y2, w2)):
        assert rel(y[:, :50], plain.rms_norm(xd, w[:50].cpu().double(), 3e-4)) < tol
        assert float(y[:, 50:].abs().max()) == 0
    rows = torch.tensor([4, 0, 2], dtype=torch.int32, device=device)
    y, _ = R.rms_rows(x, w1, 50, 3e-4, dtype, rows=rows)
    assert rel(y[:, :50], plain.rms_norm(xd[[4, 0, 2]], w1[:50].cpu().double(), 3e-4)) < tol
    emb = torch.nn.functional.pad(rnd((9, 50), 4, device, dtype), (0, 6))
    tok = torch.tensor([8, 0, 3], dtype=torch.int32, device=device)
    out = torch.full((3, 56), 7.0, device=device)
    R.embed_norm(tok, emb, w1, 50, 1e-5, out)
    e = emb[[8, 0, 3], :50].cpu().double()
    assert rel(out[:, :50], plain.rms_norm(e, w1[:50].cpu().double(), 1e-5)) < 1e-5
    assert float(out[:, 50:].abs().max()) == 0


def check_linear(device, dtype, tol):
    for M_, N_, K_ in ((1, 8, 24), (3, 40, 8), (17, 136, 72), (70, 200, 136), (300, 520, 264)):
        x, w = rnd((M_, K_), 1, device, dtype), rnd((N_, K_), 2, device, dtype)
        z = x.cpu().double() @ w.cpu().double().T
        y = torch.empty((M_, N_), dtype=dtype, device=device)
        assert rel(G.linear(x, w, y), z) < tol
        assert rel(G.linear(x, w, y, epi="relu2"), torch.relu(z).square()) < tol
        f = rnd((M_, N_), 3, device)
        start = f.cpu().double()
        assert rel(G.linear(x, w, f, accumulate=True), start + z) < tol
        assert rel(G.linear(x, w, torch.empty_like(f), softcap=4.0), plain.soft_cap(z, 4.0)) < tol


def check_attention_inputs(device, dtype, tol):
    """Convolution, rotation, value mixing and cache writes against the plain functions, one
    sequence cut at several places, in two slots at once."""
    for (H_, Gk, d, dv, taps, half, seed) in ((4, 2, 16, 8, 4, 8, 1), (3, 1, 10, 7, 2, 3, 2),
                                              (2, 2, 24, 16, 1, 0, 3), (5, 1, 8, 12, 6, 4, 4)):
        qc, kc, vc = H_ * d, Gk * d, Gk * dv
        koff = (qc + 7) // 8 * 8
        voff = koff + (kc + 7) // 8 * 8
        ld = voff + (vc + 7) // 8 * 8
        T = 75
        raws = [rnd((T, ld), seed * 10 + s, device, dtype) for s in (0, 1)]
        wt = rnd((taps, qc + kc + vc), seed + 50, device)
        f = torch.tensor([300.0 ** (-2.0 * i / max(1, 2 * half)) for i in range(half)], device=device)
        pages, table = 9, torch.tensor([[3, 1, 0], [7, 2, 8], [5, 4, 6]], dtype=torch.int32)
        table = table.to(device)
        kcache = torch.zeros((pages, PAGE, Gk, (d + 7) // 8 * 8), dtype=dtype, device=device)
        vcache = torch.zeros((pages, PAGE, Gk, (dv + 7) // 8 * 8), dtype=dtype, device=device)
        state = torch.full((3, taps - 1, qc + kc + vc), 9.0, dtype=dtype, device=device)
        firsts = [rnd((T, vc), seed + 60 + s, device, dtype) for s in (0, 1)]
        mix = torch.tensor([0.3], device=device)
        qs = [[], []]
        at = [0, 0]
        for cut in ((1, 40), (2, 1), (1, 1), (30, 2), (40, 1), (1, 30)):
            b = batch_of([(2, at[0], cut[0]), (0, at[1], cut[1])], device, False)
            raw = torch.cat([raws[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
            vf = torch.cat([firsts[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
            rope = R.rope_table(b.pos, f) if half else None
            q = R.shortconv_attn(raw, koff, voff, wt, state, H_, Gk, d, dv, b, rope, kcache, vcache,
                                 table, v_first=vf, mix=mix)
            qs[0].append(q[:cut[0]])
            qs[1].append(q[cut[0]:])
            at = [at[0] + cut[0], at[1] + cut[1]]
        for s, slot in ((0, 2), (1, 0)):
            raw = raws[s].cpu().double()
            w = wt.cpu().double().T
            u = torch.cat([raw[:, :qc], raw[:, koff:koff + kc], raw[:, voff:voff + vc]], 1)
            y = plain.causal_conv(u, w)
            want_q = plain.rotate_half(y[:, :qc].view(T, H_, d), 2 * half, 300.0) if half \
                else y[:, :qc].view(T, H_, d)
            want_k = y[:, qc:qc + kc].view(T, Gk, d)
            want_k = plain.rotate_half(want_k, 2 * half, 300.0) if half else want_k
            want_v = 0.7 * y[:, qc + kc:] + 0.3 * firsts[s].cpu().double()
            assert rel(torch.cat(qs[s]), want_q) < tol
            got_k = kcache[table[slot].long()].reshape(-1, Gk, kcache.shape[-1])[:T, :, :d]
            got_v = vcache[table[slot].long()].reshape(-1, Gk, vcache.shape[-1])[:T, :, :dv]
            assert rel(got_k, want_k) < tol
            assert rel(got_v, want_v.view(T, Gk, dv)) < tol
            if taps > 1:
                assert torch.equal(state[slot].cpu().double(), u[-(taps - 1):])
        # keeping v as the later layers' v_first
        b = batch_of([(1, 0, 5)], device, False)
        vf = torch.zeros((5, vc), dtype=dtype, device=device)
        R.shortconv_attn(raws[0][:5], koff, voff, wt, state, H_, Gk, d, dv, b,
                         R.rope_table(b.pos, f) if half else None, kcache, vcache, table, v_first=vf,
                         write_first=True)
        raw = raws[0][:5, voff:voff + vc].cpu().double()
        assert rel(vf, plain.causal_conv(raw, wt[:, qc + kc:].cpu().double().T)) < tol


def check_attention(device, dtype, tol):
    """Rows at the edges of pages and chunks, with one key that stands out placed far away, just
    inside and just outside; sinks from none to dominating; several group sizes and widths."""
    g = torch.Generator().manual_seed(0)
    for H_, Gk, d, dv, chunk in ((5, 1, 64, 40, 110), (6, 2, 40, 24, 50), (2, 2, 10, 7, 9),
                                 (9, 1, 72, 128, 200), (3, 3, 136, 200, 64), (4, 4, 128, 64, None),
                                 (2, 1, 16, 16, 1), (20, 1, 24, 32, 90), (4, 2, 64, 64, 100),
                                 (2, 1, 128, 128, 64), (3, 1, 64, 64, None), (2, 2, 128, 128, 300)):
        n = 260
        k = torch.randn((n, Gk, d), generator=g).to(dtype)
        v = torch.randn((n, Gk, dv), generator=g).to(dtype)
        table = torch.randperm(7, generator=g)[:5].int()[None].to(device)
        dp, dvp = (d + 7) // 8 * 8, (dv + 7) // 8 * 8
        kc = torch.zeros((7, PAGE, Gk, dp), dtype=dtype)
        vc = torch.zeros((7, PAGE, Gk, dvp), dtype=dtype)
        for t in range(n):
            page = int(table[0, t // PAGE])
            kc[page, t % PAGE, :, :d], vc[page, t % PAGE, :, :dv] = k[t], v[t]
        kc, vc = kc.to(device), vc.to(device)
        size = chunk or 1 << 30
        scale = 0.7 / d ** 0.5
        sink = torch.linspace(-3.0, 4.0, H_)
        span = [p for c in (chunk or 64, 64) for e in range(c, n, c) for p in (e - 1, e, e + 1)]
        pos = sorted({0, 1, n - 1, *[p for p in span if p < n]})[:40]
        rows_too = dtype == torch.bfloat16 and R.pieces_allowed(d, dv, chunk, scale)
        for start, m in [(p, 1) for p in pos] + [(0, 70), (0, 260), (50, 100), (117, 66), (n - 6, 6)]:
            m = min(m, n - start)
            q = torch.randn((m, H_, d), generator=g)
            # each row points at one key: its chunk's first, the one before it, itself, or a far one
            for r in range(m):
                i = start + r
                lo = i // size * size
                j = [lo, max(lo - 1, 0), i, (i * 7) % (i + 1)][r % 4 if m > 1 else i % 4]
                q[r] += 3.0 * k[j].double().repeat_interleave(H_ // Gk, 0)
            q = q.to(dtype)
            gate = torch.randn((m, H_ + 3), generator=g).to(dtype)
            b = batch_of([(0, start, m)], device, dtype == torch.bfloat16, chunk)
            out = torch.full((m, H_ * dv + 8), 5.0, dtype=dtype, device=device)
            args = (q.to(device), kc, vc, table, b, H_, Gk, d, dv, scale,
                    out[:, :H_ * dv])
            kw = dict(chunk=chunk, sink=sink.to(device), gate=gate.to(device)[:, 2:])
            R.ragged_attention(*args, **kw)
            want = torch.zeros(m, H_, dv, dtype=torch.float64)
            for r in range(m):
                i = start + r
                js = [j for j in range(i + 1) if plain.chunk_visible(i, j, size)]
                for h in range(H_):
                    s = (k[js, h // (H_ // Gk)].double() @ q[r, h].double()) * scale
                    want[r, h] = plain.sink_softmax(s, sink[h].double()) @ v[js, h // (H_ // Gk)].double()
            want *= torch.sigmoid(gate[:, 2:2 + H_].double())[:, :, None]
            assert rel(out[:, :H_ * dv], want.reshape(m, -1)) < tol, (H_, d, chunk, start, m)
            if rows_too:       # the same with this step's keys and values at hand, row by row
                out.fill_(5.0)
                P, rows = R.row_head(d, dv), b.kv_rows(R.AttnPlan(chunk, True))
                kr, vr = (torch.zeros((max(rows, 1), Gk, P), dtype=dtype, device=device)
                          for _ in range(2))
                qp = torch.zeros((m, H_, P), dtype=dtype, device=device)
                if rows:
                    kr[:m, :, :d], vr[:m, :, :dv] = k[start:start + m], v[start:start + m]
                qp[:, :, :d] = q
                R.ragged_attention(qp, *args[1:], **kw, k_rows=kr, v_rows=vr,
                                   plan=R.AttnPlan(chunk, True))
                assert rel(out[:, :H_ * dv], want.reshape(m, -1)) < tol, (H_, d, chunk, start, m)
            assert float((out[:, H_ * dv:].float() - 5.0).abs().max()) == 0


def check_delta(device, dtype, tol):
    """Inputs of the recurrence, the recurrence and the gated norm, cut at several places."""
    for H_, Gk, d, dv, taps, seed in ((4, 2, 16, 24, 3, 1), (3, 1, 10, 7, 1, 2), (2, 2, 70, 40, 4, 3),
                                      (1, 1, 130, 9, 2, 4), (2, 1, 200, 33, 2, 5)):
        qc, vc = Gk * d, H_ * dv
        koff = (qc + 7) // 8 * 8
        voff = koff + koff
        boff = voff + (vc + 7) // 8 * 8
        ld = boff + 8
        T = 60
        raws = [rnd((T, ld), seed * 10 + s, device, dtype) for s in (0, 1)]
        avs = [rnd((T, H_ * d), seed * 10 + 5 + s, device) for s in (0, 1)]
        wt = rnd((taps, 2 * qc + vc), seed + 50, device)
        A_log, dt = rnd((H_,), seed + 51, device), rnd((H_ * d,), seed + 52, device) - 2.0
        nw = 1 + rnd((dv,), seed + 53, device)
        conv = torch.full((3, taps - 1, 2 * qc + vc), 9.0, dtype=dtype, device=device)
        state = torch.full((3, H_, d, dv), 9.0, device=device)
        gates = [rnd((T, H_ * dv), seed + 54 + s, device, dtype) for s in (0, 1)]
        outs, at = [[], []], [0, 0]
        for cut in ((1, 20), (2, 1), (1, 1), (16, 2), (39, 1), (1, 35)):
            b = batch_of([(2, at[0], cut[0]), (0, at[1], cut[1])], device, False)
            raw = torch.cat([raws[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
            a = torch.cat([avs[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
            gt = torch.cat([gates[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
            x = R.shortconv_delta(raw, koff, voff, boff, wt, conv, H_, Gk, d, dv, b, a, A_log, dt)
            o = R.delta_scan(*x, state, b)
            y = torch.zeros((sum(cut), H_ * dv), dtype=dtype, device=device)
            R.gated_head_norm(o, gt, nw, 1e-4, y)
            outs[0].append((o[:cut[0]], y[:cut[0]]))
            outs[1].append((o[cut[0]:], y[cut[0]:]))
            at = [at[0] + cut[0], at[1] + cut[1]]
        for s, slot in ((0, 2), (1, 0)):
            raw = raws[s].cpu().double()
            u = torch.cat([raw[:, :qc], raw[:, koff:koff + qc], raw[:, voff:voff + vc]], 1)
            y = plain.silu(plain.causal_conv(u, wt.cpu().double().T))
            q = plain.unit(y[:, :qc].view(T, Gk, d)) * d ** -0.5
            k = plain.unit(y[:, qc:2 * qc].view(T, Gk, d))
            v = y[:, 2 * qc:].view(T, H_, dv)
            beta = torch.sigmoid(raw[:, boff:boff + H_])
            g = plain.channel_decay(avs[s].cpu().double().view(T, H_, d), A_log.cpu().double(),
                                    dt.cpu().double())
            per = H_ // Gk
            want = torch.empty(T, H_, dv, dtype=torch.float64)
            for h in range(H_):
                want[:, h], S = plain.delta_scan(q[:, h // per], k[:, h // per], v[:, h], g[:, h],
                                                 beta[:, h])
                assert rel(state[slot, h], S) < 5e-5
            assert rel(torch.cat([o for o, _ in outs[s]]), want) < 5e-5
            n = plain.rms_norm(want, nw.cpu().double(), 1e-4) * \
                torch.sigmoid(gates[s].cpu().double()).view(T, H_, dv)
            assert rel(torch.cat([y for _, y in outs[s]]), n.reshape(T, -1)) < tol
            if taps > 1:
                assert torch.equal(conv[slot].cpu().double(), u[-(taps - 1):])


MECHANISM_CHECKS = [check_norms, check_linear, check_attention_inputs, check_attention, check_delta]
