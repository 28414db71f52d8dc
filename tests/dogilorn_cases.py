"""Small Dogilorn configurations, weights and checks shared by the CPU and the GPU tests.  The oracle is
:mod:`plain_dogilorn`; the configurations are chosen so that sizes differ from one another (heads, key and
value widths, rotated parts, windows, kept positions, taps, experts, groups), with and without each option."""
import math

import torch

import hybrid_checks
import plain_dogilorn as plain
from coeus_b200.models import hybrid as H
from coeus_b200.ops import experts as X
from coeus_b200.ops import gemm as G
from coeus_b200.ops import ragged as R
from hybrid_checks import MODEL_CHECKS, agrees, drive, rel, rnd, single_mixer, tokens  # noqa: F401

L, M, E, Moe = H.LayerSpec, H.GluMlpSpec, H.GluSpec, H.SoftmaxMoeSpec


def A(heads, kv_heads, dim, vdim, scale, rot, base, window=None, keep=0, kv_from=None):
    return H.KeptWindowAttentionSpec(heads, kv_heads, dim, vdim, scale, rot, base, window, keep_first=keep,
                                     kv_from=kv_from)


def moe(experts, top, ff, groups=1, keep=1, shared=None, identity=0):
    return Moe(experts, top, E(ff), groups=groups, keep=keep, shared=E(shared) if shared else None,
               identity=identity)


def config(kind):
    def make(vocab, width, eps, scale, taps, *layers):
        return H.HybridConfig(vocab, width, layers, eps, architecture="Dogilorn", embed_scale=scale, conv_taps=taps)
    if kind == "odd":         # nothing is a multiple of eight
        return make(83, 44, 2e-5, 0.7, 3,
                    L(A(6, 3, 10, 14, 0.9, 6, 300.0, 9, 2), moe(6, 3, 13, 3, 2, 21, 3)),
                    L(A(5, 1, 14, 6, 0.7, 10, 1e4, 70, 5), M(50, 0.8)),
                    L(A(6, 3, 10, 14, 0.6, 6, 300.0, 21, 1, kv_from=0), None),
                    L(A(2, 2, 6, 11, 1.1, 0, 1.0, 33), moe(5, 2, 9)),
                    L(A(5, 1, 14, 6, 0.8, 10, 1e4, 9, 3, kv_from=1), M(21, 2.5)))
    if kind == "wide":        # vectorised paths, windows over pages, more than 16 queries on a key
        return make(264, 96, 1e-6, 3.0, 4,
                    L(A(8, 2, 64, 128, 0.4, 32, 1e4, 64, 4), M(128, 1.5)),
                    L(A(4, 2, 128, 96, 0.3, 128, 1e5, 150, 70), moe(12, 4, 40, 4, 2, 72, 4)),
                    L(A(4, 2, 128, 96, 0.25, 128, 1e5, 65, 8, kv_from=1), moe(10, 1, 24, 2, 1, None, 2)),
                    L(A(20, 1, 40, 64, 0.5, 24, 100.0, 100, 1), None),
                    L(A(8, 2, 64, 128, 0.5, 32, 1e4, None, kv_from=0), M(72, 0.6)))
    return make(60, 40, 1e-5, 12.5, 1,        # "large": heads that only the general kernels take, narrow windows
                L(A(2, 1, 136, 200, 0.2, 64, 1e4), None),
                L(A(3, 3, 160, 24, 0.15, 160, 1e3, 33, 66), moe(4, 2, 24, 2, 2, 8)),
                L(A(2, 1, 136, 200, 0.25, 64, 1e4, 1, 1, kv_from=0), M(24, 1.0)),
                L(A(2, 1, 24, 136, 0.5, 2, 5.0, 1), moe(3, 2, 8, 1, 1, 24, 1)),
                L(A(2, 1, 8, 8, 1.2, 8, 10.0, 130, 64), M(8, 0.3)))


def sure(z, correction, m, margin=0.01):
    """Whether the choice of experts by the logits ``z`` holds when the scores change a little."""
    c = (torch.softmax(z, -1) + correction).tolist()
    n = m.outputs // m.groups
    value = [max(c[g * n:(g + 1) * n]) for g in range(m.groups)]
    order = sorted(value, reverse=True)
    if m.keep < m.groups and order[m.keep - 1] - order[m.keep] < margin:
        return False
    left = sorted((x for e, x in enumerate(c) if value[e // n] >= order[m.keep - 1]), reverse=True)
    return m.top == len(left) or left[m.top - 1] - left[m.top] > margin


def levels(m, correction, g, scales=(1.0,), margin=None):
    """Logits of one token that are far enough apart, in random order, also when they are scaled."""
    margin = margin or 0.05 / m.outputs
    for _ in range(5000):
        z = torch.linspace(-1.5, 1.5, m.outputs)[torch.randperm(m.outputs, generator=g)]
        z = (z + 0.3 / m.outputs * torch.randn(m.outputs, generator=g)).bfloat16().float()
        if all(sure(c * z, correction, m, margin) for c in scales):
            return z
    raise AssertionError("no logits with a clear choice")


def weights(cfg, seed=1):
    """Random weights under which no choice of experts is close: every mixture has some entries of the stream
    to itself, which hold the token's logits and which no sublayer adds to.  Corrections are whole numbers, so
    that they decide between experts whatever the scale of the logits, and scores decide among equals."""
    w = H.random_state(cfg, seed, dtype=torch.float32)
    g = torch.Generator().manual_seed(seed)
    w["embed"] = torch.randn(w["embed"].shape, generator=g)
    at = 0
    for i, layer in enumerate(cfg.layers):
        if layer.mlp is not None and layer.mlp.kind == "softmax_moe":
            m = layer.mlp
            own = slice(at, at + m.outputs)
            at += m.outputs
            c = -(torch.arange(m.outputs) % 3 == 1).float() + 2.0 * (torch.arange(m.outputs) % 7 == 5).float()
            w[f"l{i}.mlp.correction"] = c
            w["embed"][:, own] = torch.stack([levels(m, c, g, (0.3, 1.0, 3.0)) for _ in range(cfg.vocab_size)])
            w[f"l{i}.mlp.router"].zero_()
            w[f"l{i}.mlp.router"][:, own] = torch.eye(m.outputs)
            w[f"l{i}.norm2"][own] = 1.0
            w[f"l{i}.norm2.b"][own] = 0.0
    assert at <= cfg.hidden_dim * 2 // 3
    for i, layer in enumerate(cfg.layers):
        w[f"l{i}.ls1"][:at] = 0
        if layer.mlp is not None:
            w[f"l{i}.ls2"][:at] = 0
    w["embed"] /= cfg.embed_scale
    return {n: t.bfloat16() for n, t in w.items()}


_made = {}


def forward(cfg, w, ids):
    return plain.forward(H.config_to_json(cfg), w, ids)


def Bench(kind, device, dtype):
    cfg = config(kind)
    if kind not in _made:
        _made[kind] = weights(cfg)
    return hybrid_checks.Bench(cfg, _made[kind], forward, device, dtype)


# --------------------------------------------------------------------------- mechanism checks
def check_norm_pass(device, dtype, tol):
    """The pass between two sublayers: layer norm, layer scale, bias, factors per row, weighted rows of which
    some are the token's own."""
    T, eps, top = 41, 3e-4, 3
    for W, ld in ((50, 56), (4100, 4104)):
        def vec(s, base=0.0):
            return torch.nn.functional.pad(base + 0.3 * rnd((W,), s, device), (0, ld - W))

        def mat(s, rows=T):
            return torch.nn.functional.pad(rnd((rows, W), s, device), (0, ld - W))
        x, y, bias, scale, gain, center = mat(1), mat(2), vec(3), vec(4, 1.0), vec(5, 1.0), vec(6)
        x[:, :W] += 3.0                                    # a mean that matters
        rows, own = mat(7, 200).to(dtype), mat(8).to(dtype)
        g = torch.Generator().manual_seed(9)
        slot = torch.randint(-60, 200, (T, top), generator=g).clamp_min(-1).int().to(device)
        weight, factor = rnd((T, top), 10, device), rnd((T,), 11, device)
        d = lambda t: t[..., :W].double().cpu()                                    # noqa: E731
        wd, sd = weight.double().cpu(), slot.long().cpu()
        spread = sum(wd[:, k, None] * torch.where(sd[:, k, None] < 0, d(own), d(rows)[sd[:, k].clamp_min(0)])
                     for k in range(top))
        sp = R.Spread(rows, slot, weight, own)
        for kw, v in ((dict(y=y, bias=bias), d(y) + d(bias)),
                      (dict(y=y.to(dtype), y_weight=factor, spread=sp),
                       d(y.to(dtype)) * factor.double().cpu()[:, None] + spread),
                      (dict(spread=sp), spread), (dict(), None)):
            want = d(x) if v is None else d(x) + v * d(scale)
            x2, h = R.add_norm(x, W, eps, dtype, gain=gain, center=center, scale=scale if kw else None, **kw)
            assert rel(x2[:, :W], want) < 2e-5
            assert rel(h[:, :W], plain.layer_norm(want, d(gain), d(center), eps)) < tol
            assert float(x2[:, W:].abs().max()) == float(h[:, W:].float().abs().max()) == 0
        pick = torch.tensor([7, 0, 40], dtype=torch.int32, device=device)
        _, h = R.add_norm(x, W, eps, dtype, y=y, scale=scale, gain=gain, center=center, rows=pick, spread=sp,
                          y_weight=factor)
        want = d(x) + (d(y) * factor.double().cpu()[:, None] + spread) * d(scale)
        assert rel(h[:, :W], plain.layer_norm(want, d(gain), d(center), eps)[[7, 0, 40]]) < tol


def check_scaled_embedding(device, dtype, tol):
    emb = torch.nn.functional.pad(rnd((9, 50), 4, device, dtype), (0, 6))
    tok = torch.tensor([8, 0, 3], dtype=torch.int32, device=device)
    out = torch.full((3, 56), 7.0, device=device)
    R.embed_norm(tok, emb, None, 50, 1e-5, out, 2.6)
    assert rel(out[:, :50], emb[[8, 0, 3], :50].cpu().double() * 2.6) < 1e-6
    assert float(out[:, 50:].abs().max()) == 0


def check_input_convolution(device, dtype, tol):
    """Two sequences cut at several places (inside a tile, at its edges, single tokens), in slots that hold
    something else; taps from one to the most; with and without a sublayer's result; narrow and wide rows."""
    eps, T = 1e-4, 75
    cuts = (((1, 30), (2, 1), (1, 2), (17, 1), (16, 33), (18, 1), (20, 7)), ((75, 3), (0, 72)), ((40, 16), (35, 59)))
    for W, ld, taps in ((44, 48, 3), (50, 56, 1), (96, 96, 4), (40, 40, 2), (24, 24, 17), (72, 72, 6), (2100, 2104, 4),
                        (4200, 4200, 2), (4096, 4096, 4)):
        def vec(s, base=0.0):
            return torch.nn.functional.pad(base + 0.3 * rnd((W,), s, device), (0, ld - W))
        w = torch.nn.functional.pad(rnd((taps, W), 3, device), (0, ld - W))
        gain, center, scale, bias = vec(4, 1.0), vec(5), vec(6, 1.0), vec(7)
        xs, ys = ([torch.nn.functional.pad(rnd((T, W), 10 * i + s, device), (0, ld - W)) for s in (0, 1)]
                  for i in (1, 2))
        d = lambda t: t[..., :W].double().cpu()                                    # noqa: E731
        for added in (True, False):
            wants = []
            for x, y in zip(xs, ys):
                v = d(x) + (d(y) + d(bias)) * d(scale) if added else d(x)
                wants.append((v, plain.conv_in(plain.layer_norm(v, d(gain), d(center), eps), d(w).T)))
            for plan in cuts:
                before = torch.full((3, taps - 1, ld), 9.0, device=device)
                at = [0, 0]
                for cut in plan:
                    take = [s for s in (0, 1) if cut[s]]
                    b = R.RaggedBatch([R.Entry((2, 0)[s], at[s], [0] * cut[s]) for s in take], torch.device(device))
                    x, y = (torch.cat([t[s][at[s]:at[s] + cut[s]] for s in take]).contiguous() for t in (xs, ys))
                    kw = dict(y=y, bias=bias, scale=scale) if added else {}
                    x2, h = R.add_norm(x, W, eps, dtype, gain=gain, center=center, taps=w, before=before, batch=b, **kw)
                    r = 0
                    for s in take:
                        v, want = (t[at[s]:at[s] + cut[s]] for t in wants[s])
                        assert rel(x2[r:r + cut[s], :W], v) < 2e-5
                        err = (d(h[r:r + cut[s]]) - want).abs().max() / wants[s][1].abs().max()
                        assert float(err) < tol, (W, taps, cut, s, float(err))
                        r, at[s] = r + cut[s], at[s] + cut[s]
                    assert W == ld or float(h[:, W:].float().abs().max()) == 0
                assert at == [T, T]


ROUTERS = (moe(6, 3, 13, 3, 2, 21, 3), moe(12, 4, 40, 4, 2, 72, 4), moe(5, 1, 9), moe(1, 1, 16, shared=8),
           moe(30, 12, 24, 40, 20, None, 10), moe(90, 6, 8, 8, 3, 136, 6), moe(12, 4, 64, 6, 2, 64),
           moe(2, 2, 136, 1, 1, None, 2))


def check_route(device, dtype, tol):
    """Choices, weights and the shared expert's gate; corrections of the size of the scores, negative ones
    too; tokens in blocks of several sizes."""
    for i, m in enumerate(ROUTERS):
        g = torch.Generator().manual_seed(i)
        n, r = m.outputs, m.routing()
        W = (n + 16) // 8 * 8
        corr = 0.5 / n * torch.randn(n, generator=g) - 1.0 / n
        for T in (1, 16, 61, 200):
            h = 0.1 * torch.randn(T, W, generator=g)
            for t in range(T):
                h[t, 3:3 + n] = levels(m, corr, g, margin=2e-3 / n)
            router = torch.zeros((n + 8) // 8 * 8, W)
            router[:n, 3:3 + n] = torch.eye(n)
            if r.shared_gate:
                router[n] = torch.randn(W, generator=g)
            h, router = h.to(dtype).to(device), router.to(dtype).to(device)
            c = X.route(h, router, r, corr.to(device))
            z = h.double().cpu()[:, 3:3 + n]
            for t in range(T):
                want, weight = plain.choose(z[t], corr.double(), m.top, m.groups, m.keep)
                got = dict(zip(c.expert[t].tolist(), c.weight[t].tolist()))
                assert set(got) == set(want), (i, t)
                assert all(abs(got[e] - float(x)) < 2e-6 for e, x in zip(want, weight)), (i, t)
            if r.shared_gate:
                gate = torch.sigmoid(h.double().cpu() @ router[n].double().cpu())
                assert float((c.shared.double().cpu() - gate).abs().max()) < 2e-5
            else:
                assert c.shared is None


def check_experts(device, dtype, tol):
    """Mixtures of experts in a model's layer, from one row to many."""
    for i, m in enumerate(ROUTERS):
        n = m.outputs
        W = 2 * n + 14
        cfg = H.HybridConfig(8, W, (L(A(1, 1, 4, 4, 0.5, 2, 10.0), m),), 1e-4, architecture="Dogilorn", conv_taps=2)
        w = H.random_state(cfg, i, dtype=torch.float32)
        w["l0.mlp.router"].zero_()
        w["l0.mlp.router"][:, :n] = torch.eye(n)
        w["l0.mlp.correction"] = torch.arange(n) % 2 * 0.5 / n
        w = {k: t.bfloat16().float() for k, t in w.items()}
        lm = H.HybridLM(cfg, w, device, dtype)
        eng, layer = lm.make_engine(max_batch=1), lm.layers[0]
        d = {k: t.double() for k, t in w.items()}
        corr = d["l0.mlp.correction"]
        g = torch.Generator().manual_seed(i)
        spec = {"router": dict(experts=m.experts, top=m.top, groups=dict(count=m.groups, keep=m.keep)),
                "shared": m.shared}
        for T in (1, 5, 16, 40, 150, 300) if i == 1 else (3, 17, 131) if n > 4 else (2, 2100):
            h = torch.randn(T, W, generator=g)
            for t in range(T):
                h[t, :n] = levels(m, corr.float(), g, margin=2e-3 / n)
            h = h.to(dtype)
            want = plain.experts(h.double(), d, "l0.mlp.", spec)
            hp = torch.nn.functional.pad(h, (0, layer.wp - W)).to(device)
            got = R.add_norm(torch.zeros((T, layer.wp), device=device), W, 1e-4, dtype, **eng._experts(layer, hp))[0]
            assert rel(got[:, :W], want) < tol, (i, T, rel(got[:, :W], want))


def check_linear_glu(device, dtype, tol):
    for M_, N_, K_ in ((1, 16, 24), (9, 80, 4104), (40, 48, 72), (17, 272, 136), (300, 528, 264)):
        x, w = rnd((M_, K_), 1, device, dtype), rnd((N_, K_), 2, device, dtype) * K_ ** -0.5 * 2
        bias = rnd((N_,), 3, device, dtype)
        z = x.cpu().double() @ w.cpu().double().T
        zb = z + bias.double().cpu()
        y = torch.empty((M_, N_ // 2), dtype=dtype, device=device)
        G.linear(x, w, y, bias=bias, glu=(1.702, 0.9, 1.0))
        assert rel(y, plain.bounded_glu(zb[:, 0::2], zb[:, 1::2], 0.9)) < tol
        G.linear(x, w, y, glu=(1.0, math.inf, 0.0))
        assert rel(y, plain.silu_glu(z[:, 0::2], z[:, 1::2])) < tol


def _turn_back(x, rot, base):
    """The inverse of the rotation: the second number of every pair changes its sign before and after."""
    if not rot:
        return x
    sign = torch.ones(x.shape[-1], dtype=x.dtype)
    sign[1:rot:2] = -1
    return plain.rotate_pairs(x * sign, rot, base) * sign


def _close(got, want, tol, dtype, what):
    err = (got.double().cpu() - want).abs().amax(1) / want.abs().max()
    # a score of 20 and more from bf16 operands moves weights that are close to one another
    assert float(err.max()) < (tol if dtype == torch.float32 else 0.08), (what, int(err.argmax()), float(err.max()))
    assert float(err.median()) < tol, (what, float(err.median()))


LONG_CUTS = (((1, 80), (2, 1), (1, 1), (140, 2), (127, 1), (9, 165), (140, 170)), ((3, 260), (5, 6), (412, 154)),
             ((420, 420),))


def _target(i, n, size, keep):
    """The key that a query at ``i`` aims at: near, far, at the edges of its window and of the kept positions,
    seen or just unseen, and at a page's border."""
    lo = max(0, i - size + 1)
    return min(i, (lo, max(lo - 1, 0), i, max(lo, i // 64 * 64), lo + (7 * i) % (i + 1 - lo), max(keep - 1, 0), keep,
                   0)[n % 8])


def _plain_mixer(spec):
    m = {"heads": spec.heads, "kv_heads": spec.kv_heads, "dim": spec.dim, "vdim": spec.vdim}
    if spec.rot_dims:
        m["rot"] = {"dims": spec.rot_dims, "base": spec.rot_base}
    return m


def _keys(raw, seg, spec, w, eps):
    """Keys and values in double precision from the projections ``raw``."""
    k = plain.unit_rms(raw[:, seg["k"]:seg["k"] + spec.kv_heads * spec.dim], eps) * w["k.norm"]
    v = raw[:, seg["v"]:seg["v"] + spec.kv_heads * spec.vdim].reshape(-1, spec.kv_heads, spec.vdim)
    return plain.rotated(k.view(-1, spec.kv_heads, spec.dim), _plain_mixer(spec)), plain.unit_rms(v, eps)


def _queries(raw, spec, w, eps):
    q = plain.unit_rms(raw[:, :spec.heads * spec.dim], eps) * w["q.norm"]
    return plain.rotated(q.view(-1, spec.heads, spec.dim), _plain_mixer(spec))


def _aim(raw, k, spec, w, shift):
    """``raw`` with queries that each point at one of the keys ``k``."""
    T, H_, d = raw.shape[0], spec.heads, spec.dim
    size = spec.window or 1 << 20
    q = torch.empty(T, H_, d, dtype=torch.float64)
    for i in range(T):
        for h in range(H_):
            q[i, h] = k[_target(i, i + h + shift, size, spec.keep_first), h // (H_ // spec.kv_heads)] / d ** 0.5
    raw = raw.clone()
    raw[:, :H_ * d] = 0.1 * raw[:, :H_ * d] + _turn_back(q, spec.rot_dims, spec.rot_base).flatten(1) / w["q.norm"]
    return raw


def check_kept_window_attention(device, dtype, tol):
    """Prompts whole and in portions, decoding; pieces, tiles and rows; kept positions of less and more than a
    page, windows narrower than what is kept, one key/value head and several."""
    T, eps = 420, 1e-4
    for spec, seed in ((A(6, 3, 10, 14, 3.0, 6, 300.0, 9, 2), 1), (A(4, 2, 64, 40, 0.5, 64, 1e4, 64, 5), 2),
                       (A(18, 1, 128, 128, 0.25, 32, 1e5, 100, 3), 3), (A(2, 2, 24, 64, 1.2, 24, 50.0, 1, 1), 4),
                       (A(2, 1, 160, 16, 0.2, 160, 1e3, 130, 66), 5), (A(4, 2, 8, 200, 3.0, 8, 1e4, 65, 64), 6),
                       (A(3, 3, 40, 72, 0.7, 0, 1.0, 300, 10), 7), (A(2, 1, 96, 80, 0.3, 16, 1e4, 70, 150), 8),
                       (A(2, 1, 56, 48, 0.5, 8, 1e2, 128), 9), (A(2, 2, 32, 32, 0.9, 32, 1e3), 10)):
        lm, w = single_mixer(spec, "Dogilorn", device, dtype, seed, conv_taps=2)
        layer = lm.layers[0]
        raws, wants = [], []
        for s in (0, 1):
            raw = rnd((T, layer.w_in.shape[0]), 10 * seed + s, "cpu", dtype).double()
            raw = _aim(raw, _keys(raw, layer.seg, spec, w, eps)[0], spec, w, s).to(dtype)
            raws.append(raw.to(device))
            raw = raw.double()
            wants.append(plain.attend(_queries(raw, spec, w, eps), *_keys(raw, layer.seg, spec, w, eps), spec.scale,
                                      w["temp"], spec.window, spec.keep_first).flatten(1))
        for cuts in LONG_CUTS:
            got, _ = drive(lm, raws, cuts, lambda e, layer, raw, out, b, rope: e._heads(
                0, layer, raw, out, b, rope, b.max_ctx))
            for y, want in zip(got, wants):
                _close(y, want, tol, dtype, (spec, cuts))


def check_shared_keys(device, dtype, tol):
    """Layers with the keys and values of an earlier one and masks of their own, wider and narrower; factors
    and signs of the scores differ by head."""
    T, eps = 420, 1e-4
    for specs, seed in (
            ((A(4, 2, 64, 40, 0.5, 64, 1e4, 64, 5), A(4, 2, 64, 40, 0.4, 64, 1e4, 130, 2, 0),
              A(4, 2, 64, 40, 0.6, 64, 1e4, 20, 0, 0), A(4, 2, 64, 40, 0.5, 64, 1e4, 64, 5, 0)), 1),
            ((A(3, 1, 20, 28, 1.0, 6, 1e2, None), A(3, 1, 20, 28, 1.0, 6, 1e2, 33, 70, 0)), 2),
            ((A(2, 1, 128, 104, 0.3, 128, 1e4, 100, 4), A(2, 1, 128, 104, 0.3, 128, 1e4, None, 0, 0)), 3),
            ((A(2, 1, 144, 16, 0.3, 16, 1e4, 30, 4), A(2, 1, 144, 16, 0.3, 16, 1e4, 90, 1, 0)), 4)):
        cfg = H.HybridConfig(16, 16, tuple(L(s, None) for s in specs), eps, architecture="Dogilorn", conv_taps=1)
        w = {n: t.bfloat16().float() for n, t in H.random_state(cfg, seed, dtype=torch.float32).items()}
        for i in range(len(specs)):
            w[f"l{i}.mix.temp"][::2] *= -0.7
        lm = H.HybridLM(cfg, w, device, dtype)
        mix = [{n[len(f"l{i}.mix."):]: t.double() for n, t in w.items() if n.startswith(f"l{i}.mix.")}
               for i in range(len(specs))]
        widths, seg = [layer.w_in.shape[0] for layer in lm.layers], lm.layers[0].seg
        for n in range(1, len(specs)):
            cols = slice(sum(widths[:n]), sum(widths[:n + 1]))
            raws, wants = [], []
            for s in (0, 1):
                raw = rnd((T, sum(widths)), 10 * seed + s, "cpu", dtype).double()
                raw[:, cols] = _aim(raw[:, cols], _keys(raw, seg, specs[0], mix[0], eps)[0], specs[n], mix[n], s)
                raw = raw.to(dtype)
                raws.append(raw.to(device))
                raw = raw.double()
                wants.append(plain.attend(_queries(raw[:, cols], specs[n], mix[n], eps),
                                          *_keys(raw, seg, specs[0], mix[0], eps), specs[n].scale,
                                          mix[n]["temp"], specs[n].window, specs[n].keep_first).flatten(1))

            def run(e, layer, raw, out, b, rope):
                at = 0
                for i, width in enumerate(widths):         # all layers, as a step runs them
                    e._heads(i, lm.layers[i], raw[:, at:at + width].contiguous(),
                             out if i == n else torch.empty_like(out), b, rope, b.max_ctx)
                    at += width
            for cuts in LONG_CUTS:
                got, eng = drive(lm, raws, cuts, run)
                assert len(eng.cache.k) == 1
                for y, want in zip(got, wants):
                    _close(y, want, tol, dtype, (specs[n], cuts))


MECHANISM_CHECKS = [check_norm_pass, check_scaled_embedding, check_input_convolution, check_route, check_experts,
                    check_linear_glu, check_kept_window_attention, check_shared_keys]
