"""Small Rupasun configurations, weights and checks shared by the CPU and the GPU tests.  The oracle is
:mod:`plain_rupasun`; the configurations are chosen so that sizes differ from one another (heads, key and
value widths, rotated parts, windows, experts, groups), with and without each option."""
import torch

import hybrid_checks
import plain_rupasun as plain
from coeus_b200.models import hybrid as H
from coeus_b200.ops import experts as X
from coeus_b200.ops import gemm as G
from coeus_b200.ops import ragged as R
from hybrid_checks import CUTS, MODEL_CHECKS, agrees, drive, rel, rnd, single_mixer, tokens  # noqa: F401

L, M, E = H.LayerSpec, H.MlpSpec, H.GluSpec


def D(heads, kv_heads, dim, vdim, diff, scale, rot, base):
    return H.DiffAttentionSpec(heads, kv_heads, dim, vdim, scale, rot, base, diff=diff)


def C(heads, kv_heads, dim, vdim, scale, rot, base, window, cap):
    return H.CappedAttentionSpec(heads, kv_heads, dim, vdim, scale, rot, base, window, cap)


def config(kind):
    def make(vocab, width, eps, *layers):
        return H.HybridConfig(vocab, width, layers, eps, architecture="Rupasun")
    if kind == "odd":         # nothing is a multiple of eight
        return make(83, 44, 2e-5,
                    L(D(6, 3, 10, 14, 0.3, 0.3, 6, 300.0), H.MoeSpec(6, 3, E(13, 0.8), 1.7, 3, 2, E(21, 1.5))),
                    L(C(5, 1, 14, 6, 0.4, 10, 1e4, 9, 5.0), M(50)),
                    L(D(3, 3, 12, 5, 0.7, 0.25, 12, 50.0), None),
                    L(C(2, 2, 6, 11, 0.6, 6, 500.0, 70, 2.0), H.MoeSpec(5, 2, E(9, 2.0), 0.6, 1, 1, None)))
    if kind == "wide":        # vectorised paths, several pages per window, more than 16 queries on a key
        return make(264, 96, 1e-6,
                    L(D(8, 2, 64, 128, 0.4, 0.125, 32, 1e4), M(128)),
                    L(C(4, 2, 128, 96, 0.09, 128, 1e4, 150, 30.0),
                      H.MoeSpec(16, 4, E(40, 1.0), 2.5, 4, 2, E(72, 3.0))),
                    L(D(18, 1, 24, 40, 0.2, 0.2, 16, 1e5), H.MoeSpec(12, 1, E(24, 0.7), 1.0, 2, 1, E(24, 0.5))),
                    L(C(20, 1, 40, 64, 0.16, 24, 100.0, 64, 8.0), None),
                    L(D(2, 2, 96, 72, 0.6, 0.1, 96, 1e4), H.MoeSpec(8, 8, E(16, 1.2), 1.0, 8, 8, None)))
    return make(60, 32, 1e-5,     # "large": heads that only the general kernels take, narrowest windows
                L(D(2, 1, 136, 200, 0.5, 0.08, 64, 1e4), None),
                L(C(3, 3, 160, 24, 0.08, 160, 1e3, 33, 12.0), H.MoeSpec(4, 2, E(24, 1.0), 1.0, 2, 2, E(8, 1.0))),
                L(D(2, 2, 72, 136, 0.1, 0.11, 72, 10.0), M(24)),
                L(C(2, 1, 24, 136, 0.3, 2, 5.0, 1, 3.0), None),
                L(C(2, 1, 8, 8, 0.4, 8, 10.0, 64, 50.0), M(8)))


def sure(z, m, margin=0.01):
    """Whether the choice of experts by the logits ``z`` holds when they change a little."""
    s = torch.sigmoid(z)
    n = m.experts // m.groups
    value = sorted((sum(sorted(s[g * n:(g + 1) * n].tolist())[-2:]) for g in range(m.groups)), reverse=True)
    if m.keep < m.groups and value[m.keep - 1] - value[m.keep] < margin:
        return False
    order = sorted(z.tolist())
    return min((b - a for a, b in zip(order, order[1:])), default=1.0) > margin


def levels(m, g, scales=(1.0,), margin=None):
    """Logits of one token that are far enough apart, in random order, also when they are scaled."""
    margin = margin or 0.3 / m.experts
    for _ in range(1000):
        z = torch.linspace(-2.0, 2.0, m.experts)[torch.randperm(m.experts, generator=g)]
        z = z + 0.3 / m.experts * torch.randn(m.experts, generator=g)
        if all(sure(c * z, m, c * margin / 2) for c in scales):
            return z
    raise AssertionError("no logits with a clear choice")


def weights(cfg, seed=1):
    """Random weights under which old tokens matter (peaked attention) and no choice of experts is close:
    every mixture has some entries of the stream to itself, which hold the token's logits and which no
    sublayer adds to."""
    w = H.random_state(cfg, seed, dtype=torch.float32)
    g = torch.Generator().manual_seed(seed)
    at = 0
    for i, layer in enumerate(cfg.layers):
        if layer.mixer.kind == "diff_attention":
            w[f"l{i}.mix.q"] *= 2.0
        if layer.mlp is not None and layer.mlp.kind == "moe":
            m = layer.mlp
            own = slice(at, at + m.experts)
            at += m.experts
            w["embed"][:, own] = torch.stack([levels(m, g, (0.5, 1.0, 2.0)) for _ in range(cfg.vocab_size)])
            w[f"l{i}.mlp.router"].zero_()
            w[f"l{i}.mlp.router"][:, own] = 2.0 * torch.eye(m.experts)
            w[f"l{i}.norm2"][own] = 1.0
    assert at <= cfg.hidden_dim // 2
    for n in w:
        if n.endswith((".mix.o", ".down")):
            w[n][:at] = 0
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
def check_spread(device, dtype, tol):
    """The pass between two sublayers that also gathers weighted rows, with and without a plain part."""
    W, ld, T, eps, top = 50, 56, 41, 3e-4, 3
    pad = lambda t: torch.nn.functional.pad(t, (0, ld - W))                    # noqa: E731
    x, y = pad(rnd((T, W), 1, device)), pad(rnd((T, W), 2, device))
    rows = pad(rnd((200, W), 3, device)).to(dtype)
    slot = torch.randint(0, 200, (T, top), generator=torch.Generator().manual_seed(4)).int().to(device)
    weight = rnd((T, top), 5, device)
    post, gain = pad(1 + 0.3 * rnd((W,), 6, device)), pad(1 + 0.3 * rnd((W,), 7, device))
    d = lambda t: t[..., :W].double().cpu()                                    # noqa: E731
    v = (d(rows)[slot.long().cpu()] * weight.double().cpu()[..., None]).sum(1)
    for yt in (None, torch.float32, dtype):
        u = v + d(y.to(yt)) if yt else v
        want = d(x) + plain.rms_norm(u, d(post), eps)
        x2, h = R.add_norm(x, W, eps, dtype, y=y.to(yt) if yt else None, post=post, gain=gain,
                           spread=R.Spread(rows, slot, weight))
        assert rel(x2[:, :W], want) < 2e-5
        assert rel(h[:, :W], plain.rms_norm(want, d(gain), eps)) < tol
        assert float(x2[:, W:].abs().max()) == float(h[:, W:].float().abs().max()) == 0
    pick = torch.tensor([7, 0, 40], dtype=torch.int32, device=device)
    _, h = R.add_norm(x, W, eps, dtype, y=y, post=post, gain=gain, rows=pick, spread=R.Spread(rows, slot, weight))
    want = d(x) + plain.rms_norm(v + d(y), d(post), eps)
    assert rel(h[:, :W], plain.rms_norm(want, d(gain), eps)[[7, 0, 40]]) < tol


ROUTERS = (H.MoeSpec(6, 3, E(13, 0.8), 1.7, 3, 2, E(21, 1.5)), H.MoeSpec(16, 4, E(40, 1.0), 2.5, 4, 2, E(72, 3.0)),
           H.MoeSpec(5, 1, E(9, 0.5), 1.0, 1, 1, None), H.MoeSpec(1, 1, E(16, 1.0), 3.0, 1, 1, E(8, 0.2)),
           H.MoeSpec(40, 12, E(24, 1.1), 0.5, 40, 20, None), H.MoeSpec(96, 6, E(8, 1.0), 1.0, 8, 3, E(136, 1.0)),
           H.MoeSpec(12, 4, E(64, 1.0), 1.0, 6, 2, E(64, 1.0)), H.MoeSpec(2, 1, E(136, 1.0), 1.0, 1, 1, None))


def check_route(device, dtype, tol):
    """Choices and weights, tokens in blocks of several sizes, groups of one, two and more experts."""
    for i, m in enumerate(ROUTERS):
        g = torch.Generator().manual_seed(i)
        W = m.experts + 9
        W += -W % 8
        for T in (1, 16, 61, 200):
            h = 0.1 * torch.randn(T, W, generator=g)
            for t in range(T):
                h[t, 3:3 + m.experts] = levels(m, g)
            router = torch.zeros(m.experts + -m.experts % 8, W)
            router[:m.experts, 3:3 + m.experts] = torch.eye(m.experts)
            h, router = h.to(dtype).to(device), router.to(dtype).to(device)
            c = X.route(h, router, m.routing())
            z = h.double().cpu()[:, 3:3 + m.experts]
            for t in range(T):
                want, weight = plain.choose(z[t], m.top, m.groups, m.keep, m.scale)
                got = dict(zip(c.expert[t].tolist(), c.weight[t].tolist()))
                if sure(z[t], m, 1e-5):
                    assert set(got) == set(want), (i, t)
                    assert all(abs(got[e] - float(x)) < 2e-6 * m.scale for e, x in zip(want, weight)), (i, t)


def check_experts(device, dtype, tol):
    """Mixtures of experts in a model's layer, from one row to many; the bounds of the gated unit bite."""
    for i, m in enumerate(ROUTERS):
        W = 2 * m.experts + 14
        cfg = H.HybridConfig(8, W, (L(D(1, 1, 4, 4, 0.5, 0.5, 2, 10.0), m),), 1e-4, architecture="Rupasun")
        w = H.random_state(cfg, i, dtype=torch.float32)
        w["l0.mlp.router"].zero_()
        w["l0.mlp.router"][:, :m.experts] = torch.eye(m.experts)
        for n in w:
            if n.endswith((".gate", ".up")):
                w[n] *= 2.0
        w = {n: t.bfloat16().float() for n, t in w.items()}
        lm = H.HybridLM(cfg, w, device, dtype)
        eng, layer = lm.make_engine(max_batch=1), lm.layers[0]
        d = {n: t.double() for n, t in w.items()}
        g = torch.Generator().manual_seed(i)
        for T in (1, 5, 16, 40, 150, 300) if i == 1 else (3, 17, 131) if m.experts > 2 else (2, 2100):
            h = torch.randn(T, W, generator=g)
            for t in range(T):
                h[t, :m.experts] = levels(m, g)
            h = h.to(dtype)
            clear = torch.tensor([sure(h[t, :m.experts].float(), m, 1e-5) for t in range(T)])
            spec = {"router": dict(top=m.top, scale=m.scale, groups=dict(count=m.groups, keep=m.keep)),
                    "expert": dict(limit=m.expert.limit)}
            if m.shared:
                spec["shared"] = dict(limit=m.shared.limit)
            want = plain.experts(h.double(), d, "l0.mlp.", spec)
            hp = torch.nn.functional.pad(h, (0, layer.wp - W)).to(device)
            got = R.add_norm(torch.zeros((T, layer.wp), device=device), W, 1e-4, dtype, **eng._experts(layer, hp))[0]
            assert rel(got[:, :W].cpu()[clear], want[clear]) < tol, (i, T, rel(got[:, :W], want))


def check_linear_glu(device, dtype, tol):
    for M_, N_, K_ in ((1, 16, 24), (40, 48, 72), (17, 272, 136), (300, 528, 264)):
        x, w = rnd((M_, K_), 1, device, dtype), rnd((N_, K_), 2, device, dtype) * K_ ** -0.5 * 2
        z = x.cpu().double() @ w.cpu().double().T
        y = torch.empty((M_, N_ // 2), dtype=dtype, device=device)
        G.linear(x, w, y, glu=(1.702, 0.9))
        assert rel(y, plain.clamped_glu(z[:, 0::2], z[:, 1::2], 0.9)) < tol


def _turn_back(x, rot, base, interleaved):
    """The inverse of the rotation: the second number of every pair changes its sign before and after."""
    sign = torch.ones(x.shape[-1], dtype=x.dtype)
    if interleaved:
        sign[1:rot:2] = -1
        return plain.rotate_pairs(x * sign, rot, base) * sign
    sign[rot // 2:rot] = -1
    return plain.rotate_halves(x * sign, rot, base) * sign


def _close(got, want, tol, dtype, what):
    err = (got.double().cpu() - want).abs().amax(1) / want.abs().max()
    # a score of 20 and more from bf16 operands moves weights that are close to one another
    assert float(err.max()) < (tol if dtype == torch.float32 else 0.08), (what, int(err.argmax()), float(err.max()))
    assert float(err.median()) < tol, (what, float(err.median()))


def check_diff_attention(device, dtype, tol):
    """Every query of every map has one key that stands out, near, far or at a page's border; prompts
    whole and in portions, decoding."""
    T = 210
    for spec, seed in ((D(6, 3, 10, 14, 0.3, 0.3, 6, 300.0), 1), (D(4, 2, 64, 128, 0.5, 0.125, 64, 1e4), 2),
                       (D(18, 2, 40, 64, 0.2, 0.2, 16, 1e5), 3), (D(2, 2, 128, 96, 0.8, 0.1, 48, 50.0), 4),
                       (D(2, 1, 136, 200, 0.4, 0.1, 136, 1e3), 5), (D(3, 1, 24, 152, 0.1, 0.3, 0, 1.0), 6)):
        lm, w = single_mixer(spec, "Rupasun", device, dtype, seed)
        layer, H_, Gr, d, dv = lm.layers[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim
        seg, m = layer.seg, dict(scale=spec.scale, diff=spec.diff)
        lam = plain.difference_weight(*(w[n] for n in ("lq1", "lk1", "lq2", "lk2")), spec.diff)
        raws, wants = [], []
        for s in (0, 1):
            raw = rnd((T, layer.w_in.shape[0]), 10 * seed + s, "cpu", dtype).double()
            k = raw[:, seg["k"]:seg["k"] + 2 * Gr * d].reshape(T, 2 * Gr, d)
            turned = plain.rotate_halves(k, spec.rot_dims, spec.rot_base).view(T, Gr, 2, d)
            aim = torch.empty(T, H_, 2, d, dtype=torch.float64)
            for i in range(T):
                for n in (0, 1):
                    j = (0, i, i // 64 * 64, max(0, i // 64 * 64 - 1), (7 * i + 3) % (i + 1))[(i + 2 * n) % 5]
                    key = turned[i - j if i % 3 == 0 else j].repeat_interleave(H_ // Gr, 0)[:, n]
                    aim[i, :, n] = key * (25.0 / spec.scale / key.square().sum(-1, keepdim=True))
            raw[:, :2 * H_ * d] += _turn_back(aim.flatten(1, 2), spec.rot_dims, spec.rot_base, False).flatten(1)
            raw = raw.to(dtype)
            raws.append(raw.to(device))
            raw = raw.double()
            q, k = (plain.rotate_halves(raw[:, at:at + 2 * c * d].reshape(T, 2 * c, d), spec.rot_dims, spec.rot_base)
                    for at, c in ((0, H_), (seg["k"], Gr)))
            v = raw[:, seg["v"]:seg["v"] + Gr * dv].reshape(T, Gr, dv)
            wants.append(plain.diff_heads(q.view(T, H_, 2, d), k.view(T, Gr, 2, d), v, m, lam, 1e-4).flatten(1))
        for cuts in CUTS + (((T, T),),):
            got, _ = drive(lm, raws, cuts, lambda e, layer, raw, out, b, rope: e._heads(
                0, layer, raw, out, b, rope, b.max_ctx))
            for y, want in zip(got, wants):
                _close(y, want, tol, dtype, (spec, cuts))


def check_capped_attention(device, dtype, tol):
    """Every query has one key that stands out: its window's first, the one before that (unseen), itself, a
    page's border, or one somewhere in between."""
    T = 210
    for spec, seed in ((C(6, 3, 10, 14, 2.0, 6, 300.0, 9, 30.0), 1), (C(4, 2, 64, 40, 0.4, 64, 1e4, 64, 25.0), 2),
                       (C(18, 1, 128, 128, 0.2, 32, 1e5, 100, 20.0), 3), (C(2, 2, 24, 64, 1.0, 24, 50.0, 1, 9.0), 4),
                       (C(2, 1, 160, 16, 0.15, 160, 1e3, 130, 60.0), 5), (C(4, 2, 8, 200, 2.5, 8, 1e4, 65, 30.0), 6),
                       (C(3, 3, 40, 72, 0.6, 0, 1.0, 300, 50.0), 7), (C(2, 2, 96, 80, 0.25, 96, 1e4, 64, 25.0), 8),
                       (C(2, 1, 56, 48, 0.4, 8, 1e2, 128, 30.0), 9), (C(2, 1, 20, 20, 1.2, 20, 1e3, 5, 60.0), 10)):
        lm, w = single_mixer(spec, "Rupasun", device, dtype, seed)
        layer, H_, Gr, d, dv, size = lm.layers[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.window
        seg, m = layer.seg, dict(scale=spec.scale, mask=dict(size=size), softcap=spec.softcap)
        raws, wants = [], []
        for s in (0, 1):
            raw = rnd((T, layer.w_in.shape[0]), 10 * seed + s, "cpu", dtype).double()
            k = raw[:, seg["k"]:seg["k"] + Gr * d].reshape(T, Gr, d)
            turned = plain.rotate_pairs(k, spec.rot_dims, spec.rot_base)
            aim = torch.empty(T, H_, d, dtype=torch.float64)
            for i in range(T):
                lo = max(0, i - size + 1)
                j = (lo, max(lo - 1, 0), i, max(lo, i // 64 * 64), lo + (7 * i) % (i + 1 - lo))[i % 5]
                aim[i] = 3.0 * turned[j].repeat_interleave(H_ // Gr, 0)
            raw[:, :H_ * d] *= 0.5
            raw[:, :H_ * d] += _turn_back(aim, spec.rot_dims, spec.rot_base, True).flatten(1)
            raw = raw.to(dtype)
            raws.append(raw.to(device))
            raw = raw.double()
            q, k = (plain.rotate_pairs(raw[:, at:at + c * d].reshape(T, c, d), spec.rot_dims, spec.rot_base)
                    for at, c in ((0, H_), (seg["k"], Gr)))
            v = raw[:, seg["v"]:seg["v"] + Gr * dv].reshape(T, Gr, dv)
            gate = torch.sigmoid(raw[:, seg["g"]:seg["g"] + H_ * dv])
            wants.append(plain.capped_heads(q, k, v, m, 1e-4).flatten(1) * gate)
        for cuts in CUTS + (((T, T),),):
            got, _ = drive(lm, raws, cuts, lambda e, layer, raw, out, b, rope: e._heads(
                0, layer, raw, out, b, rope, b.max_ctx))
            for y, want in zip(got, wants):
                _close(y, want, tol, dtype, (spec, cuts))


MECHANISM_CHECKS = [check_spread, check_route, check_experts, check_linear_glu, check_diff_attention,
                    check_capped_attention]
