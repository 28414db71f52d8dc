"""Small Bananex configurations, weights and checks shared by the CPU and the GPU tests.  The oracle
is :mod:`plain_bananex`; the configurations are chosen so that sizes differ from one another (heads,
key, value and latent widths, windows, taps, groups, loop), with and without each option."""
import torch

import hybrid_checks
import plain_bananex as plain
from coeus_b200.models import hybrid as H
from coeus_b200.ops import gemm as G
from coeus_b200.ops import latent as LT
from coeus_b200.ops import ragged as R
from hybrid_checks import CUTS, MODEL_CHECKS, agrees, drive, rel, rnd, single_mixer, tokens  # noqa: F401

A, S, U, M, L = H.LatentAttentionSpec, H.Mamba2Spec, H.MinGruSpec, H.MlpSpec, H.LayerSpec


def config(kind):
    def make(vocab, width, eps, scale, loop, *layers):
        return H.HybridConfig(vocab, width, layers, eps, architecture="Bananex", logit_scale=scale,
                              loop=H.LoopSpec(*loop) if loop else None)
    if kind == "odd":         # nothing is a multiple of eight; layers before and behind the loop
        return make(83, 44, 2e-5, 0.7, (1, 4, 3),
                    L(S(6, 7, 10, 3, 5, 2), M(50)),
                    L(A(3, 10, 6, 7, 21, 0.25, 9, 300.0), None),
                    L(U(37), M(21)),
                    L(S(2, 9, 5, 2, 1, 3), None),
                    L(A(5, 14, 2, 5, 11, 0.2, 70, 5000.0), M(36)))
    if kind == "wide":        # vectorised paths, several pages per window, more than 16 heads
        return make(264, 96, 1e-6, 1.3, (0, 3, 2),
                    L(A(4, 48, 16, 40, 72, 0.2, 150, 1e4), M(128)),
                    L(S(4, 64, 128, 2, 4, 4), M(64)),
                    L(U(136), M(72)),
                    L(A(18, 80, 32, 128, 200, 0.15, 77, 1e5), None),
                    L(S(8, 24, 64, 1, 2, 8), M(40)),
                    L(A(2, 136, 24, 40, 304, 0.12, 33, 100.0), M(64)))
    if kind == "state":       # recurrences only, no loop
        return make(40, 24, 1e-5, 1.0, None,
                    L(S(3, 80, 40, 1, 3, 1), M(24)), L(U(24), None), L(S(2, 20, 16, 2, 2, 1), M(16)),
                    L(U(50), M(40)))
    return make(40, 32, 1e-5, 2.0, (0, 3, 1),    # "latent": attention only, a loop of one pass
                L(A(2, 8, 8, 24, 16, 0.5, 1, 10.0), M(24)),
                L(A(2, 24, 40, 64, 56, 0.25, 64, 1e4), M(24)),
                L(A(3, 64, 64, 128, 80, 0.2, None, 1e3), M(24)))


def weights(cfg, seed=1):
    """Random weights under which old tokens matter: peaked attention, slow decay, strong shifts."""
    w = H.random_state(cfg, seed, dtype=torch.float32)
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}.mix."
        if isinstance(layer.mixer, A):
            w[p + "q"] *= 2.0
        elif isinstance(layer.mixer, S):
            w[p + "dt_bias"] -= 2.0
        else:
            w[p + "z.b"] -= 2.0
    return {n: t.bfloat16() for n, t in w.items()}


_made = {}


def forward(cfg, w, ids):
    return plain.forward(H.config_to_json(cfg), w, ids)


def Bench(kind, device, dtype):
    cfg = config(kind)
    if kind not in _made:
        _made[kind] = weights(cfg)
    # narrow output-norm parts and eleven runs of 44 numbers amplify the rounding of bf16 operands at
    # single positions of "odd"; its fp32 tolerance is the common one
    tol = 0.2 if kind == "odd" and dtype == torch.bfloat16 else None
    return hybrid_checks.Bench(cfg, _made[kind], forward, device, dtype, tol)


# --------------------------------------------------------------------------- mechanism checks
def check_norms_and_shift(device, dtype, tol):
    """The pass between two sublayers, two sequences in two slots cut at several places."""
    W, ld, T, eps = 50, 56, 75, 3e-4
    vec = lambda s: torch.nn.functional.pad(1 + 0.3 * rnd((W,), s, device), (0, ld - W))   # noqa: E731
    for scalar, with_x, with_post, yt in ((True, True, True, dtype), (False, True, True, torch.float32),
                                          (True, False, False, torch.float32),
                                          (True, True, False, torch.float32)):
        gain = torch.tensor([0.7], device=device) if scalar else vec(1)
        post = (torch.tensor([1.4], device=device) if scalar else vec(2)) if with_post else None
        bias, shift = vec(3) - 1.0, vec(4)
        shift[W:] = bias[W:] = 0
        pad = lambda t: torch.nn.functional.pad(t, (0, ld - W))                              # noqa: E731
        xs = [pad(rnd((T, W), 10 + s, device)) for s in (0, 1)]
        ys = [pad(rnd((T, W), 20 + s, device)).to(yt) for s in (0, 1)]
        before = torch.full((3, ld), 9.0, device=device)
        got, at = [[[], [], []], [[], [], []]], [0, 0]
        for cut in ((1, 40), (2, 1), (1, 1), (31, 2), (40, 1), (0, 30)):
            ents = [R.Entry(slot, at[s], [0] * cut[s]) for s, slot in ((0, 2), (1, 0)) if cut[s]]
            b = R.RaggedBatch(ents, device)
            x = torch.cat([xs[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
            y = torch.cat([ys[s][at[s]:at[s] + cut[s]] for s in (0, 1)])
            both = torch.full((b.T, 2 * ld), 5.0, dtype=dtype, device=device)
            x2, h = R.add_norm(x if with_x else None, W, eps, dtype, y=y, bias=bias, post=post, gain=gain,
                               shift=shift, before=before, batch=b, casts=[both[:, ld:]])
            assert float((both[:, :ld].float() - 5.0).abs().max()) == 0
            for k, t in enumerate((x2, h, both[:, ld:])):
                got[0][k].append(t[:cut[0]])
                got[1][k].append(t[cut[0]:])
            at = [at[0] + cut[0], at[1] + cut[1]]
        for s, slot in ((0, 2), (1, 0)):
            d = lambda t: t[..., :W].double().cpu()                                          # noqa: E731
            g = lambda t: t.double().cpu() if t.numel() == 1 else d(t)                       # noqa: E731
            v = d(ys[s]) + d(bias)
            v = plain.rms_norm(v, g(post), eps) if with_post else v
            want = d(xs[s]) + v if with_x else v
            h = plain.rms_norm(want, g(gain), eps)
            x2, hh, both = (torch.cat(t) for t in got[s])
            assert rel(x2[:, :W], want) < 2e-5 and rel(both[:, :W], want) < tol
            assert rel(hh[:, :W], plain.token_shift(h, d(shift))) < tol
            assert rel(before[slot, :W], h[-1]) < 2e-5
            assert float(x2[:, W:].abs().max()) == float(hh[:, W:].float().abs().max()) == 0
    rows = torch.tensor([4, 0, 71], dtype=torch.int32, device=device)
    _, h = R.add_norm(xs[0], W, eps, dtype, y=ys[0], post=torch.tensor([1.2], device=device), gain=vec(5),
                      rows=rows)
    x = d(xs[0]) + plain.rms_norm(d(ys[0]), 1.2, eps)
    assert rel(h[:, :W], plain.rms_norm(x, d(vec(5)), eps)[[4, 0, 71]]) < tol


def check_linear(device, dtype, tol):
    """Biases and the erf activation in the products, few rows and many."""
    for M_, N_, K_ in ((1, 8, 24), (3, 40, 8), (17, 136, 72), (70, 200, 136), (300, 520, 264)):
        x, w = rnd((M_, K_), 1, device, dtype), rnd((N_, K_), 2, device, dtype) * K_ ** -0.5 * 2
        b = rnd((N_,), 3, device, dtype)
        z = x.cpu().double() @ w.cpu().double().T + b.cpu().double()
        y = torch.empty((M_, N_), dtype=dtype, device=device)
        f = torch.empty((M_, N_), device=device)
        assert rel(G.linear(x, w, y, bias=b), z) < tol
        assert rel(G.linear(x, w, f, bias=b), z) < tol
        want = plain.gelu_erf(z)
        assert rel(G.linear(x, w, y, bias=b, epi="gelu_erf"), want) < tol
        # small results on the negative side too
        err = (y.double().cpu() - want).abs() / want.abs().clamp_min(1e-2)
        assert float(err.max()) < (1e-3 if dtype == torch.float32 else 0.3)


def check_linear_heads(device, dtype, tol):
    for heads, n, N_, K_, pitch in ((3, 5, 24, 16, 24), (2, 40, 150, 72, 80), (18, 17, 70, 136, 136)):
        x = rnd((n + 3, heads, pitch), 1, device, dtype)
        w = rnd((heads, N_, K_), 2, device, dtype) * K_ ** -0.5
        want = torch.einsum("ihk,hnk->ihn", x[..., :K_].double().cpu(), w.double().cpu())
        y = torch.full((n + 3, heads * N_ + 8), 5.0, dtype=dtype, device=device)
        LT.linear_heads(x, w, y[:, :heads * N_], N_)
        assert rel(y[:, :heads * N_], want.flatten(1)) < tol
        assert float((y[:, heads * N_:].float() - 5.0).abs().max()) == 0
        idx = torch.randperm(n + 3, generator=torch.Generator().manual_seed(3))[:n].int().to(device)
        few = torch.empty((n, heads * N_), dtype=dtype, device=device)
        LT.linear_heads(x, w, few, N_, x_rows=idx)
        assert rel(few, want[idx.long().cpu()].flatten(1)) < tol
        gate = rnd((n + 3, heads * N_), 4, device, dtype)
        y.fill_(5.0)
        LT.linear_heads(x[:n], w, y[:, :heads * N_], N_, y_rows=idx, gate=gate)
        g = torch.sigmoid(gate.double().cpu())[idx.long().cpu()]
        assert rel(y[idx.long(), :heads * N_], want[:n].flatten(1) * g) < tol
        rest = sorted(set(range(n + 3)) - set(idx.tolist()))
        assert float((y[rest].float() - 5.0).abs().max()) == 0


def _mixer(spec, device, dtype, seed):
    return single_mixer(spec, "Bananex", device, dtype, seed)


def check_latent_attention(device, dtype, tol):
    """Every query has one key that stands out: its window's first, the one before that, itself, or
    one somewhere in between; prompts whole and in portions, decoding, edges of pages and windows."""
    for spec, seed in ((A(3, 10, 6, 7, 21, 0.3, 9, 300.0), 1), (A(2, 48, 16, 40, 72, 0.2, 64, 1e4), 2),
                       (A(17, 64, 32, 112, 136, 0.15, 100, 1e5), 3), (A(2, 24, 40, 64, 520, 0.2, 1, 50.0), 4),
                       (A(1, 100, 60, 16, 40, 0.1, 130, 1e3), 5), (A(2, 32, 32, 64, 300, 0.2, None, 1e4), 6),
                       (A(4, 8, 8, 200, 24, 0.5, 65, 1e4), 7)):
        lm, w = _mixer(spec, device, dtype, seed)
        seg, layer = lm.layers[0].seg, lm.layers[0]
        H_, d, r, dv, rank, T = spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank, 210
        size = spec.window or T
        raws, wants = [], []
        for s in (0, 1):
            raw = rnd((T, layer.w_in.shape[0]), 10 * seed + s, "cpu", dtype).double()
            down = raw[:, seg["dkv"]:seg["dkv"] + rank + r]
            c = plain.rms_norm(down[:, :rank], w["dkv.norm"], 1e-4)
            k = (c @ w["uk"].T).view(T, H_, d)
            q = raw[:, :H_ * (d + r)].view(T, H_, d + r)
            for i in range(T):
                lo = max(0, i - size + 1)
                j = (lo, max(lo - 1, 0), i, lo + (7 * i) % (i + 1 - lo))[i % 4]
                q[i, :, :d] += k[j] * (30.0 / spec.scale / k[j].square().sum(-1, keepdim=True))
            raw = raw.to(dtype).double()
            q = raw[:, :H_ * (d + r)].view(T, H_, d + r)
            q_rot = plain.rotate_pairs(q[:, :, d:], spec.rot_base)
            k_rot = plain.rotate_pairs(down[:, None, rank:], spec.rot_base)[:, 0]
            v = (c @ w["uv"].T).view(T, H_, dv)
            o = torch.stack([plain.window_attention(
                torch.cat([q[:, h, :d], q_rot[:, h]], 1), torch.cat([k[:, h], k_rot], 1), v[:, h],
                spec.scale, size) for h in range(H_)], 1)
            g = torch.sigmoid(raw[:, seg["g"]:seg["g"] + H_ * dv])
            raws.append(raw.to(dtype).to(device))
            wants.append(o.reshape(T, -1) * g)
        for cuts in CUTS[:1] if rank > 400 else CUTS + (((T, T),),):
            got, _ = drive(lm, raws, cuts, lambda e, layer, raw, out, b, rope: e._latent(
                0, layer, raw, out, b, rope, b.max_ctx))
            for y, want in zip(got, wants):
                err = (y.double().cpu() - want).abs().amax(1) / want.abs().max()
                # a score of 30 rounded to bf16 operands moves weights that are close to one another
                assert float(err.max()) < (tol if dtype == torch.float32 else 0.06), \
                    (spec, int(err.argmax()))
                assert float(err.median()) < tol


def check_mamba2(device, dtype, tol):
    """Convolution, recurrence and output norm, cut at several places; the state at the end."""
    for spec, seed in ((S(6, 7, 10, 3, 5, 2), 1), (S(2, 64, 128, 1, 4, 1), 2), (S(4, 80, 40, 2, 3, 4), 3),
                       (S(3, 9, 200, 1, 1, 3), 4), (S(4, 32, 16, 4, 2, 1), 5), (S(2, 130, 64, 2, 17, 2), 6)):
        lm, w = _mixer(spec, device, dtype, seed)
        layer = lm.layers[0]
        seg, H_, P, N, Gr, T = layer.seg, spec.heads, spec.vdim, spec.state, spec.groups, 210
        raws = [rnd((T, layer.w_in.shape[0]), 10 * seed + s, device, dtype) for s in (0, 1)]
        for raw in raws:
            raw[:, seg["dt"]:] -= 2.0
            for n, m in (("x", H_ * P), ("B", Gr * N), ("C", Gr * N)):     # segments are padded with zeros
                raw[:, seg[n] + m:seg[n] + (m + 7) // 8 * 8] = 0
        for cuts in CUTS:
            got, eng = drive(lm, raws, cuts, lambda e, layer, raw, out, b, rope: e._mamba2(
                0, layer, raw, out, b))
            for s, slot in ((0, 2), (1, 0)):
                r = raws[s].cpu().double()
                z, x, B, C, dt = (r[:, seg[n]:seg[n] + m] for n, m in (
                    ("z", H_ * P), ("x", H_ * P), ("B", Gr * N), ("C", Gr * N), ("dt", H_)))
                conv_in = torch.cat([x, B, C], 1)
                u = plain.silu(plain.causal_conv(conv_in, w["conv"], w["conv.b"]))
                x, B, C = torch.split(u, [H_ * P, Gr * N, Gr * N], 1)
                y, St = plain.ssd_scan(x.view(T, H_, P), B.view(T, Gr, N), C.view(T, Gr, N),
                                       plain.softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
                y = plain.grouped_rms_norm(y.reshape(T, -1) * plain.silu(z), w["norm"], spec.norm_groups,
                                           1e-4)
                assert rel(got[s], y) < tol, (spec, cuts)
                assert rel(eng.state[0, "ssd"][slot, :, :, :P], St) < (2e-5 if dtype == torch.float32 else 5e-3)


def check_mingru(device, dtype, tol):
    for width, seed in ((37, 1), (64, 2), (300, 3)):
        lm, w = _mixer(U(width), device, dtype, seed)
        layer, T = lm.layers[0], 210
        seg = layer.seg
        raws = [2.0 * rnd((T, layer.w_in.shape[0]), 10 * seed + s, device, dtype) for s in (0, 1)]
        for raw in raws:
            raw[:, seg["z"]:seg["z"] + width] -= 2.0
            raw[5, seg["z"]] = 80.0           # a gate that is wide open, and one that is shut
            raw[6, seg["z"]] = -80.0
            raw[7, seg["x"]] = 0.0
            for n in ("z", "x", "g"):
                raw[:, seg[n] + width:seg[n] + (width + 7) // 8 * 8] = 0
        for cuts in CUTS:
            got, eng = drive(lm, raws, cuts, lambda e, layer, raw, out, b, rope: e._mingru(
                0, layer, raw, out, b))
            for s, slot in ((0, 2), (1, 0)):
                z, u, g = (raws[s][:, seg[n]:seg[n] + width].cpu().double() for n in ("z", "x", "g"))
                want = plain.mingru_scan(z, u)
                assert rel(got[s], want * plain.silu(g)) < tol
                assert rel(eng.state[0, "gru"][slot, :width], want[-1]) < 2e-5


MECHANISM_CHECKS = [check_norms_and_shift, check_linear, check_linear_heads, check_latent_attention,
                    check_mamba2, check_mingru]
