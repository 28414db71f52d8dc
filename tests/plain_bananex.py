"""A plain, slow restatement of the Bananex decoder in double (or single) precision: one function
per mechanism, written from the equations, loops over tokens, no cache and no batching.  The
tests compare the framework with it; it shares no code with the framework.

Notation: ``x [T, width]`` is one sequence's residual stream, ``w`` a mapping from tensor name to
tensor (linear weights ``[out, in]``), ``cfg`` the configuration as a plain dictionary.
"""
import math

import torch


def rms_norm(x, gain, eps):
    """``gain`` is one number or a vector over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def grouped_rms_norm(x, weight, groups, eps):
    """The last dimension in ``groups`` equal parts, each by its own root mean square."""
    parts = x.view(*x.shape[:-1], groups, -1)
    return rms_norm(parts, 1.0, eps).reshape(x.shape) * weight


def token_shift(h, amount):
    """``h_t + (h_(t-1) - h_t) * amount``, with zeros before the first token."""
    before = torch.zeros_like(h)
    before[1:] = h[:-1]
    return h + (before - h) * amount


def causal_conv(u, taps, bias):
    """Per-channel causal convolution over time: ``u [T, C]``, ``taps [C, n]``, the last column
    multiplies the current token, tokens before the first are zero."""
    n = taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        y[t] = bias
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] = y[t] + taps[:, j] * u[s]
    return y


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def gelu_erf(x):
    return x * 0.5 * (1 + torch.erf(x / math.sqrt(2.0)))


def rotate_pairs(x, base, first_pos=0):
    """Rotary embedding of all of ``x [T, heads, dims]``: entries ``2i`` and ``2i + 1`` form a pair
    that is turned by ``position * base^(-2i/dims)``."""
    out = x.clone()
    dims = x.shape[-1]
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a = (first_pos + t) * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            out[t, :, 2 * i] = u * c - v * s
            out[t, :, 2 * i + 1] = v * c + u * s
    return out


def window_visible(i, j, size):
    """Whether position ``i`` sees position ``j`` under a sliding causal window."""
    return 0 <= i - j < size


def window_attention(q, k, v, scale, size):
    """One head: ``q, k [T, d]``, ``v [T, dv]``."""
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for i in range(q.shape[0]):
        seen = [j for j in range(max(0, i - size - 1), q.shape[0]) if window_visible(i, j, size)]
        s = (k[seen] @ q[i]) * scale
        out[i] = torch.softmax(s, 0) @ v[seen]
    return out


def latent_attention(h, w, p, m, eps):
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :rank], w[p + "dkv.norm"], eps)
    k_rot = rotate_pairs(down[:, None, rank:], m["rot"]["base"])[:, 0]
    q_rot = rotate_pairs(q[:, :, d:], m["rot"]["base"])
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    size = m["mask"]["size"] if m.get("mask") else T
    o = torch.empty(T, H, dv, dtype=h.dtype)
    for n in range(H):
        o[:, n] = window_attention(torch.cat([q[:, n, :d], q_rot[:, n]], 1),
                                   torch.cat([k[:, n], k_rot], 1), v[:, n], m["scale"], size)
    o = o.reshape(T, H * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def ssd_scan(x, B, C, dt, A_log, D, S=None):
    """``x [T, heads, vdim]``, ``B, C [T, groups, state]``, ``dt [T, heads]`` (after softplus).
    Returns the read-outs and the last state ``[heads, state, vdim]``."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if S is None else S.clone()
    y = torch.empty_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] \
                + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def mamba2(h, w, p, m, eps):
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    T, inner, bc = h.shape[0], H * P, G * N
    z, conv_in, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * bc, H], 1)
    u = silu(causal_conv(conv_in, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(u, [inner, bc, bc], 1)
    dt = softplus(dt + w[p + "dt_bias"])
    y, _ = ssd_scan(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), dt, w[p + "A_log"], w[p + "D"])
    y = grouped_rms_norm(y.reshape(T, inner) * silu(z), w[p + "norm"], m["norm_groups"], eps)
    return y @ w[p + "o"].T


def mingru_scan(zl, u, S=None):
    """``zl, u [T, width]``: logit of the update gate and the raw candidate."""
    S = torch.zeros_like(u[0]) if S is None else S
    out = torch.empty_like(u)
    for t in range(u.shape[0]):
        z = torch.sigmoid(zl[t])
        cand = torch.where(u[t] >= 0, u[t] + 0.5, torch.sigmoid(u[t]))
        S = (1 - z) * S + z * cand
        out[t] = S
    return out


def mingru(h, w, p, m, eps):
    S = mingru_scan(h @ w[p + "z"].T + w[p + "z.b"], h @ w[p + "x"].T + w[p + "x.b"])
    return (S * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mlp(h, w, p):
    return gelu_erf(h @ w[p + "up"].T + w[p + "up.b"]) @ w[p + "down"].T + w[p + "down.b"]


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2, "mingru": mingru}


def layer(x, w, i, entry, eps):
    p = f"l{i}."
    h = token_shift(rms_norm(x, w[p + "norm1"], eps), w[p + "shift"])
    y = MIXERS[entry["type"]](h, w, p + "mix.", entry["mixer"], eps)
    x = x + rms_norm(y, w[p + "norm1b"], eps)
    if entry.get("mlp"):
        y = mlp(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        x = x + rms_norm(y, w[p + "norm2b"], eps)
    return x


def order(cfg):
    """``(layer, number of the pass it starts or None)`` in the order of the runs."""
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, layers=None, dtype=torch.float64):
    """Logits of every position of one sequence; ``layers`` collects the stream after each run."""
    w = {n: t.to(dtype) for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = w["embed"][torch.as_tensor(tokens)]
    for i, start in order(cfg):
        if start is not None:
            x = torch.cat([x, x0], 1) @ w["loop.in"].T + w["loop.step"][start]
        x = layer(x, w, i, cfg["layers"][i], eps)
        if layers is not None:
            layers.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
