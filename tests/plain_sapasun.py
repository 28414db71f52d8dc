"""A plain, slow restatement of the Sapasun decoder in double (or single) precision: one function
per mechanism, written from the equations, loops over tokens, no cache and no batching.  The
tests compare the framework with it; it shares no code with the framework.

Notation: ``x [T, width]`` is one sequence's residual stream, ``w`` a mapping from tensor name to
tensor (linear weights ``[out, in]``), ``cfg`` the configuration as a plain dictionary.
"""
import math

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def causal_conv(u, taps):
    """Per-channel causal convolution over time: ``u [T, C]``, ``taps [C, n]``, the last column
    multiplies the current token, tokens before the first are zero."""
    n = taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


def rotate_half(x, dims, base, first_pos=0):
    """Rotary embedding of the first ``dims`` entries of every head of ``x [T, heads, dim]``;
    entry ``i`` is paired with entry ``i + dims/2``."""
    out = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = (first_pos + t) * base ** (-2.0 * i / dims)
            c, s = math.cos(a), math.sin(a)
            u, v = x[t, :, i], x[t, :, i + half]
            out[t, :, i] = u * c - v * s
            out[t, :, i + half] = v * c + u * s
    return out


def chunk_visible(i, j, size):
    """Whether position ``i`` sees position ``j`` under a chunked causal mask."""
    return j <= i and i // size == j // size


def sink_softmax(scores, sink):
    """Weights of a softmax whose denominator also holds ``exp(sink)``."""
    m = torch.maximum(scores.max(), sink)
    e = torch.exp(scores - m)
    return e / (e.sum() + torch.exp(sink - m))


def chunked_attention(q, k, v, scale, sink, size):
    """``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, dv]`` -> ``[T, H, dv]``."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(i + 1) if chunk_visible(i, j, size)]
        for h in range(H):
            s = (k[js, h // per] @ q[i, h]) * scale
            out[i, h] = sink_softmax(s, sink[h]) @ v[js, h // per]
    return out


def attention_mixer(h, w, p, m, v_first):
    """Returns ``(output, v_first)``; ``v_first`` is None until a value-mixing layer has run."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ w[p + n].T, w[p + n + ".conv"]) for n in "qkv")
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv)
    q = rotate_half(q, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_half(k, m["rot"]["dims"], m["rot"]["base"])
    if m.get("v_mix"):
        if v_first is None:
            v_first = v
        else:
            lam = w[p + "vmix"]
            v = (1 - lam) * v + lam * v_first
    o = chunked_attention(q, k, v, m["scale"], w[p + "sink"], m["mask"]["size"])
    gate = torch.sigmoid(h @ w[p + "g"].T)
    o = o * gate[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T, v_first


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def delta_scan(q, k, v, g, beta, state=None):
    """Gated delta rule of one head, token by token: ``q, k, g [T, d]``, ``v [T, dv]``,
    ``beta [T]``; the state is ``[d, dv]``.  Returns ``(o [T, dv], state)``."""
    T, d = q.shape
    S = torch.zeros(d, v.shape[1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out, S


def channel_decay(a, A_log, dt_bias):
    """``a [T, heads, d]`` -> the per-channel decay factors of the same shape."""
    return torch.exp(-torch.exp(A_log)[None, :, None] * softplus(a + dt_bias.view(a.shape[1:])))


def channel_delta_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q, k, v = unit(q.view(T, G, d)) * d ** -0.5, unit(k.view(T, G, d)), v.view(T, H, dv)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = channel_decay((h @ w[p + "a1"].T @ w[p + "a2"].T).view(T, H, d), w[p + "A_log"],
                      w[p + "dt_bias"])
    o = torch.stack([delta_scan(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i],
                                beta[:, i])[0] for i in range(H)], 1)
    gate = torch.sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T).view(T, H, dv)
    o = rms_norm(o, w[p + "norm"], eps) * gate
    return o.reshape(T, H * dv) @ w[p + "o"].T


def feed_forward(h, w, p):
    return torch.relu(h @ w[p + "up"].T).square() @ w[p + "down"].T


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, w, ids, dtype=torch.float64, layers=None):
    """Logits ``[T, vocab]`` of one sequence; ``layers`` (a list) collects the residual stream
    after every layer."""
    w = {n: t.to(dtype) for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = rms_norm(w["embed"][torch.as_tensor(ids)], w["embed.norm"], eps)
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "attention":
            y, v_first = attention_mixer(h, w, p + "mix.", layer["mixer"], v_first)
        else:
            y = channel_delta_mixer(h, w, p + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        x = x + y
        if layers is not None:
            layers.append(x)
    z = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    return soft_cap(z, cfg["logit_softcap"])
