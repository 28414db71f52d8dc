"""A plain, slow restatement of the Rupasun decoder in double (or single) precision: one function per
mechanism, written from the equations, whole sequences, no cache and no batching.  The tests compare
the framework with it; it shares no code with the framework.

Notation: ``x [T, width]`` is one sequence's residual stream, ``w`` a mapping from tensor name to
tensor (linear weights ``[out, in]``), ``cfg`` the configuration as a plain dictionary.
"""
import functools
import math

import torch


def unit_rms(x, eps):
    """``x`` divided by the root mean square of its last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, gain, eps):
    return unit_rms(x, eps) * gain


def _angles(T, dims, base):
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    return torch.arange(T, dtype=torch.float64)[:, None, None] * f


def rotate_halves(x, dims, base):
    """Rotary embedding of the first ``dims`` entries of ``x [T, heads, d]``: entry ``i`` turns together
    with entry ``i + dims/2`` by ``t * base^(-2i/dims)``."""
    a, n = _angles(x.shape[0], dims, base).to(x.dtype), dims // 2
    out = x.clone()
    u, v = x[..., :n], x[..., n:dims]
    out[..., :n] = u * a.cos() - v * a.sin()
    out[..., n:dims] = v * a.cos() + u * a.sin()
    return out


def rotate_pairs(x, dims, base):
    """The same with neighbours: entry ``2i`` turns together with entry ``2i + 1``."""
    a = _angles(x.shape[0], dims, base).to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * a.cos() - v * a.sin()
    out[..., 1:dims:2] = v * a.cos() + u * a.sin()
    return out


def visible(i, j, size=None):
    """Whether position ``i`` sees position ``j``, under a sliding window of ``size`` positions."""
    return j <= i and (size is None or i - j < size)


@functools.lru_cache(maxsize=None)
def visibility(T, size=None):
    return torch.tensor([[visible(i, j, size) for j in range(T)] for i in range(T)])


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def attention(q, k, v, scale, size=None, cap=None):
    """One head: ``q, k [T, d]``, ``v [T, dv]``."""
    s = (q @ k.T) * scale
    if cap is not None:
        s = soft_cap(s, cap)
    s = s.masked_fill(~visibility(q.shape[0], size), -math.inf)
    return torch.softmax(s, -1) @ v


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + diff


def difference(a1, a2, lam, diff, eps):
    """Outputs of the two maps of one head to the head's output."""
    return unit_rms(a1 - lam * a2, eps) * (1 - diff)


def diff_heads(q, k, v, m, lam, eps):
    """``q [T, H, 2, d]``, ``k [T, G, 2, d]`` (rotated), ``v [T, G, dv]``: the heads' outputs."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    o = torch.empty(T, H, v.shape[2], dtype=v.dtype)
    for h in range(H):
        g = h // per
        a1, a2 = (attention(q[:, h, n], k[:, g, n], v[:, g], m["scale"]) for n in (0, 1))
        o[:, h] = difference(a1, a2, lam, m["diff"], eps)
    return o


def diff_attention(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = ((h @ w[p + n].T).view(T, 2 * c, d) for n, c in (("q", H), ("k", G)))
    v = (h @ w[p + "v"].T).view(T, G, dv)
    q, k = (rotate_halves(t, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    lam = difference_weight(*(w[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    o = diff_heads(q.view(T, H, 2, d), k.view(T, G, 2, d), v, m, lam, eps)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def capped_heads(q, k, v, m, eps):
    """``q [T, H, d]``, ``k [T, G, d]`` (rotated), ``v [T, G, dv]``: the heads' outputs, ungated."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    return torch.stack([attention(q[:, h], k[:, h // per], v[:, h // per], m["scale"], m["mask"]["size"],
                                  m["softcap"]) for h in range(H)], 1)


def capped_attention(h, w, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ w[p + n].T).view(T, c, s) for n, c, s in (("q", H, d), ("k", G, d), ("v", G, dv)))
    q, k = (rotate_pairs(t, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    o = capped_heads(q, k, v, m, eps).reshape(T, H * dv) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def dense(h, w, p):
    return torch.relu(h @ w[p + "up"].T).square() @ w[p + "down"].T


def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def expert(h, w, p, limit):
    return clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def choose(z, top, groups, keep, scale):
    """One token's router logits ``z [experts]``: the chosen experts and their weights."""
    s = torch.sigmoid(z)
    n = len(s) // groups
    value = [sum(sorted(s[g * n:(g + 1) * n].tolist())[-2:]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -value[g])[:keep]
    allowed = [e for e in range(len(s)) if e // n in kept]
    chosen = sorted(allowed, key=lambda e: -float(s[e]))[:top]
    weight = s[chosen] / (s[chosen].sum() + 1e-20) * scale
    return chosen, weight


def experts(h, w, p, m):
    r = m["router"]
    z = h @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(*choose(z[t], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"])):
            out[t] += c * expert(h[t], w, f"{p}e{e}.", m["expert"]["limit"])
    return out + expert(h, w, p + "shared.", m["shared"]["limit"]) if m.get("shared") else out


MIXERS = {"attention": diff_attention, "attention_2": capped_attention}


def layer(x, w, i, entry, eps):
    p = f"l{i}."
    y = MIXERS[entry["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", entry["mixer"], eps)
    x = x + rms_norm(y, w[p + "norm1b"], eps)
    m = entry.get("mlp")
    if m:
        h = rms_norm(x, w[p + "norm2"], eps)
        y = dense(h, w, p + "mlp.") if m["kind"] == "dense" else experts(h, w, p + "mlp.", m)
        x = x + rms_norm(y, w[p + "norm2b"], eps)
    return x


def forward(cfg, w, tokens, layers=None, dtype=torch.float64):
    """Logits of every position of one sequence; ``layers`` collects the stream after each layer."""
    w = {n: t.to(dtype) for n, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, w, i, entry, eps)
        if layers is not None:
            layers.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
