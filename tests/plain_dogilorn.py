"""A plain, slow restatement of the Dogilorn decoder in double (or single) precision: one function per
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


def layer_norm(x, gain, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * gain + bias


def conv_in(h, taps):
    """``h`` plus its causal convolution over time, channel by channel: ``taps [width, n]``, the last for the
    position itself."""
    T, n = h.shape[0], taps.shape[1]
    out = h.clone()
    for j in range(n):
        back = n - 1 - j
        out[back:] = out[back:] + taps[:, j] * h[:max(T - back, 0)]
    return out


def rotate_pairs(x, dims, base):
    """Rotary embedding of the first ``dims`` entries of ``x [T, heads, d]``: entry ``2i`` turns together
    with entry ``2i + 1`` by ``t * base^(-2i/dims)``."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = (torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f).to(x.dtype)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * a.cos() - v * a.sin()
    out[..., 1:dims:2] = v * a.cos() + u * a.sin()
    return out


def visible(i, j, size=None, keep=0):
    """Whether position ``i`` sees position ``j``, under a sliding window of ``size`` positions beside which the
    first ``keep`` positions stay visible."""
    return (j <= i) & ((i - j < (size or math.inf)) | (j < keep))


@functools.lru_cache(maxsize=None)
def visibility(T, size=None, keep=0):
    i = torch.arange(T)
    return visible(i[:, None], i[None], size, keep)


def weights_beside_one(s):
    """Softmax of the last dimension with one more term ``exp(0)`` in the denominator."""
    top = s.amax(-1, keepdim=True).clamp_min(0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attend(q, k, v, scale, temp, size=None, keep=0):
    """``q [T, H, d]``, ``k [T, G, d]`` (normalised, rotated), ``v [T, G, dv]`` (normalised): the heads'
    outputs ``[T, H, dv]``."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale * temp[h]
        s = s.masked_fill(~visibility(T, size, keep).to(s.device), -math.inf)
        out.append(weights_beside_one(s) @ v[:, h // per])
    return torch.stack(out, 1)


def rotated(t, m):
    r = m.get("rot")
    return rotate_pairs(t, r["dims"], r["base"]) if r else t


def queries(h, w, p, m, eps):
    q = unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    return rotated(q.view(-1, m["heads"], m["dim"]), m)


def keys_values(h, w, p, m, eps):
    k = unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(-1, m["kv_heads"], m["vdim"])
    return rotated(k.view(-1, m["kv_heads"], m["dim"]), m), unit_rms(v, eps)


def attention(h, w, p, m, eps, kv):
    """``kv``: keys and values of the layer that this one shares them with, or None."""
    kv = keys_values(h, w, p, m, eps) if kv is None else kv
    mask = m.get("mask") or {"size": None}
    o = attend(queries(h, w, p, m, eps), *kv, m["scale"], w[p + "temp"], mask["size"], mask.get("keep_first", 0))
    return o.flatten(1) @ w[p + "o"].T, kv


def bounded_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense(h, w, p, m):
    g, u = (h @ w[p + n].T + w[p + n + ".b"] for n in ("gate", "up"))
    return bounded_glu(g, u, m["limit"]) @ w[p + "down"].T + w[p + "down.b"]


def silu_glu(g, u):
    return g * torch.sigmoid(g) * u


def expert(h, w, p):
    return silu_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T) @ w[p + "down"].T


def choose(z, correction, top, groups, keep):
    """One token's router logits ``z``: the chosen experts and their weights."""
    s = torch.softmax(z, -1)
    c = (s + correction).tolist()
    n = len(c) // groups
    value = [max(c[g * n:(g + 1) * n]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -value[g])[:keep]
    chosen = sorted((e for e in range(len(c)) if e // n in kept), key=lambda e: -c[e])[:top]
    return chosen, s[chosen]


def experts(h, w, p, m):
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(*choose(z[t], w[p + "correction"], r["top"], groups["count"], groups["keep"])):
            out[t] += c * (expert(h[t], w, f"{p}e{e}.") if e < r["experts"] else h[t])
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return out


def forward(cfg, w, tokens, layers=None, dtype=torch.float64):
    """Logits of every position of one sequence; ``layers`` collects the stream after each layer."""
    w = {n: t.to(dtype) for n, t in w.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    made = {}
    for i, entry in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", entry["mixer"], entry.get("mlp")
        h = conv_in(norm(x, p + "norm1"), w[p + "canon1"])
        y, made[i] = attention(h, w, p + "mix.", m, eps, made.get(m.get("kv_from")))
        x = x + y * w[p + "ls1"]
        if f:
            h = norm(x, p + "norm2")
            x = x + (dense if f["kind"] == "dense" else experts)(h, w, p + "mlp.", f) * w[p + "ls2"]
        if layers is not None:
            layers.append(x)
    return norm(x, "final.norm") @ w["embed"].T
