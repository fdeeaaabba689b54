"""Plain, slow restatement of the Relulix decoder: one function per mechanism, whole sequences only, no cache, no pages, no
batching, no chunks. The tests compare the framework with it; it shares no code with the package.

A model is ``(cfg, w)``: ``cfg`` the dictionary of a config.json, ``w`` a dictionary of tensors under their checkpoint names
(see :func:`cast`)."""
import math

import torch


def cast(w, dtype=torch.float64):
    return {k: t.to(dtype) for k, t in w.items()}


def rms(x, eps):
    """x divided by its root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    """One learned number for all coordinates."""
    return rms(x, eps) * gain


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---- rotation --------------------------------------------------------------------------------------------------------
def rotation(rot, dtype=torch.float64):
    """(angle per position of every pair, factor of its sine and cosine)."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base**(-2 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return torch.tensor(f, dtype=dtype), 1.0

    def index_with(turns):
        """The (real) index of the pair that makes this many turns within the original length."""
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(index_with(sc["fast"])), 0), min(math.ceil(index_with(sc["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / sc["factor"] * ramp + x * (1 - ramp))
    return torch.tensor(out, dtype=dtype), 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot):
    """x [n, heads, dim] at positions 0..n-1: of the first rot.dims values of each head, i is turned with i + dims / 2."""
    half = rot["dims"] // 2
    freq, factor = rotation(rot, x.dtype)
    ang = (torch.arange(x.shape[0], dtype=x.dtype)[:, None] * freq)[:, None]
    y = x.clone()
    for i in range(half):
        u, v, c, s = x[..., i], x[..., i + half], torch.cos(ang[..., i]) * factor, torch.sin(ang[..., i]) * factor
        y[..., i], y[..., i + half] = u * c - v * s, v * c + u * s
    return y


# ---- retention -------------------------------------------------------------------------------------------------------
def retention_recurrence(q, k, v, decay):
    """S_t = decay S_(t-1) + k_t v_t^T, read by q_t; q, k [n, heads, dim], v [n, heads, vdim], decay [heads]. Returns the read-outs."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def retention_inputs(h, w, p, mx):
    n, H, d = h.shape[0], mx["heads"], mx["dim"]
    q = rotate((h @ w[p + "q"].T).reshape(n, H, d), mx["rot"])
    k = rotate((h @ w[p + "k"].T).reshape(n, H, d), mx["rot"]) * d**-0.5
    return q, k, (h @ w[p + "v"].T).reshape(n, H, mx["vdim"])


def retention(h, w, p, mx, eps):
    q, k, v = retention_inputs(h, w, p, mx)
    o = rms(retention_recurrence(q, k, v, torch.tensor(mx["decay"], dtype=h.dtype)), eps).reshape(h.shape[0], -1)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- attention -------------------------------------------------------------------------------------------------------
def visible(n, size):
    """[n, n] boolean: may the query of a row see the key of a column (``size`` None: every earlier one)."""
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) & (back < (n if size is None else size))


def soft_capped(s, cap):
    return cap * torch.tanh(s / cap)


def softmax_one_more(s, see):
    """Weights [n, n] of one head; a score of zero that has no value stands beside the keys."""
    s = s.masked_fill(~see, -math.inf)
    m = s.max(-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def project(h, w, p, name, heads):
    return (h @ w[p + name].T + w[p + name + ".b"]).reshape(h.shape[0], heads, -1)


def keys_and_values(h, w, p, mx):
    """What a layer caches: rotated keys, and values."""
    return rotate(project(h, w, p, "k", mx["kv_heads"]), mx["rot"]), project(h, w, p, "v", mx["kv_heads"])


def attention(h, w, p, mx, kv):
    k, v = kv
    q = rotate(project(h, w, p, "q", mx["heads"]), mx["rot"])
    group, see = mx["heads"] // mx["kv_heads"], visible(h.shape[0], (mx.get("mask") or {}).get("size"))
    o = []
    for a in range(mx["heads"]):
        s = soft_capped((q[:, a] @ k[:, a // group].T) * mx["scale"], mx["softcap"])
        o.append(softmax_one_more(s, see) @ v[:, a // group])
    return torch.cat(o, -1) @ w[p + "o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def route(h, w, p, top):
    """(chosen experts, their weights), each [n, top]: the largest logits, bias included; softmax over those alone."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best, chosen = torch.topk(z, top, -1)
    e = torch.exp(best - best.max(-1, keepdim=True).values)
    return chosen, e / e.sum(-1, keepdim=True)


def expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def mixture(h, w, p, f):
    chosen, weight = route(h, w, p, f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        for j in range(f["router"]["top"]):
            t = chosen[:, j] == e
            out[t] += weight[t, j, None] * expert(h[t], w, f"{p}e{e}.", f["expert"]["limit"])
    return out


# ---- the model -------------------------------------------------------------------------------------------------------
def residual_stream(cfg, w, tokens):
    """The stream after every layer: a list of [tokens, width]."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    cached, out = {}, []
    for i, lc in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", lc["mixer"]
        h = scalar_norm(x, w[p + "norm1"], eps)
        if lc["type"] == "retention":
            y = retention(h, w, p + "mix.", mx, eps)
        else:
            src = mx.get("kv_from")
            if src is None:
                cached[i] = keys_and_values(h, w, p + "mix.", mx)
            y = attention(h, w, p + "mix.", mx, cached[i if src is None else src])
        if lc["mlp"] is not None:
            y = y + mixture(h, w, p + "mlp.", lc["mlp"])
        x = x + y
        out.append(x)
    return out


def logits(cfg, w, tokens):
    return scalar_norm(residual_stream(cfg, w, tokens)[-1], w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
