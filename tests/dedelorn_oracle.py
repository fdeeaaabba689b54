"""Plain, slow restatement of the Dedelorn decoder: one function per mechanism, whole sequences only, no cache, no pages,
no batching, no chunks. The tests compare the framework with it; it shares no code with the package.

A model is ``(cfg, w)``: ``cfg`` the dictionary of a config.json, ``w`` a dictionary of tensors under their checkpoint names
(see :func:`cast`)."""
import math

import torch

#: added under the root that makes a query or key of the delta rule a unit vector
UNIT_EPS = 1e-6


def cast(w, dtype=torch.float64):
    return {k: t.to(dtype) for k, t in w.items()}


def rms(x, eps):
    """x divided by its root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z**3)))


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


# ---- gated delta rule ------------------------------------------------------------------------------------------------
def causal_conv(u, taps):
    """Per-channel causal convolution, ``taps`` [channels, taps]: the last column meets the current token."""
    n, K = u.shape[0], taps.shape[1]
    padded = torch.cat([u.new_zeros(K - 1, u.shape[1]), u])
    return sum(padded[j:j + n] * taps[:, j] for j in range(K))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_recurrence(q, k, v, g, beta):
    """q, k [n, heads, dim] (unit vectors, q scaled), v [n, heads, vdim], g and beta [n, heads]. Every token first lets the
    state fade, then moves what the key reads out of it towards v by the share beta, then reads with the query. Returns the
    read-outs [n, heads, vdim] and the last state [heads, dim, vdim]."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def delta_inputs(h, w, p, mx):
    """(q, k, v, g, beta) of :func:`delta_recurrence` from the mixer's input."""
    n, H, G, d, dv = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + x].T, w[p + x + ".conv"])) for x in "qkv")
    of = torch.arange(H) // (H // G)
    q = (unit(q.reshape(n, G, d)) * d**-0.5)[:, of]
    k = unit(k.reshape(n, G, d))[:, of]
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    return q, k, v.reshape(n, H, dv), g, beta


def norm_then_gate(o, z, w, eps):
    """o [n, heads, vdim] by its own root mean square per head, times the weight shared by the heads, times silu of the gate."""
    return (rms(o, eps) * w).reshape(z.shape) * silu(z)


def delta(h, w, p, mx, eps):
    o, _ = delta_recurrence(*delta_inputs(h, w, p, mx))
    return norm_then_gate(o, h @ w[p + "g"].T, w[p + "norm"], eps) @ w[p + "o"].T


# ---- latent attention ------------------------------------------------------------------------------------------------
def rotate_pairs(x, base):
    """x [n, ..., dims]: the pair (2i, 2i + 1) turned by position * base^(-2i / dims)."""
    n, dims = x.shape[0], x.shape[-1]
    ang = torch.arange(n, dtype=x.dtype)[:, None] * base**(-torch.arange(0, dims, 2, dtype=x.dtype) / dims)
    ang = ang.reshape((n, ) + (1, ) * (x.dim() - 2) + (-1, ))
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * torch.cos(ang) - v * torch.sin(ang), v * torch.cos(ang) + u * torch.sin(ang)], -1).flatten(-2)


def visible(n, size):
    """[n, n] boolean: may the query of a row see the key of a column (``size`` None: every earlier one)."""
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) & (back < (n if size is None else size))


def latent_of(h, w, p, mx, eps):
    """What a layer caches of every token: the normed latent [n, kv_rank] and the rotated key part [n, rot_dim]."""
    y = h @ w[p + "dkv"].T
    R = mx["kv_rank"]
    return rms(y[:, :R], eps) * w[p + "dkv.norm"], rotate_pairs(y[:, R:], mx["rot"]["base"])


def latent_attention(h, w, p, mx, latent):
    n, H, d, dr, dv = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    c, kr = latent
    q = (h @ w[p + "q"].T).reshape(n, H, d + dr)
    qr = rotate_pairs(q[..., d:], mx["rot"]["base"])
    k = (c @ w[p + "uk"].T).reshape(n, H, d)
    v = (c @ w[p + "uv"].T).reshape(n, H, dv)
    see = visible(n, (mx.get("mask") or {}).get("size"))
    heads = []
    for a in range(H):
        s = (q[:, a, :d] @ k[:, a].T + qr[:, a] @ kr.T) * mx["scale"]
        s = s.masked_fill(~see, -math.inf)
        s = torch.exp(s - s.max(-1, keepdim=True).values)
        heads.append(s / s.sum(-1, keepdim=True) @ v[:, a])
    return torch.cat(heads, -1) @ w[p + "o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, router):
    """(chosen experts, their weights), each [n, top]: chosen by softmax score + correction, weighted by score * scale."""
    s = torch.softmax(h @ w[p + "router"].T, -1)
    chosen = torch.topk(s + w[p + "correction"], router["top"], -1).indices
    return chosen, s.gather(-1, chosen) * router["scale"]


def expert(h, w, p):
    return gelu_erf(h @ w[p + "up"].T) @ w[p + "down"].T


def mixture(h, w, p, router):
    chosen, weight = route(h, w, p, router)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, f in zip(chosen[t].tolist(), weight[t]):
            out[t] += f * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


def feed_forward(h, w, p, mlp):
    if mlp is None:
        return torch.zeros_like(h)
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp["router"])


# ---- the model -------------------------------------------------------------------------------------------------------
def residual_stream(cfg, w, tokens):
    """The stream after every layer: a list of [tokens, width]. Both sublayers of a layer read the same norm."""
    eps = cfg["norm"]["eps"]
    x = rms(w["embed"][tokens], eps) * w["embed.norm"]
    latents, out = {}, []
    for i, lc in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", lc["mixer"]
        h = rms(x, eps) * w[p + "norm1"]
        if lc["type"] == "delta":
            y = delta(h, w, p + "mix.", mx, eps)
        else:
            latents[i] = latents[mx["kv_from"]] if mx.get("kv_from") is not None else latent_of(h, w, p + "mix.", mx, eps)
            y = latent_attention(h, w, p + "mix.", mx, latents[i])
        x = x + (y + feed_forward(h, w, p + "mlp.", lc["mlp"]))
        out.append(x)
    return out


def logits(cfg, w, tokens):
    x = residual_stream(cfg, w, tokens)[-1]
    return (rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T
