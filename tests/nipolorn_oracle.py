"""Plain, slow restatement of the Nipolorn decoder: one function per mechanism, whole sequences only, no cache, no pages,
no batching. The tests compare the framework with it; it shares no code with the package.

A model is ``(cfg, w)``: ``cfg`` the dictionary of a config.json, ``w`` a dictionary of tensors under their checkpoint names.
Every function takes and returns tensors of one floating type (float64 by default: see :func:`cast`)."""
import math

import torch


def cast(w, dtype=torch.float64):
    """Checkpoint tensors in one floating type (integer tables stay integers)."""
    return {k: (t.to(dtype) if t.is_floating_point() else t.long()) for k, t in w.items()}


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """Root-mean-square norm whose weight is stored as a difference from one."""
    return unit_rms(x, eps) * (1 + w)


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def visible(n, size, keep_first):
    """[n, n] boolean: may the query of a row see the key of a column."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def attention(h, w, p, mx):
    """Grouped-query softmax attention without positions over a sliding window plus the first tokens."""
    n, H, G, d, dv = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = (h @ w[p + "q"].T).reshape(n, H, d)
    k = (h @ w[p + "k"].T).reshape(n, G, d)
    v = (h @ w[p + "v"].T).reshape(n, G, dv)
    see = visible(n, mx["mask"]["size"], mx["mask"]["keep_first"])
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = q[:, a] @ k[:, g].T * mx["scale"]
        s = s.masked_fill(~see, -math.inf)
        s = torch.exp(s - s.max(-1, keepdim=True).values)
        heads.append(s / s.sum(-1, keepdim=True) @ v[:, g])
    return torch.cat(heads, -1) @ w[p + "o"].T


def causal_conv(u, taps, bias):
    """Per-channel causal convolution: the last column of ``taps`` [channels, taps] meets the current token."""
    n, K = u.shape[0], taps.shape[1]
    padded = torch.cat([u.new_zeros(K - 1, u.shape[1]), u])
    return sum(padded[j:j + n] * taps[:, j] for j in range(K)) + bias


def recurrence(x, B, C, dt, A_log, D):
    """x [n, heads, P], B and C [n, groups, N], dt [n, heads] (already positive). Token by token; returns y and the final
    state [heads, N, P]."""
    n, H, P = x.shape
    G, N = B.shape[1], B.shape[2]
    S = x.new_zeros(H, N, P)
    of = torch.arange(H) // (H // G)
    ys = []
    for t in range(n):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t, of][:, :, None] * x[t][:, None, :]
        ys.append((S * C[t, of][:, :, None]).sum(1) + D[:, None] * x[t])
    return torch.stack(ys), S


def gated_group_norm(y, z, w, groups, eps):
    """Gate first, then each of ``groups`` equal parts by its own root mean square, then the weight."""
    g = y * silu(z)
    return unit_rms(g.reshape(g.shape[0], groups, -1), eps).reshape(g.shape) * w


def state_space(h, w, p, mx, eps):
    n, H, P, N, G = h.shape[0], mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * P
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].reshape(n, H, P)
    B = xbc[:, inner:inner + G * N].reshape(n, G, N)
    C = xbc[:, inner + G * N:].reshape(n, G, N)
    y, _ = recurrence(x, B, C, softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(n, inner), z, w[p + "norm"], mx["norm_groups"], eps) @ w[p + "o"].T


def parallel_mixer(h, w, p, mx, eps):
    return (mx["left_scale"] * attention(h, w, p + "left.", mx["left"])
            + mx["right_scale"] * state_space(h, w, p + "right.", mx["right"], eps))


def clamped_mlp(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def table_moe(h, tokens, w, p, mlp):
    """Every token id has its experts in a table; equal weights; an optional shared expert sees every token."""
    top = mlp["router"]["top"]
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens.tolist()):
        for e in w[p + "table"][tok].tolist():
            out[t] += expert(h[t:t + 1], w, f"{p}e{e}.")[0] / top
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.")
    return out


def feed_forward(h, tokens, w, p, mlp):
    if mlp["kind"] == "dense":
        return clamped_mlp(h, w, p, mlp["limit"])
    return table_moe(h, tokens, w, p, mlp)


def layer(x, tokens, w, i, lc, eps):
    p = f"l{i}."
    x = x + norm(parallel_mixer(norm(x, w[p + "norm1"], eps), w, p + "mix.", lc["mixer"], eps), w[p + "norm1b"], eps)
    if lc["mlp"]:
        x = x + norm(feed_forward(norm(x, w[p + "norm2"], eps), tokens, w, p + "mlp.", lc["mlp"]), w[p + "norm2b"], eps)
    return x


def residual_stream(cfg, w, tokens):
    """The stream after every layer: a list of [tokens, width]."""
    x = w["embed"][tokens]
    out = []
    for i, lc in enumerate(cfg["layers"]):
        x = layer(x, tokens, w, i, lc, cfg["norm"]["eps"])
        out.append(x)
    return out


def logits(cfg, w, tokens):
    return norm(residual_stream(cfg, w, tokens)[-1], w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
