"""Plain, slow restatement of the Lotelix decoder: one function per mechanism, whole sequences only, no cache, no pages,
no batching, no chunks. The tests compare the framework with it; it shares no code with the package.

A model is ``(cfg, w)``: ``cfg`` the dictionary of a config.json, ``w`` a dictionary of tensors under their checkpoint names
(see :func:`cast`)."""
import math

import torch


def cast(w, dtype=torch.float64):
    return {k: t.to(dtype) for k, t in w.items()}


def rms(x, eps):
    """x divided by its root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_rms(x, groups, eps):
    """Each of ``groups`` equal consecutive parts of x divided by its own root mean square."""
    return rms(x.reshape(*x.shape[:-1], groups, -1), eps).reshape(x.shape)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---- minGRU ----------------------------------------------------------------------------------------------------------
def gru_recurrence(z, c):
    """S_t = (1 - z_t) S_(t-1) + z_t c_t element by element from S = 0; z, c [n, width]. Returns every S_t."""
    S, out = torch.zeros_like(z[0]), []
    for t in range(z.shape[0]):
        S = (1 - z[t]) * S + z[t] * c[t]
        out.append(S)
    return torch.stack(out)


def gru_inputs(h, w, p):
    z = sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    u = h @ w[p + "x"].T + w[p + "x.b"]
    return z, torch.where(u >= 0, u + 0.5, sigmoid(u))


def mingru(h, w, p):
    return (gru_recurrence(*gru_inputs(h, w, p)) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- rotation --------------------------------------------------------------------------------------------------------
def frequencies(rot, dtype=torch.float64):
    """Angle per position of each rotated pair; long wavelengths are slowed down when the rotation is scaled."""
    f = float(rot["base"])**(-2 * torch.arange(rot["dims"] // 2, dtype=dtype) / rot["dims"])
    sc = rot.get("scaling")
    if sc is None:
        return f
    out = []
    for x in f.tolist():
        wave = 2 * math.pi / x
        if wave < sc["original"] / sc["high"]:
            out.append(x)
        elif wave > sc["original"] / sc["low"]:
            out.append(x / sc["factor"])
        else:
            s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1 - s) * x / sc["factor"] + s * x)
    return torch.tensor(out, dtype=dtype)


def rotate(x, rot, interleaved):
    """x [n, heads, dim] at positions 0..n-1: the first rot.dims values of each head turned pair by pair."""
    n, half = x.shape[0], rot["dims"] // 2
    ang = (torch.arange(n, dtype=x.dtype)[:, None] * frequencies(rot, x.dtype))[:, None]
    y = x.clone()
    for i in range(half):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        u, v, c, s = x[..., a], x[..., b], torch.cos(ang[..., i]), torch.sin(ang[..., i])
        y[..., a], y[..., b] = u * c - v * s, v * c + u * s
    return y


# ---- attention -------------------------------------------------------------------------------------------------------
def visible(n, size):
    """[n, n] boolean: may the query of a row see the key of a column (``size`` None: every earlier one)."""
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) & (back < (n if size is None else size))


def softmax_with_sink(s, see, sink):
    """Weights [n, n] of one head; ``sink`` is one more score in the denominator."""
    s = s.masked_fill(~see, -math.inf)
    m = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def sigmoid_weights(s, see, bias):
    return sigmoid(s + bias) * see


def attention_inputs(h, w, p, mx, v_first=None):
    """(q, k, v) of a windowed layer [n, heads, .], rotated, the values mixed with those of the first mixing layer."""
    n = h.shape[0]
    q = (h @ w[p + "q"].T).reshape(n, mx["heads"], mx["dim"])
    k = (h @ w[p + "k"].T).reshape(n, mx["kv_heads"], mx["dim"])
    v = (h @ w[p + "v"].T).reshape(n, mx["kv_heads"], mx["vdim"])
    if v_first is not None:
        v = (1 - w[p + "vmix"]) * v + w[p + "vmix"] * v_first
    return rotate(q, mx["rot"], False), rotate(k, mx["rot"], False), v


def attend(q, k, v, scale, weights):
    """Heads side by side; ``weights(head, scores)`` turns the scores of a head into weights."""
    group = q.shape[1] // k.shape[1]
    return torch.cat([weights(a, (q[:, a] @ k[:, a // group].T) * scale) @ v[:, a // group] for a in range(q.shape[1])], -1)


def attention(h, w, p, mx, v_first=None):
    """Returns the mixer's output and its values."""
    q, k, v = attention_inputs(h, w, p, mx, v_first)
    see = visible(h.shape[0], (mx.get("mask") or {}).get("size"))
    o = attend(q, k, v, mx["scale"], lambda a, s: softmax_with_sink(s, see, w[p + "sink"][a]))
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T, v


# ---- two mixers side by side -----------------------------------------------------------------------------------------
def sigmoid_attention(h, w, p, mx, eps):
    n = h.shape[0]
    q, k, v = (h @ w[p + x].T + w[p + x + ".b"] for x in "qkv")
    q = (rms(q, eps) * w[p + "q.norm"]).reshape(n, mx["heads"], mx["dim"])
    k = (rms(k, eps) * w[p + "k.norm"]).reshape(n, mx["kv_heads"], mx["dim"])
    see = visible(n, None)
    o = attend(rotate(q, mx["rot"], True), rotate(k, mx["rot"], True), v.reshape(n, mx["kv_heads"], mx["vdim"]), mx["scale"],
               lambda a, s: sigmoid_weights(s, see, w[p + "pb"][a]))
    return o @ w[p + "o"].T + w[p + "o.b"]


def linear_recurrence(q, k, v, alpha):
    """S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, read by q_t; q, k, alpha [n, heads, dim], v [n, heads, vdim]. Returns the read-outs."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def linear_inputs(h, w, p, mx):
    n, H, d = h.shape[0], mx["heads"], mx["dim"]
    q = (h @ w[p + "q"].T).reshape(n, H, d) * d**-0.5
    k, v = (h @ w[p + "k"].T).reshape(n, H, d), (h @ w[p + "v"].T).reshape(n, H, mx["vdim"])
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    return q, k, v, (sigmoid(z)**(1 / mx["tau"])).reshape(n, H, d)


def linear_attention(h, w, p, mx, eps):
    o = rms(linear_recurrence(*linear_inputs(h, w, p, mx)), eps) * w[p + "norm"]
    g = h @ w[p + "g"].T
    return (o.reshape(g.shape) * silu(g)) @ w[p + "o"].T


def parallel(h, w, p, mx, eps):
    left, right = sigmoid_attention(h, w, p + "left.", mx["left"], eps), linear_attention(h, w, p + "right.", mx["right"], eps)
    return (rms(left, eps) * w[p + "left.out"] + rms(right, eps) * w[p + "right.out"]) / 2


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def route(h, w, p, router):
    """(chosen experts, their weights), each [n, top]: the largest sigmoid scores, which are the weights as they are."""
    s = sigmoid(h @ w[p + "router"].T)
    chosen = torch.topk(s, router["top"], -1).indices
    return chosen, s.gather(-1, chosen)


def expert(h, w, p):
    return torch.clamp(h @ w[p + "up"].T, min=0)**2 @ w[p + "down"].T


def mixture(h, w, p, router):
    """A token's weight for an expert multiplies what the expert reads."""
    chosen, weight = route(h, w, p, router)
    out = torch.zeros_like(h)
    for e in range(w[p + "router"].shape[0]):
        for j in range(router["top"]):
            t = chosen[:, j] == e
            out[t] += expert(weight[t, j, None] * h[t], w, f"{p}e{e}.")
    return out


# ---- the model -------------------------------------------------------------------------------------------------------
def norm(x, w, cfg):
    return grouped_rms(x, cfg["norm"]["groups"], cfg["norm"]["eps"]) * w


def residual_stream(cfg, w, tokens):
    """The stream after every layer: a list of [tokens, width]."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    v_first, out = None, []
    for i, lc in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", lc["mixer"]
        h = norm(x, w[p + "norm1"], cfg)
        if lc["type"] == "mingru":
            y = mingru(h, w, p + "mix.")
        elif lc["type"] == "parallel":
            y = parallel(h, w, p + "mix.", mx, eps)
        else:
            y, v = attention(h, w, p + "mix.", mx, v_first if mx.get("v_mix") else None)
            if mx.get("v_mix") and v_first is None:
                v_first = v
        x = x + y
        if lc["mlp"] is not None:
            x = x + mixture(norm(x, w[p + "norm2"], cfg), w, p + "mlp.", lc["mlp"]["router"])
        out.append(x)
    return out


def logits(cfg, w, tokens):
    return norm(residual_stream(cfg, w, tokens)[-1], w["final.norm"], cfg) @ w["head"].T
