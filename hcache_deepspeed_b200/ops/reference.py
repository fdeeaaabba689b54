"""Plain-PyTorch restatements of every device op (fp32 math, device-agnostic).

Two uses: (1) the numerics oracle the GPU kernel tests compare against, (2) the CPU execution
backend of the engines (``init_inference`` on CPU, CPU-only CI). They are never used on a CUDA
device by the framework itself.

The math follows the reference kernels cited in ``include/hds_b200.h``; differences that matter for
tolerances: normalisation statistics and both multiplies are fp32 here (the reference truncates the
reciprocal to the I/O dtype, ``rms_norm_cuda.cu:57,73-74``), RoPE angles are ``pos * inv_freq`` in fp32.
"""
from __future__ import annotations

import math
from typing import Optional

import torch
import torch.nn.functional as F


def apply_act(x: torch.Tensor, act: int) -> torch.Tensor:
    if act == 1:
        return F.gelu(x)
    if act == 2:
        return F.relu(x)
    if act == 3:
        return F.silu(x)
    if act == 4:
        return F.gelu(x, approximate="tanh")
    if act == 6:
        return F.relu(x)**2
    return x


#: sharpness of the sigmoid in the clamped gated unit
CLAMPED_GLU_ALPHA = 1.702


def clamped_glu(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    """Gate bounded above, up bounded on both sides: min(g, L) * sigmoid(alpha * min(g, L)) * (clamp(u, -L, L) + 1)."""
    g = g.clamp(max=limit)
    return g * torch.sigmoid(CLAMPED_GLU_ALPHA * g) * (u.clamp(-limit, limit) + 1.0)


def gemm(a: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, act: int = 0, gated: bool = False,
         out_dtype: Optional[torch.dtype] = None, limit: float = 0.0) -> torch.Tensor:
    y = a.float() @ w.float().t()
    if bias is not None:
        y = y + bias.float()
    if gated and act == 5:
        y = clamped_glu(y[:, 0::2], y[:, 1::2], limit)
    elif gated:
        y = apply_act(y[:, 0::2], act) * y[:, 1::2]
    else:
        y = apply_act(y, act)
    return y.to(out_dtype or a.dtype)


def norm(x: torch.Tensor, gamma: torch.Tensor, beta: Optional[torch.Tensor] = None, eps: float = 1e-5,
         layer_norm: bool = False) -> torch.Tensor:
    xf = x.float()
    if layer_norm:
        mean = xf.mean(-1, keepdim=True)
        var = ((xf - mean) ** 2).mean(-1, keepdim=True)
        y = (xf - mean) * torch.rsqrt(var + eps) * gamma.float()
        if beta is not None:
            y = y + beta.float()
    else:
        y = xf * torch.rsqrt((xf * xf).mean(-1, keepdim=True) + eps) * gamma.float()
    return y.to(x.dtype)


def rope_rotate_half(x: torch.Tensor, pos: torch.Tensor, inv_freq: torch.Tensor, rotary_dim: int) -> torch.Tensor:
    """x: [T, heads, d]; rotate-half RoPE over the first ``rotary_dim`` dims (HF Llama convention)."""
    xf = x.float()
    half = rotary_dim // 2
    ang = pos.float()[:, None] * inv_freq.float()[None, :half]  # [T, half]
    cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
    lo, hi = xf[..., :half], xf[..., half:rotary_dim]
    out = xf.clone()
    out[..., :half] = lo * cos - hi * sin
    out[..., half:rotary_dim] = hi * cos + lo * sin
    return out.to(x.dtype)


def kv_append(kv_cache_layer: torch.Tensor, k: torch.Tensor, v: torch.Tensor, tok_slot: torch.Tensor) -> None:
    """kv_cache_layer: [blocks, 2, kvh, bs, d]; k, v: [T, kvh, d]; tok_slot: [T] (negative = skip)."""
    bs = kv_cache_layer.shape[3]
    valid = tok_slot >= 0
    slots = tok_slot[valid].long()
    blk, off = slots // bs, slots % bs
    kv_cache_layer[blk, 0, :, off, :] = k[valid].to(kv_cache_layer.dtype)
    kv_cache_layer[blk, 1, :, off, :] = v[valid].to(kv_cache_layer.dtype)


def gather_kv(kv_cache_layer: torch.Tensor, block_table_row: torch.Tensor, kv_len: int):
    """Dense K, V ([kv_len, kvh, d]) of one sequence out of the paged cache."""
    bs = kv_cache_layer.shape[3]
    nb = (kv_len + bs - 1) // bs
    blocks = kv_cache_layer[block_table_row[:nb].long()]  # [nb, 2, kvh, bs, d]
    k = blocks[:, 0].permute(0, 2, 1, 3).reshape(nb * bs, blocks.shape[2], blocks.shape[4])[:kv_len]
    v = blocks[:, 1].permute(0, 2, 1, 3).reshape(nb * bs, blocks.shape[2], blocks.shape[4])[:kv_len]
    return k, v


def paged_attention(q: torch.Tensor, kv_cache_layer: torch.Tensor, block_tables: torch.Tensor, items: torch.Tensor,
                    n_q_heads: int, n_kv_heads: int, scale: float, out: Optional[torch.Tensor] = None,
                    alibi: Optional[torch.Tensor] = None, window: int = 0, keep_first: int = 0, sink: Optional[torch.Tensor] = None,
                    sigmoid_bias: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, softcap: float = 0.0) -> torch.Tensor:
    """q: [T, n_q_heads, d]; items: int32 [n, 4] rows (seq, q_row0, n_q, pos0). Causal over absolute positions.
    ``alibi``: [n_q_heads] slopes, score += slope * (key position - query position). ``window`` > 0: a query at position p
    sees the keys (p - window, p] only, and the first ``keep_first`` positions of its sequence. ``sink`` [n_q_heads]: one more
    score in every softmax, without a key. ``sigmoid_bias`` [n_q_heads]: weights are sigmoid(score + bias) instead, not
    normalized. ``gate`` [T, n_q_heads * d]: the output is multiplied by its sigmoid. ``softcap`` > 0: scaled scores are bounded by
    softcap * tanh(score / softcap) before anything else."""
    T, _, d = q.shape
    if out is None:
        out = torch.zeros_like(q)
    G = n_q_heads // n_kv_heads
    for seq, q_row0, n_q, pos0 in items.tolist():
        kv_len = pos0 + n_q
        k, v = gather_kv(kv_cache_layer, block_tables[seq], kv_len)
        k = k.float().repeat_interleave(G, dim=1)  # [kv_len, n_q_heads, d]
        v = v.float().repeat_interleave(G, dim=1)
        qq = q[q_row0:q_row0 + n_q].float()  # [n_q, H, d]
        s = torch.einsum("qhd,khd->hqk", qq, k) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        kv_pos = torch.arange(kv_len, device=q.device)[None, None, :]
        q_pos = (pos0 + torch.arange(n_q, device=q.device))[None, :, None]
        if alibi is not None:
            s = s + alibi.float().to(s.device)[:, None, None] * (kv_pos - q_pos).float()
        s = s.masked_fill(kv_pos > q_pos, float("-inf"))
        if window:
            s = s.masked_fill((kv_pos <= q_pos - window) & (kv_pos >= keep_first), float("-inf"))
        if sigmoid_bias is not None:
            p = torch.sigmoid(s + sigmoid_bias[:, None, None])
        elif sink is not None:
            p = torch.softmax(torch.cat([s, sink[:, None, None].expand(-1, n_q, 1)], dim=-1), dim=-1)[..., :-1]
        else:
            p = torch.softmax(s, dim=-1)
        o = torch.einsum("hqk,khd->qhd", p, v)
        if gate is not None:
            o = o * torch.sigmoid(gate[q_row0:q_row0 + n_q].float().reshape(o.shape))
        out[q_row0:q_row0 + n_q] = o.to(out.dtype)
    return out


def embed(ids: torch.Tensor, weight: torch.Tensor, pos_weight: Optional[torch.Tensor] = None,
          tok_pos: Optional[torch.Tensor] = None, pos_offset: int = 0) -> torch.Tensor:
    out = weight[ids.long().clamp_min(0)].float()
    out = torch.where((ids >= 0)[:, None], out, torch.zeros_like(out))
    if pos_weight is not None:
        p = (tok_pos.long() + pos_offset).clamp(0, pos_weight.shape[0] - 1)
        out = (out.to(weight.dtype).float() + pos_weight[p].float())
    return out.to(weight.dtype)


def default_inv_freq(rotary_dim: int, theta: float = 10000.0, device=None) -> torch.Tensor:
    return 1.0 / (theta ** (torch.arange(0, rotary_dim, 2, dtype=torch.float32, device=device) / rotary_dim))


def alibi_slopes(n_heads: int) -> torch.Tensor:
    """ALiBi head slopes (Press et al.): a geometric sequence for the largest power of two <= n_heads, interleaved with
    the odd terms of the next power's sequence for the remaining heads. fp32 [n_heads]."""
    base = 2 ** math.floor(math.log2(n_heads))
    first = [2.0 ** (-8.0 * (i + 1) / base) for i in range(base)]
    if base < n_heads:
        first += [2.0 ** (-4.0 * (2 * i + 1) / base) for i in range(n_heads - base)]
    return torch.tensor(first, dtype=torch.float32)


def attention_scale(head_dim: int) -> float:
    return 1.0 / math.sqrt(head_dim)


# ---------------------------------------------------------------------------------------------------
# fp32 residual stream with norms on both sides of a sublayer; state-space mixer; expert choice by table
# ---------------------------------------------------------------------------------------------------
def norm_residual(resid: torch.Tensor, gamma: torch.Tensor, delta: Optional[torch.Tensor], factor: float,
                  post: Optional[torch.Tensor], cols: int, eps: float, groups: int = 1, delta2: Optional[torch.Tensor] = None,
                  post2: Optional[torch.Tensor] = None):
    """Returns (new fp32 stream, normed stream): stream += rms(factor * delta) * post (+ rms(delta2) * post2), then
    rms(stream) * gamma, the latter over each of ``groups`` equal parts of a row. Rows hold ``cols`` values and zeros behind them.
    ``post`` None: stream += factor * delta."""

    def rms(d):
        return d * torch.rsqrt((d * d).sum(-1, keepdim=True) / cols + eps)

    x = resid
    if delta is not None:
        d = delta.float() * factor
        x = x + (d if post is None else rms(d) * post)
    if delta2 is not None:
        x = x + rms(delta2.float()) * post2
    if groups == 1:
        return x, rms(x) * gamma
    p = x[:, :cols].reshape(x.shape[0], groups, -1)
    y = (p * torch.rsqrt((p * p).mean(-1, keepdim=True) + eps)).reshape(x.shape[0], cols)
    return x, F.pad(y, (0, x.shape[1] - cols)) * gamma


def gated_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, groups: int, eps: float, scale: float = 1.0,
               gate_after: bool = False) -> torch.Tensor:
    """rms of each of ``groups`` equal parts of y * silu(z), times weight, times scale; with ``gate_after`` the norm is of y alone
    and silu(z) multiplies its result."""
    gate = F.silu(z.float())
    g = y.float() if gate_after else y.float() * gate
    p = g.reshape(g.shape[0], groups, -1)
    out = (p * torch.rsqrt((p * p).mean(-1, keepdim=True) + eps)).reshape(g.shape) * weight * scale
    return out * gate if gate_after else out


def short_conv(u: torch.Tensor, conv_state: torch.Tensor, w: torch.Tensor, b: torch.Tensor, pos0: int) -> torch.Tensor:
    """Causal convolution + silu of ``u`` [n, channels] at positions pos0.. of one sequence; ``w`` [taps, channels].
    ``conv_state`` [taps, channels] is a ring by position modulo taps, advanced in place."""
    taps, n = w.shape[0], u.shape[0]
    past = [conv_state[p % taps] if p >= 0 else torch.zeros_like(u[0], dtype=torch.float32) for p in range(pos0 - taps + 1, pos0)]
    full = torch.cat([torch.stack(past), u.float()]) if past else u.float()
    out = sum(full[k:k + n] * w[k] for k in range(taps)) + b
    for i in range(max(0, n - taps), n):
        conv_state[(pos0 + i) % taps] = u[i].float()
    return F.silu(out)


def selective_scan(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, a: torch.Tensor, d: torch.Tensor,
                   state: torch.Tensor) -> torch.Tensor:
    """S <- exp(a dt) S + dt x B^T, y = S C + d x for every token of one sequence. x [n, heads, P], B / C [n, groups, N],
    dt [n, heads], a / d [heads]; ``state`` [heads, P, N] fp32 is advanced in place."""
    n, H, P = x.shape
    rep = H // B.shape[1]
    y = torch.empty((n, H, P), dtype=torch.float32)
    for t in range(n):
        Bt, Ct = B[t].repeat_interleave(rep, 0), C[t].repeat_interleave(rep, 0)
        xt = x[t].float()
        state.mul_(torch.exp(a * dt[t])[:, None, None]).add_((dt[t][:, None] * xt)[:, :, None] * Bt.float()[:, None, :])
        y[t] = (state * Ct.float()[:, None, :]).sum(-1) + d[:, None] * xt
    return y


#: added under the root when the delta rule's queries and keys are made unit vectors
DELTA_UNIT_EPS = 1e-6


def delta_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, beta: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
    """S <- decay S; S <- S + beta (v - S k) k^T; y = S q for every token of one sequence. q / k [n, groups, N] (as they come out of
    the convolution: made unit vectors here, q also times N^-1/2), v [n, heads, P], decay / beta [n, heads]; ``state``
    [heads, P, N] fp32 is advanced in place."""
    n, H, P = v.shape
    rep, N = H // k.shape[1], k.shape[2]

    def unit(x):
        return x.float() * torch.rsqrt((x.float()**2).sum(-1, keepdim=True) + DELTA_UNIT_EPS)

    q, k = (unit(q) * N**-0.5).repeat_interleave(rep, 1), unit(k).repeat_interleave(rep, 1)
    y = torch.empty((n, H, P), dtype=torch.float32)
    for t in range(n):
        state.mul_(decay[t][:, None, None])
        u = beta[t][:, None] * (v[t].float() - (state * k[t][:, None, :]).sum(-1))
        state.add_(u[:, :, None] * k[t][:, None, :])
        y[t] = (state * q[t][:, None, :]).sum(-1)
    return y


def rotate_pairs(x: torch.Tensor, pos: torch.Tensor, freq: torch.Tensor) -> torch.Tensor:
    """x [T, ..., dims]: the pair (2i, 2i + 1) turned by pos * freq[i]; fp32."""
    ang = (pos.float()[:, None] * freq[None, :]).reshape((x.shape[0], ) + (1, ) * (x.dim() - 2) + (-1, ))
    c, s = ang.cos(), ang.sin()
    u, v = x[..., 0::2].float(), x[..., 1::2].float()
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def latent_rows(y: torch.Tensor, pos: torch.Tensor, rank: int, freq: torch.Tensor, weight: torch.Tensor, eps: float, width: int) -> torch.Tensor:
    """What a token caches, ``[T, width]``: the normed latent, the rotated key part, zeros. ``y`` [T, rank + rot]."""
    c = y[:, :rank].float()
    c = c * torch.rsqrt((c * c).mean(-1, keepdim=True) + eps) * weight
    return F.pad(torch.cat([c, rotate_pairs(y[:, rank:], pos, freq)], 1), (0, width - y.shape[1]))


def paged_latent_attention(q: torch.Tensor, pages: torch.Tensor, block_tables: torch.Tensor, items: torch.Tensor, rank: int, scale: float,
                           window: int = 0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention in the latent space: q [T, heads, rank + rot], pages [blocks, 1, 1, bs, width]; returns the heads' mean latents
    [T, heads, rank]. Items and windows as in :func:`paged_attention`."""
    if out is None:
        out = torch.zeros(q.shape[0], q.shape[1], rank, dtype=q.dtype, device=q.device)
    bs = pages.shape[3]
    for seq, row0, n, pos0 in items.tolist():
        kv_len = pos0 + n
        rows = pages[block_tables[seq, :-(-kv_len // bs)].long(), 0, 0].flatten(0, 1)[:kv_len, :q.shape[2]].float()
        s = torch.einsum("qhd,kd->hqk", q[row0:row0 + n].float(), rows) * scale
        back = (pos0 + torch.arange(n, device=q.device))[:, None] - torch.arange(kv_len, device=q.device)[None, :]
        s = s.masked_fill((back < 0) | (back >= (window or kv_len)), float("-inf"))
        out[row0:row0 + n] = torch.einsum("hqk,kd->qhd", torch.softmax(s, -1), rows[:, :rank]).to(out.dtype)
    return out


def attention_append(qkv: torch.Tensor, kv_cache_layer: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, n_q: int, n_kv: int,
                     freq: Optional[torch.Tensor], q_norm: Optional[torch.Tensor], k_norm: Optional[torch.Tensor], q_cols: int, k_cols: int,
                     eps: float, first: Optional[torch.Tensor], share: Optional[torch.Tensor], amp: Optional[torch.Tensor] = None,
                     head_dim: int = 0) -> torch.Tensor:
    """What lies between a layer's projections ``qkv`` = [q heads | k heads | v heads] and its attention: all of q (k) normed over its
    ``q_cols`` (``k_cols``) values, heads rotated by halves with the angles pos * freq (and times ``amp``), values mixed with those that
    the layer with the pages ``first`` cached of the same tokens. K and V go to their pages; returns q, fp32 [T, n_q * D].
    ``n_kv`` = 0: queries alone, heads of ``head_dim``, no pages."""
    T, D = qkv.shape[0], kv_cache_layer.shape[4] if n_kv else head_dim
    q, k, v = qkv[:, :(n_q + 2 * n_kv) * D].float().split([n_q * D, n_kv * D, n_kv * D], 1)

    def normed(x, w, cols):
        return x if w is None else x * torch.rsqrt((x * x).sum(-1, keepdim=True) / cols + eps) * w

    def rotated(x):
        return x if freq is None else rotate_halves(x, pos, freq, amp)

    if n_kv == 0:
        return rotated(normed(q, q_norm, q_cols).reshape(T, n_q, D)).reshape(T, n_q * D)
    q, k = normed(q, q_norm if n_q else None, q_cols).reshape(T, n_q, D), normed(k, k_norm, k_cols).reshape(T, n_kv, D)
    v = v.reshape(T, n_kv, D)
    if first is not None:
        v = mixed_values(v, first, slot, share)
    kv_append(kv_cache_layer, rotated(k), v, slot)
    return rotated(q).reshape(T, n_q * D)


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, freq: torch.Tensor, amp: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [T, heads, D]: the values c and D / 2 + c turned by pos * freq[c] and multiplied by amp[c]; fp32."""
    y = rope_rotate_half(x.float(), pos, freq, x.shape[-1])
    return y if amp is None else y * torch.cat([amp, amp])


def mixed_values(v: torch.Tensor, first: torch.Tensor, slot: torch.Tensor, share: torch.Tensor) -> torch.Tensor:
    """v [T, n_kv, D] and the values of the same tokens in another layer's pages, by ``share``; widths may be padded differently."""
    bs, s = first.shape[3], slot.long().clamp_min(0)
    n = min(v.shape[2], first.shape[4])
    other = F.pad(first[s // bs, 1, :, s % bs, :n].float(), (0, v.shape[2] - n))
    return (1.0 - share) * v.float() + share * other


def gru_scan(z: torch.Tensor, u: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
    """S <- (1 - sigmoid(z)) S + sigmoid(z) c for every token of one sequence, c = u + 1/2 where u >= 0, else sigmoid(u); z, u
    [n, width], ``state`` [width] fp32 is advanced in place."""
    z, u = torch.sigmoid(z.float()), u.float()
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    out = torch.empty_like(z)
    for t in range(z.shape[0]):
        state.copy_((1.0 - z[t]) * state + z[t] * c[t])
        out[t] = state
    return out


def linear_decay(z: torch.Tensor, tau: float) -> torch.Tensor:
    """sigmoid(z)^(1 / tau)"""
    return torch.exp(F.logsigmoid(z.float()) / tau)


def linear_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
    """S <- S diag(decay) + v k^T, y = S q dim^-1/2 for every token of one sequence; q / k / decay [n, heads, N], v [n, heads, P];
    ``state`` [heads, P, N] fp32 is advanced in place."""
    y = torch.empty(v.shape, dtype=torch.float32)
    q = q.float() * q.shape[2]**-0.5
    for t in range(v.shape[0]):
        state.mul_(decay[t][:, None, :]).add_(v[t].float()[:, :, None] * k[t].float()[:, None, :])
        y[t] = (state * q[t][:, None, :]).sum(-1)
    return y


def retention_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, log2_decay: torch.Tensor, scale: float, state: torch.Tensor) -> torch.Tensor:
    """S <- decay S + v (scale k)^T, y = S q for every token of one sequence; q / k [n, heads, N], v [n, heads, P], log2_decay [heads];
    ``state`` [heads, P, N] fp32 is advanced in place."""
    y, decay = torch.empty(v.shape, dtype=torch.float32), torch.exp2(log2_decay)[:, None, None]
    k = k.float() * scale
    for t in range(v.shape[0]):
        state.mul_(decay).add_(v[t].float()[:, :, None] * k[t][:, None, :])
        y[t] = (state * q[t].float()[:, None, :]).sum(-1)
    return y
