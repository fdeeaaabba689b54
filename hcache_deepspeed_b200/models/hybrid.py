"""Layers of stacks that mix attention with recurrent state (``ArchSpec.layers``), for the one executor.

The executor's loop, cache, state manager, batch, capture and restore are those of :class:`RaggedTransformer`; this module
supplies what such a layer does between them, and how its checkpoint pieces are laid out for the kernels:

* ``w_qkv`` stacks every projection that reads the layer's normed input: ``[q heads | k heads | v heads | z | x | B | C | dt]``.
  Decode-size batches run it as ONE GEMM; larger ones as two (the QKV rows keep their fused paged-KV epilogue).
* head sizes are zero padded to the page size of the attention kernels (``AttentionSpec.page_dim``): padded rows of the
  projections make the GEMM itself produce the zeros, padded columns of the output projection ignore them.
* ``w_o`` is ``[attention columns | state-space columns]``: both mixers write into one buffer and ONE GEMM projects and adds
  them. Of their two weights only the ratio is applied there (to the state-space part, in fp32, inside its gated norm); the
  common factor goes into the norm behind the mixer, which reads its input times that factor.
* rows and columns of width ``hidden`` are zero padded to 16-byte rows.
* latent attention: ``w_qkv`` is ``[q heads | latent | rotated key part]``, heads padded to the page size of the attention kernels.
  Short portions and decode steps attend in the latent space (``w_uk`` takes the queries there, ``w_uv`` the results back); prompts
  project the cached rows they see to per-head K / V pages (``w_kv``, whose identity rows copy the rotated part) and use the
  ordinary attention kernels on those.
* a gated delta rule's ``w_qkv`` is ``[gate | v | k | q | decay input | step input]``: the columns of a state-space mixer
  (``[z | x | B | C | dt]``) and one more per head.
* rotated heads: the rows of a head's queries and keys are reordered so that the two values of pair i lie at i and at half the page
  size + i, whatever pairing the design has; values that are not rotated fill the other places with frequency zero. The
  kernels then know one pairing, whole heads, and every page size.
* a minGRU's ``w_qkv`` is ``[gate | candidate | output gate]``; gated linear attention adds ``[q | k | v | gate | decay's first
  projection]`` behind the attention's columns, each padded to 16-byte rows.
* attention on another layer's keys and values: ``w_qkv`` holds the queries alone, the pages are those of that layer.
* retention: ``w_qkv`` = ``[q | k | v | gate]``, heads padded, queries and keys reordered like those of attention. Prompts rotate them
  in the projection's epilogue, decode steps and fp32 models inside the recurrence's kernels.
* two mixers with a norm each: ``w_o`` and ``w_o2`` project their parts of the buffer separately; the norm kernel behind norms both,
  with halved weights, while adding them to the stream.
* ``parallel_residual``: mixer and dense feed-forward read the same norm, so ``w_o`` is ``[mixer columns | feed-forward columns]``
  and ONE GEMM projects and adds both.

The residual stream is fp32. A sublayer leaves ``(output, factor, weight of the norm behind it, if any)`` pending; the next norm
kernel applies that norm, adds to the stream, and norms the stream for its own sublayer in the same pass.
"""
from __future__ import annotations

from typing import Dict, List, NamedTuple, Optional, Tuple

import torch

from ..inference.v2.ragged import RaggedBatchWrapper, RecurrentLayerConfig
from ..inference.v2.ragged.manager_configs import KVCacheConfig
from ..ops.backend import (LatentBuffers, latent_launches, pick_decode_splits, pick_packed_splits, pick_prefill_splits, use_packed_decode,
                           windowed_len)
from ..ops.kernels import ACT_CODES
from .arch import (ArchSpec, AttentionSpec, DeltaSpec, FeedForwardSpec, GRUSpec, LatentAttentionSpec, LayerSpec, LinearAttentionSpec, MixerSpec,
                   RetentionSpec, RotationSpec, StateSpaceSpec)
from .transformer import ACCUM_MAX_TOKENS, RaggedTransformer, ceil_div
from .weights import ExpertWeights, LayerWeights, ModelWeights, interleave_gate_up


def pad8(n: int) -> int:
    return -(-n // 8) * 8


# ---------------------------------------------------------------------------------------------------
# weights
# ---------------------------------------------------------------------------------------------------
def required_pieces(spec: ArchSpec, l: LayerSpec) -> List[str]:
    req = ["norm1.g"] + (["norm1b.g"] if spec.post_norms else [])
    c = l.mixer.latent
    if c is not None:
        req += ["latent." + n for n in ("q", "uk", "uv", "o")] + (["latent.dkv", "latent.norm"] if c.kv_from is None else [])
    if l.mixer.delta is not None:
        req += ["delta." + n for n in ("q", "k", "v", "q_conv", "k_conv", "v_conv", "a", "b", "A_log", "dt_bias", "g", "norm", "o")]
    if l.mixer.attn is not None:
        a = l.mixer.attn
        own = "qkv" if a.kv_from is None else "q"
        req += ["attn." + n for n in own + "o"] + (["attn.g"] if a.gate else []) + (["attn.sink"] if a.sink else [])
        req += ["attn.pb"] if a.weights == "sigmoid" else []
        req += ([f"attn.{n}_b" for n in own] if a.bias else []) + (["attn.o_b"] if a.o_bias else [])
        req += ["attn.q_norm", "attn.k_norm"] if a.qk_norm else []
        req += ["attn.vmix"] if a.v_first is not None else []
    if l.mixer.linear is not None:
        req += ["linear." + n for n in ("q", "k", "v", "g", "a1", "a2", "a2_b", "norm", "o")]
    if l.mixer.normed_mean:
        req += ["attn.out_norm", "linear.out_norm"]
    if l.mixer.gru is not None:
        req += ["gru." + n for n in ("z", "z_b", "x", "x_b", "g", "o")]
    if l.mixer.retention is not None:
        req += ["retention." + n for n in "qkvgo"]
    if l.mixer.ssm is not None:
        req += ["ssm." + n for n in ("in", "conv", "conv_b", "dt_bias", "A_log", "D", "norm", "o")]
    if l.mlp is not None:
        if not spec.parallel_residual:
            req += ["norm2.g"] + (["norm2b.g"] if spec.post_norms else [])
        parts = ("gate", "up", "down") if l.mlp.gated else ("up", "down")
        if l.mlp.experts:
            req += [f"moe.experts.{e}.{n}" for e in range(l.mlp.experts) for n in parts]
            req += {"table": ["moe.table"], "softmax": ["moe.router", "moe.correction"], "sigmoid": ["moe.router"],
                    "chosen": ["moe.router", "moe.router_b"]}[l.mlp.routing]
            if l.mlp.shared_ff:
                req += ["moe.shared." + n for n in parts]
        else:
            req += ["mlp." + n for n in parts]
    return req


def _pad(t: torch.Tensor, dim: int, n: int) -> torch.Tensor:
    if t.shape[dim] == n:
        return t
    shape = list(t.shape)
    shape[dim] = n - t.shape[dim]
    return torch.cat([t, t.new_zeros(shape)], dim=dim)


def _head_rows(w: torch.Tensor, heads: int, d: int, page_dim: int) -> torch.Tensor:
    """[heads * d, K] -> [heads * page_dim, K]"""
    return _pad(w.reshape(heads, d, -1), 1, page_dim).reshape(heads * page_dim, -1)


def rotated_places(a: AttentionSpec) -> torch.Tensor:
    """Place inside a page row of every value of a query or key head."""
    return torch.tensor(a.rot.places(a.dim, a.page_dim), dtype=torch.long)


def _rotated_rows(w: torch.Tensor, heads: int, dim: int, width: int, rot: Optional[RotationSpec]) -> torch.Tensor:
    """Rows (or values) of query or key heads [heads * dim, ...] -> [heads * width, ...], in the kernels' order."""
    flat = w.reshape(heads, dim, -1)
    if rot is None:
        out = _pad(flat, 1, width)
    else:
        out = flat.new_zeros(heads, width, flat.shape[2])
        out[:, torch.tensor(rot.places(dim, width), dtype=torch.long, device=flat.device)] = flat
    return out.reshape((heads * width, ) + tuple(w.shape[1:]))


def _query_rows(w: torch.Tensor, heads: int, a: AttentionSpec) -> torch.Tensor:
    return _rotated_rows(w, heads, a.dim, a.page_dim, a.rot)


def rotation_table(rot: RotationSpec, width: int) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """(angle per position, amplitude) of the value pairs (c, width / 2 + c) of a row, fp64; amplitudes None: all one."""
    n, half = rot.dims // 2, width // 2
    freq = torch.tensor(rot.frequencies() + [0.0] * (half - n), dtype=torch.float64)
    return freq, None if rot.amplitude == 1.0 else torch.tensor([rot.amplitude] * n + [1.0] * (half - n), dtype=torch.float64)


def mixer_factors(m: MixerSpec) -> Tuple[float, float]:
    """(factor of the whole mixer output, weight of the state-space part inside it). The attention part has weight 1 inside
    (its columns of the output projection are dropped when its weight is 0)."""
    if m.ssm is None and m.attn is None or m.normed_mean or m.gru is not None:
        return 1.0, 1.0
    if m.attn is not None and m.attn_weight != 0.0:
        return m.attn_weight, m.ssm_weight / m.attn_weight
    return (m.ssm_weight if m.ssm is not None else 0.0), 1.0


def layer_weights(spec: ArchSpec, l: LayerSpec, p: Dict[str, torch.Tensor], dtype: torch.dtype, device: torch.device) -> LayerWeights:
    """Checkpoint pieces of one layer in the kernels' layout."""
    Hp = spec.padded_hidden

    def to(t: torch.Tensor) -> torch.Tensor:
        return t.to(device=device, dtype=dtype).contiguous()

    def f32(t: torch.Tensor) -> torch.Tensor:
        return t.to(device=device, dtype=torch.float32).contiguous()

    def gamma(name: str) -> torch.Tensor:
        return f32(_pad(norm_weight(spec, p[name]), 0, Hp))

    def ff_weights(prefix: str, ff: int, gated: bool) -> ExpertWeights:
        ffp = pad8(ff)
        up = _pad(p[prefix + "up"], 0, ffp)
        if gated:
            up = interleave_gate_up(_pad(p[prefix + "gate"], 0, ffp), up)
        return ExpertWeights(to(_pad(up, 1, Hp)), to(_pad(_pad(p[prefix + "down"], 1, ffp), 0, Hp)))

    lw = LayerWeights(norm1_g=gamma("norm1.g"))
    if spec.post_norms:
        lw.norm1b_g = gamma("norm1b.g")
    a, m, c, d, g, r = l.mixer.attn, l.mixer.ssm, l.mixer.latent, l.mixer.delta, l.mixer.linear, l.mixer.gru
    rows, cols = [], []
    if c is not None:
        D, R = c.head_width, c.kv_rank
        sign = 0.0 if c.scale == 0 else -1.0 if c.scale < 0 else 1.0      # (as for ordinary attention below)
        rows.append(_head_rows(p["latent.q"] * sign, c.heads, c.dim + c.rot_dim, D))
        if c.kv_from is None:
            rows.append(p["latent.dkv"])
            lw.latent_norm = f32(p["latent.norm"])
        cols.append(_pad(p["latent.o"].reshape(spec.hidden, c.heads, c.vdim), 2, D).reshape(spec.hidden, c.heads * D))
        uk, uv = p["latent.uk"].reshape(c.heads, c.dim, R), p["latent.uv"].reshape(c.heads, c.vdim, R)
        lw.w_uk, lw.w_uv = to(uk), to(uv.transpose(1, 2))
        lw.rot_freq = f32(rotation_frequencies(c.rot_dim, c.rot_base))
        if latent_expands(c, dtype):
            w_k, w_v = uk.new_zeros(c.heads, D, c.page_width), uk.new_zeros(c.heads, D, c.page_width)
            w_k[:, :c.dim, :R] = uk
            w_k[:, c.dim:c.dim + c.rot_dim, R:R + c.rot_dim] = torch.eye(c.rot_dim, dtype=uk.dtype, device=uk.device)
            w_v[:, :c.vdim, :R] = uv
            lw.w_kv = to(torch.cat([w_k, w_v]).reshape(2 * c.heads * D, c.page_width))
    if d is not None:
        rows += [p["delta." + n] for n in ("g", "v", "k", "q", "a", "b")]
        cols.append(_pad(p["delta.o"], 1, pad8(d.inner)))
        lw.ssm_conv_w = f32(torch.cat([p[f"delta.{n}_conv"] for n in "vkq"]).t())
        lw.ssm_conv_b = torch.zeros(d.conv_dim, dtype=torch.float32, device=device)
        lw.ssm_dt_bias, lw.ssm_a = f32(p["delta.dt_bias"]), f32(-torch.exp(p["delta.A_log"].float()))
        lw.ssm_norm = f32(p["delta.norm"].repeat(d.heads))
    if a is not None:
        D = a.page_dim
        # a scale of zero or less cannot be the factor of a running maximum: its sign (or zero) moves into the query rows
        sign = 0.0 if a.scale == 0 else -1.0 if a.scale < 0 else 1.0
        q_sign = 1.0 if a.qk_norm else sign       # (behind a norm it is the norm's weight that carries it)
        rows.append(_query_rows(p["attn.q"] * q_sign, a.heads, a))
        if a.kv_from is None:
            rows += [_query_rows(p["attn.k"], a.kv_heads, a), _head_rows(p["attn.v"], a.kv_heads, a.vdim, D)]
        if a.gate:
            rows.append(_head_rows(p["attn.g"], a.heads, a.vdim, D))
        if a.rot is not None:
            freq, amp = rotation_table(a.rot, D)
            lw.rot_freq, lw.rot_amp = f32(freq), None if amp is None else f32(amp)
        if a.qk_norm:
            lw.q_norm = f32(_query_rows(p["attn.q_norm"].float() * sign, a.heads, a))
            lw.k_norm = f32(_query_rows(p["attn.k_norm"].float(), a.kv_heads, a))
        if a.sink:
            lw.attn_sink = f32(p["attn.sink"])
        elif a.one_more:
            lw.attn_sink = torch.zeros(a.heads, dtype=torch.float32, device=device)
        if a.weights == "sigmoid":
            lw.attn_bias = f32(p["attn.pb"])
        if a.v_first is not None:
            lw.v_mix = f32(p["attn.vmix"].reshape(1))
        o = _pad(p["attn.o"].reshape(spec.hidden, a.heads, a.vdim), 2, D).reshape(spec.hidden, a.heads * D)
        cols.append(o if m is None or l.mixer.attn_weight != 0.0 else torch.zeros_like(o))
    if m is not None:
        rows.append(p["ssm.in"])
        cols.append(_pad(p["ssm.o"], 1, pad8(m.inner)))
        lw.ssm_conv_w, lw.ssm_conv_b = f32(p["ssm.conv"].t()), f32(p["ssm.conv_b"])
        lw.ssm_dt_bias, lw.ssm_a, lw.ssm_d = f32(p["ssm.dt_bias"]), f32(-torch.exp(p["ssm.A_log"].float())), f32(p["ssm.D"])
        lw.ssm_norm = f32(p["ssm.norm"])
    if g is not None:
        g.rank = rank = p["linear.a1"].shape[0]       # (a checkpoint's own; its config does not say)
        rows += [_pad(p["linear." + n], 0, w) for n, w in (("q", g.keys), ("k", g.keys), ("v", g.inner), ("g", g.inner), ("a1", pad8(rank)))]
        lw.w_decay = to(_pad(_pad(p["linear.a2"], 1, pad8(rank)), 0, g.keys))
        lw.decay_bias = f32(p["linear.a2_b"])
        lw.ssm_norm = f32(p["linear.norm"].repeat(g.heads))
        o = _pad(p["linear.o"], 1, g.inner)
        if l.mixer.normed_mean:
            lw.w_o2 = to(_pad(o, 0, Hp))
            lw.mean_g1, lw.mean_g2 = (f32(_pad(p[n].float() * 0.5, 0, Hp)) for n in ("attn.out_norm", "linear.out_norm"))
        else:
            cols.append(o)
    if r is not None:
        rows += [_pad(p["gru." + n], 0, r.inner) for n in "zxg"]
        cols.append(_pad(p["gru.o"], 1, r.inner))
        lw.gru_bias = f32(torch.cat([_pad(p[n], 0, r.inner) for n in ("gru.z_b", "gru.x_b")]))
    t = l.mixer.retention
    if t is not None:
        rows += [_rotated_rows(p["retention." + n], t.heads, t.dim, t.width, t.rot) for n in "qk"]
        rows += [_head_rows(p["retention." + n], t.heads, t.vdim, t.vwidth) for n in "vg"]
        cols.append(_pad(p["retention.o"].reshape(spec.hidden, t.heads, t.vdim), 2, t.vwidth).reshape(spec.hidden, t.inner))
        # (logarithms to base 2 from fp64: a power of the decay is one rounded product away)
        lw.ret_decay = f32(torch.tensor(t.decay, dtype=torch.float64).clamp(min=0).log2().clamp(min=RETENTION_LOG_FLOOR))
        lw.ssm_norm = torch.ones(t.inner, dtype=torch.float32, device=device)
        freq, amp = rotation_table(t.rot or RotationSpec(0, 1.0), t.width)
        lw.rot_freq, lw.rot_amp = f32(freq), None if amp is None else f32(amp)
    lw.w_qkv = to(_pad(torch.cat(rows, dim=0), 1, Hp))
    if a is not None and a.bias:
        b = [_query_rows(p["attn.q_b"] * q_sign, a.heads, a)]
        if a.kv_from is None:
            b += [_query_rows(p["attn.k_b"], a.kv_heads, a), _head_rows(p["attn.v_b"][:, None], a.kv_heads, a.vdim, a.page_dim).reshape(-1)]
        lw.b_qkv = to(_pad(torch.cat(b), 0, lw.w_qkv.shape[0]))
    if a is not None and a.o_bias:
        lw.b_o = to(_pad(p["attn.o_b"], 0, Hp))
    f = l.mlp
    if f is not None:
        if not spec.parallel_residual:
            lw.norm2_g = gamma("norm2.g")
            if spec.post_norms:
                lw.norm2b_g = gamma("norm2b.g")
        if f.experts:
            lw.experts = [ff_weights(f"moe.experts.{e}.", f.ff, f.gated) for e in range(f.experts)]
            lw.stack_experts()
            if f.routing == "table":
                lw.moe_table = p["moe.table"].to(device=device, dtype=torch.int32).contiguous()
            else:
                lw.w_router = to(_pad(_pad(p["moe.router"], 0, pad8(f.experts)), 1, Hp))
                bias = {"softmax": "moe.correction", "chosen": "moe.router_b"}.get(f.routing)
                lw.router_bias = f32(p[bias]) if bias else None
            if f.shared_ff:
                lw.shared_expert = ff_weights("moe.shared.", f.shared_ff, f.gated)
        else:
            dense = ff_weights("mlp.", f.ff, f.gated)
            lw.w_up, lw.w_down = dense.w_up, dense.w_down
            if spec.parallel_residual:
                cols.append(lw.w_down[:spec.hidden].to(cols[0]))
                lw.w_down = None
    lw.w_o = to(_pad(torch.cat(cols, dim=1), 0, Hp))
    return lw


#: log2 of the least decay per token: what it leaves is zero to everything behind it
RETENTION_LOG_FLOOR = -200.0


def norm_weight(spec: ArchSpec, t: torch.Tensor) -> torch.Tensor:
    """A stored norm weight as one value per coordinate."""
    t = spec.norm_weight_offset + t.float()
    return t.reshape(1).expand(spec.hidden) if spec.norm_scalar else t


def rotation_frequencies(dims: int, base: float) -> torch.Tensor:
    """Angle per position of each rotated pair (computed in fp64)."""
    return (float(base)**(-torch.arange(0, dims, 2, dtype=torch.float64) / dims)).float()


def latent_expands(c: LatentAttentionSpec, dtype: torch.dtype) -> bool:
    """Can prompts project cached latents to K / V pages of the tensor-core attention kernels?"""
    return dtype != torch.float32 and c.head_width <= 128


def top_weights(spec: ArchSpec, top: Dict[str, torch.Tensor], out: ModelWeights, dtype: torch.dtype,
                device: torch.device) -> ModelWeights:
    Hp = spec.padded_hidden
    out.embed = _pad(top["embed"], 1, Hp).to(device=device, dtype=dtype).contiguous()

    def gamma(name: str) -> torch.Tensor:
        return _pad(norm_weight(spec, top[name]), 0, Hp).to(device=device).contiguous()

    out.final_norm_g = gamma("final_norm.g")
    if spec.embed_norm:
        if "embed_norm.g" not in top:
            raise ValueError("checkpoint has no norm of the embeddings but the architecture needs one")
        out.embed_norm_g = gamma("embed_norm.g")
    out.lm_head = _pad(top["lm_head"], 1, Hp).to(device=device, dtype=dtype).contiguous() if "lm_head" in top else out.embed
    return out


def random_pieces(spec: ArchSpec, l: LayerSpec, gen: torch.Generator, device: torch.device, std: float = 0.02) -> Dict[str, torch.Tensor]:
    """Random checkpoint pieces of one layer."""
    H = spec.hidden

    def rnd(*shape, scale=std):
        return torch.randn(shape, generator=gen, device=device, dtype=torch.float32) * scale

    def norm_g():
        return 1.0 - spec.norm_weight_offset + rnd(1 if spec.norm_scalar else H, scale=0.05)

    p = {"norm1.g": norm_g(), "norm1b.g": norm_g()}
    a, m, f, c, d, g, r = l.mixer.attn, l.mixer.ssm, l.mlp, l.mixer.latent, l.mixer.delta, l.mixer.linear, l.mixer.gru
    if g is not None:
        kd, vd, rank = g.heads * g.dim, g.heads * g.vdim, g.rank or 16
        p.update({"linear.q": rnd(kd, H), "linear.k": rnd(kd, H), "linear.v": rnd(vd, H), "linear.g": rnd(vd, H), "linear.a1": rnd(rank, H),
                  "linear.a2": rnd(kd, rank, scale=0.3), "linear.a2_b": rnd(kd, scale=0.5) + 2.0, "linear.norm": 1.0 + rnd(g.vdim, scale=0.05),
                  "linear.o": rnd(H, vd)})
    if l.mixer.normed_mean:
        p.update({"attn.out_norm": 1.0 + rnd(H, scale=0.05), "linear.out_norm": 1.0 + rnd(H, scale=0.05)})
    if r is not None:
        p.update({"gru.z": rnd(r.width, H), "gru.z_b": rnd(r.width, scale=0.5) - 1.0, "gru.x": rnd(r.width, H), "gru.x_b": rnd(r.width),
                  "gru.g": rnd(r.width, H), "gru.o": rnd(H, r.width)})
    if c is not None:
        p.update({"latent.q": rnd(c.heads * (c.dim + c.rot_dim), H), "latent.uk": rnd(c.heads * c.dim, c.kv_rank),
                  "latent.uv": rnd(c.heads * c.vdim, c.kv_rank), "latent.o": rnd(H, c.heads * c.vdim)})
        if c.kv_from is None:
            p.update({"latent.dkv": rnd(c.kv_rank + c.rot_dim, H), "latent.norm": 1.0 + rnd(c.kv_rank, scale=0.05)})
    if d is not None:
        kd = d.kv_heads * d.dim
        p.update({"delta.q": rnd(kd, H), "delta.k": rnd(kd, H), "delta.v": rnd(d.inner, H), "delta.g": rnd(d.inner, H),
                  "delta.q_conv": rnd(kd, d.conv, scale=0.3), "delta.k_conv": rnd(kd, d.conv, scale=0.3),
                  "delta.v_conv": rnd(d.inner, d.conv, scale=0.3), "delta.a": rnd(d.heads, H), "delta.b": rnd(d.heads, H),
                  "delta.dt_bias": rnd(d.heads, scale=0.5) - 3.0, "delta.A_log": rnd(d.heads, scale=0.5),
                  "delta.norm": 1.0 + rnd(d.vdim, scale=0.05), "delta.o": rnd(H, d.inner)})
    if a is not None:
        p.update({"attn.q": rnd(a.heads * a.dim, H), "attn.k": rnd(a.kv_heads * a.dim, H), "attn.v": rnd(a.kv_heads * a.vdim, H),
                  "attn.o": rnd(H, a.heads * a.vdim), "attn.g": rnd(a.heads * a.vdim, H), "attn.sink": rnd(a.heads, scale=1.0),
                  "attn.pb": rnd(a.heads, scale=0.5) - 4.0, "attn.vmix": 0.5 + rnd(1, scale=0.1)[0], "attn.q_b": rnd(a.heads * a.dim),
                  "attn.k_b": rnd(a.kv_heads * a.dim), "attn.v_b": rnd(a.kv_heads * a.vdim), "attn.o_b": rnd(H),
                  "attn.q_norm": 1.0 + rnd(a.heads * a.dim, scale=0.05), "attn.k_norm": 1.0 + rnd(a.kv_heads * a.dim, scale=0.05)})
    t = l.mixer.retention
    if t is not None:
        p.update({"retention.q": rnd(t.heads * t.dim, H), "retention.k": rnd(t.heads * t.dim, H), "retention.v": rnd(t.heads * t.vdim, H),
                  "retention.g": rnd(t.heads * t.vdim, H), "retention.o": rnd(H, t.heads * t.vdim)})
    if m is not None:
        p.update({"ssm.in": rnd(m.in_dim, H), "ssm.conv": rnd(m.conv_dim, m.conv, scale=0.3), "ssm.conv_b": rnd(m.conv_dim),
                  "ssm.dt_bias": rnd(m.heads, scale=0.5) - 3.0, "ssm.A_log": rnd(m.heads, scale=0.5), "ssm.D": rnd(m.heads, scale=1.0),
                  "ssm.norm": 1.0 + rnd(m.inner, scale=0.05), "ssm.o": rnd(H, m.inner)})
    if f is not None:
        p.update({"norm2.g": norm_g(), "norm2b.g": norm_g()})

        def glu(prefix, ff):
            p.update({prefix + "up": rnd(ff, H), prefix + "down": rnd(H, ff)})
            if f.gated:
                p[prefix + "gate"] = rnd(ff, H)

        if f.experts:
            for e in range(f.experts):
                glu(f"moe.experts.{e}.", f.ff)
            if f.routing == "table":
                p["moe.table"] = torch.argsort(torch.rand((spec.vocab, f.experts), generator=gen, device=device), dim=1)[:, :f.top].int()
            else:
                p.update({"moe.router": rnd(f.experts, H), "moe.correction": rnd(f.experts, scale=0.05), "moe.router_b": rnd(f.experts, scale=0.05)})
            if f.shared_ff:
                glu("moe.shared.", f.shared_ff)
        else:
            glu("mlp.", f.ff)
    return p


def random_stack_weights(spec: ArchSpec, dtype: torch.dtype, device: torch.device, seed: int = 0, std: float = 0.02) -> ModelWeights:
    gen = torch.Generator(device=device).manual_seed(seed)
    mw = ModelWeights(layers=[layer_weights(spec, l, random_pieces(spec, l, gen, device, std), dtype, device) for l in spec.layers])
    top = {"embed": torch.randn((spec.vocab, spec.hidden), generator=gen, device=device) * std,
           "final_norm.g": 1.0 - spec.norm_weight_offset + torch.randn(1 if spec.norm_scalar else spec.hidden, generator=gen, device=device) * 0.05,
           "embed_norm.g": 1.0 - spec.norm_weight_offset + torch.randn(spec.hidden, generator=gen, device=device) * 0.05,
           "lm_head": torch.randn((spec.vocab, spec.hidden), generator=gen, device=device) * std}
    return top_weights(spec, top, mw, dtype, device)


# ---------------------------------------------------------------------------------------------------
# executor
# ---------------------------------------------------------------------------------------------------
class Pending(NamedTuple):
    """A sublayer's output on its way into the residual stream: stream += norm(factor * delta) * weight, or, without a weight,
    stream += factor * delta. ``delta2``: a second output, added likewise."""
    delta: torch.Tensor
    factor: float
    weight: Optional[torch.Tensor]
    delta2: Optional[torch.Tensor] = None
    weight2: Optional[torch.Tensor] = None


class HybridTransformer(RaggedTransformer):

    def __init__(self, spec: ArchSpec, *args, tp_size: int = 1, **kw) -> None:
        if tp_size > 1:
            raise NotImplementedError(f"{spec.model_type}: layers with recurrent state run on one GPU (no tensor-parallel split)")
        super().__init__(spec, *args, tp_size=tp_size, **kw)

    # ---- geometry ----------------------------------------------------------------------------------
    @property
    def kv_block_size(self) -> int:
        return 64

    def attention_group(self) -> int:
        return max((l.mixer.attn.group for l in self.spec.layers if l.mixer.attn is not None), default=1)

    def kv_cache_config(self) -> Tuple[KVCacheConfig, ...]:
        base = super().kv_cache_config()[0]

        def shape(m: MixerSpec):
            if m.attn is not None:
                return (2, m.attn.kv_heads, m.attn.page_dim) if m.attn.kv_from is None else None
            if m.latent is not None and m.latent.kv_from is None:
                return 1, 1, m.latent.page_width
            return None

        return (base.model_copy(update={"layer_shapes": [shape(l.mixer) for l in self.spec.layers]}), )

    def recurrent_state_config(self):
        if not self.spec.has_recurrent_state:
            return None
        return [None if m is None else RecurrentLayerConfig(heads=m.heads, vdim=m.vwidth if isinstance(m, RetentionSpec) else m.vdim, state=m.state, conv_dim=m.conv_dim, taps=m.conv)
                for m in (l.mixer.recurrent for l in self.spec.layers)]

    def graphable_decode(self, batch: RaggedBatchWrapper) -> bool:
        return True

    def decode_graph_key(self, batch: RaggedBatchWrapper) -> tuple:
        key = [batch.current_sequences, batch.rows_per_small_item]
        for a in {(l.mixer.attn.heads, l.mixer.attn.kv_heads, l.mixer.attn.page_dim, l.mixer.attn.window, l.mixer.attn.keep_first)
                  for l in self.spec.layers if l.mixer.attn is not None}:
            n_q, n_kv, d, window, keep = a
            if batch.n_items_small:
                pick = pick_packed_splits if use_packed_decode(n_q, n_kv, d) else pick_decode_splits
                key.append((a, pick(batch.n_items_small, n_kv, windowed_len(batch.max_kv_len_small, window, keep))))
            if batch.n_items_large:
                key.append((a, pick_prefill_splits(batch.n_items_large, n_q, windowed_len(batch.max_kv_len_large, window, keep))))
        if self.dtype != torch.float32:
            for c in {(c.heads, c.kv_rank, c.page_width, c.window) for c in (l.mixer.latent for l in self.spec.layers) if c is not None}:
                if self.ops.k.latent_attention_supported(c[1], c[2]):
                    key.append((c, latent_launches(batch, *c, batch.n_items_large > 0)))
        return tuple(key)

    def _alloc_buffers(self) -> None:
        s, c = self.spec, self._state_config
        T, S, Hp = c.max_ragged_batch_size, c.max_ragged_sequence_count, s.padded_hidden
        dev, dt = self.device, self.dtype

        def buf(*shape, dtype=dt):
            return torch.zeros(shape, dtype=dtype, device=dev)

        self._tp_fused, self._tp_wait_next, self._tp_scatter_ok = False, False, False
        attn = [l.mixer.attn for l in s.layers if l.mixer.attn is not None]
        latents = [l.mixer.latent for l in s.layers if l.mixer.latent is not None]
        rec = [l.mixer.recurrent for l in s.layers if l.mixer.recurrent is not None]
        mlps = [l.mlp for l in s.layers if l.mlp is not None]
        moes = [f for f in mlps if f.experts]
        self.residual = buf(T, Hp, dtype=torch.float32)
        self.xn, self.xn2 = buf(T, Hp), buf(T, Hp)
        self.latent_buf = buf(s.n_layers, T, Hp) if self.capture_enabled else None
        self.in_buf = buf(T * max(pad8(lw.w_qkv.shape[0]) for lw in self.w.layers))
        self.q_buf = buf(T * max([a.heads * a.page_dim for a in attn] + [c.heads * c.head_width for c in latents] +
                                 [2 * m.keys for m in rec if isinstance(m, RetentionSpec)] + [8]))
        self.mix_buf = buf(T * max(lw.w_o.shape[1] + (lw.w_o2.shape[1] if lw.w_o2 is not None else 0) for lw in self.w.layers))
        self.conv_buf = buf(T * max((pad8(m.conv_dim) for m in rec), default=8))
        self.dt_buf = buf(T * max((m.heads for m in rec), default=1), dtype=torch.float32)
        self.scan_buf = buf(T * max((m.inner for m in rec if not isinstance(m, GRUSpec)), default=1), dtype=torch.float32)
        linear = [m for m in rec if isinstance(m, LinearAttentionSpec)]
        self.decay_buf = buf(T * max((m.keys for m in linear), default=0))
        self.act_buf = buf(T * max([pad8(f.ff) for f in mlps if not f.experts] + [pad8(f.shared_ff) for f in moes] + [8]))
        self._delta_bufs = [buf(T, Hp, dtype=torch.float32)]
        self._delta_idx = 0
        self.delta32 = self._delta_bufs[0]
        self.delta16 = buf(T, Hp)
        two = any(l.mixer.normed_mean for l in s.layers)      # a second pending output
        self.second32, self.second16 = (buf(min(T, ACCUM_MAX_TOKENS), Hp, dtype=torch.float32), buf(T, Hp)) if two else (None, None)
        self.hidden_last = buf(S, Hp)
        self.logits_local = buf(S, self.info.vocab)
        self.logits_full = self.partial16 = self.kv_scratch = None
        self.ws_gemm = self.ws_small = self.ws_large = self.io_stream = None
        self._moe_bufs: Dict[Tuple[int, int, int], dict] = {}
        self._latent_bufs: Optional[LatentBuffers] = None
        self._delta_ws: Optional[torch.Tensor] = None
        self._scan_ws: Optional[torch.Tensor] = None
        if dev.type != "cuda":
            return
        k = self.ops.k
        if latents:
            self._latent_bufs = LatentBuffers(latents, self._state_config, self.kv_block_size, dt, dev)
        n_ws = max([k.gru_workspace_bytes(T, S, m.inner) for m in rec if isinstance(m, GRUSpec)] +
                   [k.retention_workspace_bytes(T, S, m.heads, m.vwidth, m.width) for m in rec if isinstance(m, RetentionSpec) and dt == torch.bfloat16] +
                   [k.linear_attention_workspace_bytes(T, S, m.heads, m.vdim, m.dim) for m in linear if dt == torch.bfloat16], default=0)
        self._scan_ws = torch.empty(n_ws, dtype=torch.uint8, device=dev) if n_ws else None
        if dt != torch.float32:
            n_ws = max((k.delta_workspace_bytes(T, min(S, 64), m.heads, m.kv_heads) for m in rec if isinstance(m, DeltaSpec)), default=0)
            self._delta_ws = torch.empty(n_ws, dtype=torch.uint8, device=dev) if n_ws else None
        for f in moes:
            key = (f.experts, f.top, f.ff)
            if key not in self._moe_bufs:
                rows = k.moe_padded_rows(T, f.experts, f.top)
                self._moe_bufs[key] = dict(
                    scores=buf(T, f.top, dtype=torch.float32), expert_ids=buf(T, f.top, dtype=torch.int32),
                    offsets=buf(T, f.top, dtype=torch.int32), mapped_slots=buf(T, f.top, dtype=torch.int32),
                    counts=buf(f.experts, dtype=torch.int32), pad_off=buf(f.experts + 1, dtype=torch.int32),
                    logits=buf(T, pad8(f.experts), dtype=torch.float32),
                    xs=buf(rows, Hp), hs=buf(rows, pad8(f.ff)), ys=buf(rows, Hp))
        if dt != torch.float32:
            n_max = max([self.info.vocab, Hp] + [lw.w_qkv.shape[0] for lw in self.w.layers] +
                        [w.shape[0] for lw in self.w.layers for w in [lw.w_up, lw.shared_expert and lw.shared_expert.w_up] if w is not None])
            self.ws_gemm = torch.zeros(k.gemm_splitk_workspace_bytes(128, n_max), dtype=torch.uint8, device=dev)
            small, large = 16, 16
            for a in {(a.heads, a.kv_heads, a.page_dim) for a in attn if a.page_dim <= 128}:
                b_small, b_large = self._attention_workspace_bytes(S, *a, rows=8)
                small, large = max(small, b_small), max(large, b_large)
            for c in {(c.heads, c.heads, c.head_width) for c in latents if latent_expands(c, dt)}:
                large = max(large, self._attention_workspace_bytes(S, *c, rows=8)[1])
            self.ws_small = torch.zeros(small, dtype=torch.uint8, device=dev)
            self.ws_large = torch.zeros(large, dtype=torch.uint8, device=dev)
        self._alloc_restore_buffers(T, S, Hp)

    def _view(self, flat: torch.Tensor, T: int, cols: int) -> torch.Tensor:
        return flat[:T * cols].view(T, cols)

    # ---- layer -------------------------------------------------------------------------------------
    def _embed(self, batch: RaggedBatchWrapper) -> torch.Tensor:
        return self.ops.embed_f32(batch.input_ids(), self.w.embed, self.residual[:batch.current_tokens], gamma=self.w.embed_norm_g,
                                  cols=self.spec.hidden, eps=self.spec.norm_eps, scale=self.spec.embed_scale)

    def _norm_into(self, resid: torch.Tensor, gamma: torch.Tensor, out: torch.Tensor, pending: Optional[Pending],
                   keep_resid: bool = True) -> torch.Tensor:
        delta, factor, post, delta2, post2 = pending if pending is not None else (None, 1.0, None, None, None)
        return self.ops.norm_residual(resid, gamma, out, delta=delta, factor=factor, post=post, cols=self.spec.hidden,
                                      eps=self.spec.norm_eps, store_resid=keep_resid, groups=self.spec.norm_groups, delta2=delta2, post2=post2)

    def _layer(self, li: int, resid: torch.Tensor, pending: Optional[Pending], xn: torch.Tensor, batch: RaggedBatchWrapper) -> Pending:
        l, lw, ops, T = self.spec.layers[li], self.w.layers[li], self.ops, batch.current_tokens
        self._norm_into(resid, lw.norm1_g, xn, pending)
        self._kv_ready(li)
        mix = self._view(self.mix_buf, T, lw.w_o.shape[1] + (lw.w_o2.shape[1] if lw.w_o2 is not None else 0))
        if l.mixer.latent is not None:
            n_mix = self._latent_mixer(li, l.mixer.latent, lw, xn, mix, batch)
        elif l.mixer.delta is not None:
            n_mix = self._delta_mixer(li, l.mixer.delta, lw, xn, mix, batch)
        elif l.mixer.gru is not None:
            n_mix = self._gru_mixer(li, l.mixer.gru, lw, xn, mix, batch)
        elif l.mixer.retention is not None:
            n_mix = self._retention_mixer(li, l.mixer.retention, lw, xn, mix, batch)
        else:
            n_mix = self._attention_and_scan(li, l, lw, xn, mix, batch)
        factor, f = mixer_factors(l.mixer)[0], l.mlp
        if self.spec.parallel_residual and f is not None:
            if not f.experts:      # both sublayers' columns meet one output projection
                ops.gemm(xn, lw.w_up, mix[:, n_mix:], act=ACT_CODES[f.act], gated=f.gated, workspace=self.ws_gemm, limit=f.limit)
                return Pending(self._row_parallel(mix, lw.w_o, None, T, force_accum=False), factor, None)
            delta = self._row_parallel(mix, lw.w_o, None, T, force_accum=False)
            return Pending(self._feed_forward(xn, f, lw, T, batch, base=delta), factor, None)
        if l.mixer.normed_mean:
            pending = Pending(self._row_parallel(mix[:, :n_mix], lw.w_o, lw.b_o, T, force_accum=False), factor, lw.mean_g1,
                              self._second_output(mix[:, n_mix:], lw.w_o2, T), lw.mean_g2)
        else:
            pending = Pending(self._row_parallel(mix, lw.w_o, lw.b_o, T, force_accum=False), factor, lw.norm1b_g)
        if f is None:
            return pending
        x2 = self._norm_into(resid, lw.norm2_g, self.xn2[:T], pending)
        return Pending(self._feed_forward(x2, f, lw, T, batch), 1.0, lw.norm2b_g)

    def _attention_and_scan(self, li: int, l: LayerSpec, lw: LayerWeights, xn: torch.Tensor, mix: torch.Tensor,
                            batch: RaggedBatchWrapper) -> int:
        """Attention and / or a recurrent mixer on the same input, side by side in ``mix``; returns their columns (those of the
        attention alone where the other has an output projection of its own)."""
        ops, T, kv = self.ops, batch.current_tokens, self._state_manager
        a, m, g = l.mixer.attn, l.mixer.ssm, l.mixer.linear
        proj = self._view(self.in_buf, T, pad8(lw.w_qkv.shape[0]))
        n_attn = n_out = 0
        if a is not None:
            D = a.page_dim
            n_attn, n_out = (a.heads + 2 * a.cached_heads) * D, a.heads * D
            q = self._view(self.q_buf, T, n_out)
            ops.mixer_in_proj(xn, lw, a, proj, q, kv.get_cache(li), self._first_values(a), batch.tok_pos(), batch.tok_slot(),
                              kv.kv_block_size, self.spec.norm_eps, workspace=self.ws_gemm)
            ops.attention(q, mix[:, :n_out], kv.get_cache(li if a.kv_from is None else a.kv_from), batch, a.heads, a.kv_heads, D,
                          abs(a.scale) or 1.0, ws_small=self.ws_small, ws_large=self.ws_large, window=a.window, keep_first=a.keep_first,
                          sink=lw.attn_sink, sigmoid_bias=lw.attn_bias, gate=proj[:, n_attn:n_attn + n_out] if a.gate else None,
                          softcap=a.softcap)
        else:
            ops.gemm(xn, lw.w_qkv, proj[:, :lw.w_qkv.shape[0]], workspace=self.ws_gemm)
        if g is not None:
            self._linear(li, g, lw, proj[:, n_attn:], batch.spans(), batch.n_single_token_seqs, mix[:, n_out:n_out + g.inner])
            return n_out if l.mixer.normed_mean else n_out + g.inner
        if m is None:
            return n_out
        y = self._scan(li, m, lw, proj[:, n_attn:n_attn + m.in_dim], batch.spans(), batch.n_single_token_seqs)
        ops.gated_norm(y, proj[:, n_attn:n_attn + m.inner], lw.ssm_norm, mix[:, n_out:n_out + m.inner], m.norm_groups,
                       self.spec.norm_eps, mixer_factors(l.mixer)[1])
        return n_out + pad8(m.inner)

    def _latent_mixer(self, li: int, c: LatentAttentionSpec, lw: LayerWeights, xn: torch.Tensor, mix: torch.Tensor,
                      batch: RaggedBatchWrapper) -> int:
        ops, T, kv = self.ops, batch.current_tokens, self._state_manager
        proj = self._view(self.in_buf, T, pad8(lw.w_qkv.shape[0]))
        n_q = c.heads * c.head_width
        q = self._view(self.q_buf, T, n_q)
        cache = kv.get_cache(li if c.kv_from is None else c.kv_from)
        ops.gemm(xn, lw.w_qkv, proj[:, :lw.w_qkv.shape[0]], workspace=self.ws_gemm)
        ops.latent_append(proj, q, cache if c.kv_from is None else None, batch.tok_pos(), batch.tok_slot(), c, lw, self.spec.norm_eps)
        ops.latent_attention(q, mix[:, :n_q], cache, batch, c, lw, self._latent_bufs, ws_large=self.ws_large)
        return n_q

    def _delta_mixer(self, li: int, d: DeltaSpec, lw: LayerWeights, xn: torch.Tensor, mix: torch.Tensor, batch: RaggedBatchWrapper) -> int:
        proj = self._view(self.in_buf, batch.current_tokens, pad8(lw.w_qkv.shape[0]))[:, :d.in_dim]
        self.ops.gemm(xn, lw.w_qkv, proj, workspace=self.ws_gemm)
        self._scan(li, d, lw, proj, batch.spans(), batch.n_single_token_seqs, mix[:, :d.inner])
        return pad8(d.inner)

    def _first_values(self, a: AttentionSpec) -> Optional[torch.Tensor]:
        """Pages of the layer whose values this one mixes in: that layer caches its values as they are, so the share of every token,
        a restored one too, is found there."""
        return None if a.v_first is None else self._state_manager.get_cache(a.v_first)

    def _second_output(self, x: torch.Tensor, w: torch.Tensor, T: int) -> torch.Tensor:
        """As ``_row_parallel``, into buffers of its own."""
        if T <= ACCUM_MAX_TOKENS:
            self.ops.gemm_accum(x, w, self.second32[:T])
            return self.second32[:T]
        return self.ops.gemm(x, w, self.second16[:T])

    def _gru_mixer(self, li: int, r: GRUSpec, lw: LayerWeights, xn: torch.Tensor, mix: torch.Tensor, batch: RaggedBatchWrapper) -> int:
        proj = self._view(self.in_buf, batch.current_tokens, r.in_dim)
        self.ops.gemm(xn, lw.w_qkv, proj, workspace=self.ws_gemm)
        self.ops.gru(proj, lw, r, self._state_manager.recurrent_states.ssm(li), batch.spans(), batch.n_single_token_seqs, mix[:, :r.inner],
                     self._scan_ws)
        return r.inner

    def _retention_mixer(self, li: int, t: RetentionSpec, lw: LayerWeights, xn: torch.Tensor, mix: torch.Tensor, batch: RaggedBatchWrapper) -> int:
        self._retention(li, t, lw, xn, batch.tok_pos(), batch.spans(), batch.n_single_token_seqs, mix[:, :t.inner])
        return t.inner

    def _retention(self, li: int, t: RetentionSpec, lw: LayerWeights, x: torch.Tensor, pos: torch.Tensor, spans: torch.Tensor, n_single: int,
                   out: Optional[torch.Tensor]) -> None:
        """Retention of the tokens whose normed inputs are ``x``; without ``out`` its state alone."""
        T = x.shape[0]
        q, k, v, gate, turned = self.ops.retention_in_proj(x, lw, t, self._view(self.in_buf, T, lw.w_qkv.shape[0]), self._view(self.q_buf, T, 2 * t.keys),
                                                           pos, n_single < spans.shape[0], workspace=self.ws_gemm)
        self.ops.retention(q, k, v, gate, lw, t, turned, self._state_manager.recurrent_states.ssm(li), spans, n_single,
                           self._view(self.scan_buf, T, t.inner), out, self.spec.norm_eps, self._scan_ws)

    def _linear(self, li: int, g: LinearAttentionSpec, lw: LayerWeights, proj: torch.Tensor, spans: torch.Tensor, n_single: int,
                out: Optional[torch.Tensor]) -> None:
        """Gated linear attention of the tokens whose projections are ``proj`` = [q | k | v | gate | decay's first projection]; without
        ``out`` its state alone."""
        T, nk, nv = proj.shape[0], g.keys, g.inner
        low = 2 * nk + 2 * nv
        z = self.ops.gemm(proj[:, low:low + lw.w_decay.shape[1]], lw.w_decay, self._view(self.decay_buf, T, nk), workspace=self.ws_gemm)
        self.ops.linear_attention(proj[:, :nk], proj[:, nk:2 * nk], proj[:, 2 * nk:2 * nk + nv], proj[:, 2 * nk + nv:low], z, lw, g,
                                  self._state_manager.recurrent_states.ssm(li), spans, n_single, self._view(self.scan_buf, T, nv), out,
                                  self.spec.norm_eps, self._scan_ws)

    def _scan(self, li: int, m, lw: LayerWeights, proj: torch.Tensor, spans: torch.Tensor, n_single: int,
              out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Convolution and recurrence of the tokens whose projections are ``proj`` = [z | x | B | C | dt] (delta rule:
        [gate | v | k | q | decay | step]); advances the sequences' state. Returns the recurrence's output (before gate and
        norm), fp32 ``[tokens, inner]``; a delta rule also writes its normed and gated output to ``out`` when given."""
        T, st = proj.shape[0], self._state_manager.recurrent_states
        bufs = (self._view(self.conv_buf, T, pad8(m.conv_dim)), self._view(self.dt_buf, T, m.heads), self._view(self.scan_buf, T, m.inner))
        if isinstance(m, DeltaSpec):
            return self.ops.delta_rule(proj, lw, m, st.ssm(li), st.conv(li), spans, n_single, *bufs, out, self.spec.norm_eps, self._delta_ws)
        return self.ops.state_space(proj, lw, m, st.ssm(li), st.conv(li), spans, n_single, *bufs)

    def _feed_forward(self, x: torch.Tensor, f: FeedForwardSpec, lw: LayerWeights, T: int, batch: RaggedBatchWrapper,
                      base: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``base``: the other sublayer's pending output, which a mixture of experts is added to."""
        ops = self.ops
        act = ACT_CODES[f.act]

        def hidden(w: ExpertWeights):
            h = self._view(self.act_buf, T, w.w_down.shape[1])
            return ops.gemm(x, w.w_up, h, act=act, gated=f.gated, workspace=self.ws_gemm, limit=f.limit)

        if not f.experts:
            return self._row_parallel(hidden(ExpertWeights(lw.w_up, lw.w_down)), lw.w_down, None, T, force_accum=False)
        if lw.shared_expert is not None:
            assert base is None
            base = ops.gemm(hidden(lw.shared_expert), lw.shared_expert.w_down, self.delta16[:T], workspace=self.ws_gemm)
        bufs = self._moe_bufs.get((f.experts, f.top, f.ff))
        if f.routing == "table":
            ops.table_route(batch.input_ids(), lw, f, bufs)
        elif f.routing == "sigmoid":
            ops.sigmoid_route(x, lw, f, bufs)
        elif f.routing == "chosen":
            ops.chosen_route(x, lw, f, bufs)
        else:
            ops.softmax_route(x, lw, f, bufs)
        return ops.routed_experts(x, batch.input_ids(), lw, f, act, base, self.delta32[:T], bufs)

    def _final_hidden(self, resid: torch.Tensor, pending: Optional[Pending], T: int) -> torch.Tensor:
        return self._norm_into(resid, self.w.final_norm_g, self.xn2[:T], pending, keep_resid=False)

    def _drop_pending(self, pending: Optional[Pending], T: int) -> None:
        self.delta32[:T].zero_()
        if self.second32 is not None:
            self.second32[:T].zero_()

    # ---- restore from saved hidden states ------------------------------------------------------------
    def _restore_layer(self, li: int, latents: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, spans: torch.Tensor,
                       n_single: int) -> None:
        """K/V pages as for any layer; the recurrent state by projecting and scanning the saved inputs once more."""
        l, lw, ops, T = self.spec.layers[li], self.w.layers[li], self.ops, latents.shape[0]
        kv = self._state_manager
        a, m, c = l.mixer.attn, l.mixer.recurrent, l.mixer.latent
        n_attn = 0
        proj = self._view(self.in_buf, T, pad8(lw.w_qkv.shape[0]))
        if c is not None and c.kv_from is None:
            part = proj[:, c.heads * c.head_width:lw.w_qkv.shape[0]]
            ops.gemm(latents, lw.w_qkv[c.heads * c.head_width:], part, workspace=self.ws_gemm)
            ops.latent_append(proj, None, kv.get_cache(li), pos, slot, c, lw, self.spec.norm_eps)
        if a is not None and a.kv_from is None:
            n_q = a.heads * a.page_dim
            n_attn = n_q + 2 * a.kv_heads * a.page_dim
            if a.rot is not None or a.qk_norm or a.v_first is not None:
                part = proj[:, n_q:n_attn]
                ops.gemm(latents, lw.w_qkv[n_q:n_attn], part, bias=None if lw.b_qkv is None else lw.b_qkv[n_q:n_attn], workspace=self.ws_gemm)
                ops.attention_append(part, lw, a, None, kv.get_cache(li), self._first_values(a), pos, slot, kv.kv_block_size, self.spec.norm_eps)
            else:
                ops.restore_kv_proj(latents, lw.w_qkv[n_q:n_attn], None, kv.get_cache(li), pos, slot, None, a.kv_heads, a.page_dim,
                                    a.page_dim, kv.kv_block_size, scratch=proj[:, n_q:n_attn])
        if isinstance(m, GRUSpec):
            ops.gemm(latents, lw.w_qkv, proj, workspace=self.ws_gemm)
            ops.gru(proj, lw, m, kv.recurrent_states.ssm(li), spans, n_single, None, self._scan_ws)
        elif isinstance(m, RetentionSpec):
            self._retention(li, m, lw, latents, pos, spans, n_single, None)
        elif isinstance(m, LinearAttentionSpec):
            ops.gemm(latents, lw.w_qkv[n_attn:], proj[:, n_attn:], workspace=self.ws_gemm)
            self._linear(li, m, lw, proj[:, n_attn:], spans, n_single, None)
        elif m is not None:
            part = proj[:, n_attn:n_attn + m.in_dim]
            ops.gemm(latents, lw.w_qkv[n_attn:], part, workspace=self.ws_gemm)
            self._scan(li, m, lw, part, spans, n_single)
