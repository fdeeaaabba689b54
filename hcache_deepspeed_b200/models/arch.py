"""Declarative description of a decoder-only transformer family.

The reference spends one ``container.py`` + ``model.py`` + ``policy.py`` per family on parameter
metaprogramming (``deepspeed/inference/v2/model_implementations/{llama_v2,opt,mistral,...}/``,
``layer_container_base.py:42-355``, ``parameter_base.py:54-255``). Here a family is an
:class:`ArchSpec` (what the network looks like) plus a weight-name map (where its tensors live in a
HuggingFace checkpoint); ONE executor (:mod:`hcache_deepspeed_b200.models.transformer`) runs every
spec on the sm_100a kernels.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field, replace
from typing import Any, Callable, Dict, List, Optional


# ---------------------------------------------------------------------------------------------------
# layer descriptions of stacks whose layers are not all alike (ArchSpec.layers)
# ---------------------------------------------------------------------------------------------------
@dataclass
class RotationSpec:
    """Rotation of the first ``dims`` values of every query and key head by position * base^(-2i / dims): value i is paired with
    i + dims / 2, or, ``adjacent``, 2i with 2i + 1. ``slow_factor`` > 0: pairs whose wavelength exceeds ``original / slow_low``
    positions turn slower by that factor, those below ``original / slow_high`` as they are, the ones between by a linear mixture;
    with ``ramp`` that mixture is linear in the pair's index, between the whole indices next to those two wavelengths. ``amplitude``
    multiplies the rotated values."""
    dims: int
    base: float
    adjacent: bool = False
    slow_factor: float = 0.0
    slow_low: float = 1.0
    slow_high: float = 1.0
    original: float = 0.0
    ramp: bool = False
    amplitude: float = 1.0

    def index_of(self, turns: float) -> float:
        """Index of the pair (a real number) that turns this often within ``original`` positions."""
        return self.dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))

    def frequencies(self) -> List[float]:
        out = []
        for i in range(self.dims // 2):
            f = float(self.base)**(-2.0 * i / self.dims)
            if self.slow_factor and self.ramp:
                lo, hi = max(math.floor(self.index_of(self.slow_high)), 0), min(math.ceil(self.index_of(self.slow_low)), self.dims - 1)
                s = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
                f = f / self.slow_factor * s + f * (1.0 - s)
            elif self.slow_factor:
                wave = 2.0 * math.pi / f
                if wave > self.original / self.slow_low:
                    f /= self.slow_factor
                elif wave >= self.original / self.slow_high:
                    s = (self.original / wave - self.slow_low) / (self.slow_high - self.slow_low)
                    f = (1.0 - s) * f / self.slow_factor + s * f
            out.append(f)
        return out

    def places(self, dim: int, width: int) -> List[int]:
        """Place of every value of a head of ``dim`` in rows of ``width`` whose value c is paired with c + width / 2: the values of
        rotated pair i at i and width / 2 + i, the others in what is free."""
        half, n = width // 2, self.dims // 2
        place = [0] * dim
        for i in range(n):
            u, v = (2 * i, 2 * i + 1) if self.adjacent else (i, i + n)
            place[u], place[v] = i, half + i
        place[self.dims:] = [p for p in range(width) if p % half >= n][:dim - self.dims]
        return place


@dataclass
class AttentionSpec:
    """Grouped-query attention. ``window`` > 0: a query at position p sees the keys (p - window, p] and, always, the first
    ``keep_first`` positions of its sequence. Without ``rot`` positions enter through the mask only.

    ``weights`` = "softmax"; with ``sink`` its denominator holds one more term per head, exp of a learned number. "sigmoid": a
    visible key weighs sigmoid(score + a learned number per head), not normalized over keys. ``bias``: q, k and v have
    biases. ``qk_norm``: all of q, and all of k, normed at once before the rotation. ``gate``: the heads are
    multiplied by the sigmoid of one more projection of the layer's input. ``v_first``: values are mixed, by a learned share, with
    the values that this earlier layer caches of the same token (the same heads and sizes).

    ``one_more``: the softmax's denominator holds a one more (a score of zero without a value). ``softcap`` > 0: scores are bounded,
    softcap * tanh(score / softcap). ``o_bias``: the output projection has a bias. ``kv_from``: use the keys and values that this
    earlier layer caches instead of own ones (both layers' heads, sizes and rotation agree)."""
    heads: int
    kv_heads: int
    dim: int                 # query / key size of a head
    vdim: int                # value size of a head
    scale: float
    window: int = 0
    keep_first: int = 0
    rot: Optional[RotationSpec] = None
    weights: str = "softmax"
    sink: bool = False
    bias: bool = False
    qk_norm: bool = False
    gate: bool = False
    v_first: Optional[int] = None
    one_more: bool = False
    softcap: float = 0.0
    o_bias: bool = False
    kv_from: Optional[int] = None

    @property
    def cached_heads(self) -> int:
        """Key / value heads of its own."""
        return 0 if self.kv_from is not None else self.kv_heads

    @property
    def page_dim(self) -> int:
        """Head size of the KV pages (and of q and of the attention output): the kernels' tile sizes 64 and 128, zero
        padded; larger heads are served unpadded (rounded up to 8) by the generic kernel."""
        d = max(self.dim, self.vdim)
        return 64 if d <= 64 else 128 if d <= 128 else -(-d // 8) * 8

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads


@dataclass
class StateSpaceSpec:
    """Mamba-2 mixer: heads of size ``vdim`` with a ``state`` x ``vdim`` recurrent state each; B and C are shared by the
    heads of a group; a causal convolution of ``conv`` taps in front, a gated norm of ``norm_groups`` parts behind."""
    heads: int
    vdim: int
    state: int
    groups: int = 1
    conv: int = 4
    norm_groups: int = 1

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_dim(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @property
    def in_dim(self) -> int:
        """Rows of the input projection: z | x | B | C | dt."""
        return self.inner + self.conv_dim + self.heads


@dataclass
class LatentAttentionSpec:
    """Attention over a shared latent: every token caches one normed vector of ``kv_rank`` values and one rotated key part of
    ``rot_dim`` values, from which each head projects its own key and value. A head's query has ``dim`` unrotated and
    ``rot_dim`` rotated values (adjacent pairs, ``rot_base``). ``window`` as in :class:`AttentionSpec`. ``kv_from``: use what
    that layer caches instead of an own latent (both layers' sizes and rotation agree)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int = 0
    rot_base: float = 10000.0
    kv_from: Optional[int] = None

    @property
    def page_width(self) -> int:
        """Values of a cached token: latent | rotated key part, zero padded to whole 128-byte rows of 16-bit values."""
        return -(-(self.kv_rank + self.rot_dim) // 64) * 64

    @property
    def head_width(self) -> int:
        """Head size of q and of the attention output, and of K / V pages projected from the latents (see AttentionSpec.page_dim)."""
        d = max(self.dim + self.rot_dim, self.vdim)
        return 64 if d <= 64 else 128 if d <= 128 else -(-d // 8) * 8


@dataclass
class DeltaSpec:
    """Gated delta rule: heads with a ``dim`` x ``vdim`` recurrent state each, which fades by a decay per head and is corrected
    along the current key; queries and keys are shared by the value heads of a group (``kv_heads`` groups). A causal
    convolution of ``conv`` taps in front of q, k and v; a norm per head and a gate behind."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int = 4

    @property
    def state(self) -> int:
        return self.dim

    @property
    def groups(self) -> int:
        return self.kv_heads

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_dim(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @property
    def in_dim(self) -> int:
        """Rows of the input projection: gate | v | k | q | decay input | step input."""
        return self.inner + self.conv_dim + 2 * self.heads


@dataclass
class LinearAttentionSpec:
    """Gated linear attention: heads with a ``dim`` x ``vdim`` recurrent state each, whose rows (key channels) fade by a decay of
    their own, sigmoid(z)^(1 / tau), z a projection through ``rank`` values (0: as the checkpoint has it) plus a bias. A norm per
    head and a gate behind."""
    heads: int
    dim: int
    vdim: int
    tau: float = 1.0
    rank: int = 0

    conv = conv_dim = 0

    @property
    def state(self) -> int:
        return self.dim

    @property
    def keys(self) -> int:
        """Columns of all heads' queries (keys, decays), padded to 16-byte rows."""
        return -(-self.heads * self.dim // 8) * 8

    @property
    def inner(self) -> int:
        return -(-self.heads * self.vdim // 8) * 8


@dataclass
class RetentionSpec:
    """Retention: linear attention whose heads' ``dim`` x ``vdim`` states fade by a constant each (``decay``); queries and keys
    rotated by position; a norm per head and a gate behind. Queries and keys are zero padded to the kernels' tile sizes 64 and 128
    (larger ones, and values, to multiples of 16)."""
    heads: int
    dim: int
    vdim: int
    decay: List[float]
    rot: Optional[RotationSpec] = None

    conv = conv_dim = 0

    @property
    def width(self) -> int:
        """Size of a query or key row of a head."""
        return 64 if self.dim <= 64 else 128 if self.dim <= 128 else -(-self.dim // 16) * 16

    @property
    def vwidth(self) -> int:
        return -(-self.vdim // 16) * 16

    @property
    def keys(self) -> int:
        return self.heads * self.width

    @property
    def inner(self) -> int:
        return self.heads * self.vwidth

    @property
    def state(self) -> int:
        return self.width


@dataclass
class GRUSpec:
    """minGRU: ``width`` independent values, S <- (1 - z) S + z c, gate z and candidate c projections of the current token only;
    an output gate behind."""
    width: int

    heads = state = 1
    conv = conv_dim = 0

    @property
    def vdim(self) -> int:
        return self.inner

    @property
    def inner(self) -> int:
        return -(-self.width // 8) * 8

    @property
    def in_dim(self) -> int:
        """Rows of the input projection: z | candidate input | output gate."""
        return 3 * self.inner


@dataclass
class MixerSpec:
    """Token mixer of a layer: attention, a state-space mixer, or both side by side on the same input, each with a weight; or
    latent attention; or a gated delta rule; or a minGRU; or retention; or attention beside gated linear attention, each with an
    output projection and a norm of its own, of which the result is the mean."""
    attn: Optional[AttentionSpec] = None
    ssm: Optional[StateSpaceSpec] = None
    attn_weight: float = 1.0
    ssm_weight: float = 1.0
    latent: Optional[LatentAttentionSpec] = None
    delta: Optional[DeltaSpec] = None
    linear: Optional[LinearAttentionSpec] = None
    gru: Optional[GRUSpec] = None
    retention: Optional[RetentionSpec] = None

    @property
    def recurrent(self):
        """The part with per-sequence state, if any."""
        return next((m for m in (self.ssm, self.delta, self.linear, self.gru, self.retention) if m is not None), None)

    @property
    def normed_mean(self) -> bool:
        """Two outputs, each normed, instead of one?"""
        return self.attn is not None and self.linear is not None


@dataclass
class FeedForwardSpec:
    """``experts`` = 0: dense gated MLP of size ``ff``. Otherwise a mixture of experts of size ``ff`` each, ``top`` per token.
    ``routing`` = "table": a table gives every token id its experts, all with weight 1 / top. ``routing`` = "softmax": the
    largest softmax scores of a router, each plus the expert's correction, choose; the scores themselves times
    ``router_scale`` weigh. ``routing`` = "sigmoid": the largest sigmoid scores choose and weigh; the weight multiplies what the
    expert reads, not what it returns. ``routing`` = "chosen": the largest logits (a bias per expert included) choose, the softmax over
    the chosen ones alone weighs. ``shared_ff`` > 0: one more expert that sees every token. ``gated`` = False: down(act(up x)).
    ``act`` = "swiglu_clamped" clamps gate and up to ``limit`` (see ops.reference)."""
    ff: int
    act: str = "silu"
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    routing: str = "table"
    shared_ff: int = 0
    gated: bool = True
    router_scale: float = 1.0

    @property
    def weighs_inputs(self) -> bool:
        """Does an expert's weight multiply its input instead of its output?"""
        return self.routing == "sigmoid"


@dataclass
class LayerSpec:
    mixer: MixerSpec
    mlp: Optional[FeedForwardSpec] = None


@dataclass
class ArchSpec:
    model_type: str
    n_layers: int
    hidden: int
    n_heads: int
    n_kv_heads: int
    head_dim: int
    intermediate: int
    vocab: int
    # normalisation
    norm: str = "rms"  # "rms" | "layer"
    norm_eps: float = 1e-5
    # MLP
    act: str = "silu"
    gated_mlp: bool = True
    # positions
    pos_emb: str = "rope"  # "rope" | "learned" | "alibi" | "none"
    alibi_scale: float = 1.0  # multiplies the ALiBi slopes (Falcon adds the bias BEFORE its 1/sqrt(d): scale = 1/sqrt(d))
    embed_norm: bool = False  # LayerNorm on the token embeddings (Bloom's word_embeddings_layernorm)
    sliding_window: int = 0  # > 0: a query at position p attends to the keys (p - window, p] (Mistral, Phi-3)
    layer_windows: Optional[List[int]] = None  # per-layer override of sliding_window (GPT-Neo: global / local alternate)
    rope_theta: float = 10000.0
    rotary_dim: Optional[int] = None  # None = head_dim
    rope_scaling: Optional[Dict[str, Any]] = None
    learned_pos_offset: int = 0  # OPT: 2
    max_positions: int = 4096
    # biases
    qkv_bias: bool = False
    attn_out_bias: bool = False
    mlp_bias: bool = False
    lm_head_bias: bool = False
    norm_bias: bool = False  # LayerNorm beta present
    # topology
    parallel_residual: bool = False  # attention and MLP both read the same pre-norm (Falcon, Phi)
    parallel_two_norms: bool = False  # Falcon new architecture: separate norms for the two branches
    tie_word_embeddings: bool = False
    final_norm: bool = True
    attn_scale: Optional[float] = None
    # mixture of experts (0 experts = dense)
    n_experts: int = 0
    top_k: int = 0
    moe_intermediate: int = 0
    shared_expert_intermediate: int = 0  # Qwen2-MoE shared expert (with sigmoid gate)
    norm_topk_prob: bool = True
    #: one entry per layer for stacks of unlike layers; the scalar sizes above then hold the largest values. Such stacks
    #: keep the residual stream in fp32 (models/hybrid.py). With ``parallel_residual`` mixer and feed-forward read one norm
    layers: Optional[List[LayerSpec]] = None
    post_norms: bool = False  # ``layers`` stacks: every sublayer's OUTPUT is normed as well
    norm_weight_offset: float = 0.0  # ``layers`` stacks: stored norm weights are differences from this
    norm_scalar: bool = False  # ``layers`` stacks: the weight of a norm is one number for all coordinates
    norm_groups: int = 1  # ``layers`` stacks: the layers' norms and the final one norm equal consecutive parts of a row, each by itself
    embed_scale: float = 1.0  # ``layers`` stacks: factor of the token embeddings
    extras: Dict[str, Any] = field(default_factory=dict)

    # ---- derived -------------------------------------------------------------------------------
    @property
    def rot_dim(self) -> int:
        return self.rotary_dim if self.rotary_dim is not None else self.head_dim

    @property
    def q_dim(self) -> int:
        return self.n_heads * self.head_dim

    @property
    def kv_dim(self) -> int:
        return self.n_kv_heads * self.head_dim

    @property
    def is_moe(self) -> bool:
        return self.n_experts > 0

    def hidden_state_bytes_per_token_layer(self, elem: int = 2) -> int:
        """Bytes HCache stores per token per layer (the QKV GEMM input)."""
        return self.padded_hidden * elem

    def kv_bytes_per_token_layer(self, elem: int = 2) -> int:
        """Bytes plain KV offload stores per token per layer."""
        return 2 * self.kv_dim * elem

    @property
    def padded_hidden(self) -> int:
        """Row width of the activation buffers of a ``layers`` stack (16-byte rows for every operand type)."""
        return self.hidden if self.layers is None else -(-self.hidden // 8) * 8

    @property
    def has_recurrent_state(self) -> bool:
        return self.layers is not None and any(l.mixer.recurrent is not None for l in self.layers)

    @property
    def pages_hold_context(self) -> bool:
        """Do the K / V pages of a sequence alone bring every layer's context back?"""
        return self.layers is None or (not self.has_recurrent_state and all(
            l.mixer.latent is None and (l.mixer.attn is None or (l.mixer.attn.v_first is None and l.mixer.attn.kv_from is None))
            for l in self.layers))

    def window_of(self, layer: int) -> int:
        return int(self.layer_windows[layer]) if self.layer_windows is not None else int(self.sliding_window)

    def scaled(self, **kw) -> "ArchSpec":
        return replace(self, **kw)

    def param_count(self) -> int:
        h, i = self.hidden, self.intermediate
        if self.layers is not None:
            n = 1 if self.norm_scalar else h
            total = self.vocab * h * (1 if self.tie_word_embeddings else 2) + n
            for l in self.layers:
                a, m, f, c, d = l.mixer.attn, l.mixer.ssm, l.mlp, l.mixer.latent, l.mixer.delta
                total += n * (1 + self.post_norms)
                if a is not None:
                    total += h * (a.heads * (a.dim + a.vdim) + a.cached_heads * (a.dim + a.vdim))
                    total += h * a.heads * a.vdim * a.gate + a.heads * (a.sink + (a.weights == "sigmoid")) + (a.v_first is not None)
                    total += (a.heads + a.kv_heads) * a.dim * a.qk_norm + ((a.heads + a.cached_heads) * a.dim + a.cached_heads * a.vdim) * a.bias + h * a.o_bias
                if m is not None:
                    total += h * (m.in_dim + m.inner) + m.conv_dim * (m.conv + 1) + 3 * m.heads + m.inner
                if c is not None:
                    total += c.heads * (h * (c.dim + c.rot_dim + c.vdim) + c.kv_rank * (c.dim + c.vdim))
                    total += (h * (c.kv_rank + c.rot_dim) + c.kv_rank) if c.kv_from is None else 0
                if d is not None:
                    total += h * (d.in_dim + d.inner) + d.conv_dim * d.conv + 2 * d.heads + d.vdim
                g, r = l.mixer.linear, l.mixer.gru
                if g is not None:
                    total += g.heads * (h * (2 * g.dim + 3 * g.vdim) + g.dim * (g.rank + 1)) + h * g.rank + g.vdim + 2 * h * l.mixer.normed_mean
                if r is not None:
                    total += r.width * (4 * h + 2)
                t = l.mixer.retention
                if t is not None:
                    total += h * t.heads * (2 * t.dim + 3 * t.vdim)
                if f is not None:
                    total += 0 if self.parallel_residual else n * (1 + self.post_norms)
                    total += (3 if f.gated else 2) * h * (f.ff * max(1, f.experts) + f.shared_ff)
                    if f.experts:
                        total += self.vocab * f.top if f.routing == "table" else (h + (f.routing in ("softmax", "chosen"))) * f.experts
            return total
        attn = h * (self.q_dim + 2 * self.kv_dim) + self.q_dim * h
        if self.is_moe:
            mlp = self.n_experts * (3 if self.gated_mlp else 2) * h * self.moe_intermediate + h * self.n_experts
            if self.shared_expert_intermediate:
                mlp += 3 * h * self.shared_expert_intermediate + h
        else:
            mlp = (3 if self.gated_mlp else 2) * h * i
        emb = self.vocab * h * (1 if self.tie_word_embeddings else 2)
        return self.n_layers * (attn + mlp + 2 * h) + emb + h


#: HF ``model_type`` -> function(hf_config) -> ArchSpec
ARCH_BUILDERS: Dict[str, Callable[[Any], ArchSpec]] = {}


def register_arch(*model_types: str):

    def deco(fn):
        for mt in model_types:
            ARCH_BUILDERS[mt] = fn
        return fn

    return deco


def _get(cfg: Any, *names: str, default=None):
    for n in names:
        if isinstance(cfg, dict):
            if n in cfg and cfg[n] is not None:
                return cfg[n]
        elif getattr(cfg, n, None) is not None:
            return getattr(cfg, n)
    return default


def arch_from_hf_config(cfg: Any) -> ArchSpec:
    mt = _get(cfg, "model_type")
    if mt not in ARCH_BUILDERS:
        raise ValueError(f"Unsupported model type {mt}; supported: {sorted(ARCH_BUILDERS)}")
    return ARCH_BUILDERS[mt](cfg)


def supported_model_types() -> List[str]:
    return sorted(ARCH_BUILDERS)


# ---------------------------------------------------------------------------------------------------
# family builders (ref: each family's model.py property block, e.g. llama_v2/model.py:36-116)
# ---------------------------------------------------------------------------------------------------
def _rope_theta(cfg, default=10000.0) -> float:
    theta = _get(cfg, "rope_theta")
    if theta is None:
        rp = _get(cfg, "rope_parameters", "rope_scaling")
        if isinstance(rp, dict) and rp.get("rope_theta") is not None:
            theta = rp["rope_theta"]
    return float(theta if theta is not None else default)


def _window_fields(cfg, mt) -> Dict[str, Any]:
    """Sliding-window settings of the llama-like families. Mistral / Phi-3: ``sliding_window`` on every layer. Qwen2:
    only with ``use_sliding_window``, and then on the layers HF marks ``sliding_attention`` (``layer_types``) or, for
    older configs, on layers >= ``max_window_layers``."""
    w = _get(cfg, "sliding_window")
    if not w or mt not in ("mistral", "phi3", "qwen2", "mixtral", "qwen2_moe"):
        return {}
    n = _get(cfg, "num_hidden_layers")
    if mt in ("qwen2", "qwen2_moe"):
        if not _get(cfg, "use_sliding_window", default=False):
            return {}
        types = _get(cfg, "layer_types")
        if types:
            return {"layer_windows": [int(w) if t == "sliding_attention" else 0 for t in types]}
        first = _get(cfg, "max_window_layers", default=n)
        return {"layer_windows": [int(w) if i >= first else 0 for i in range(n)]}
    types = _get(cfg, "layer_types")
    if types and any(t != "sliding_attention" for t in types):
        return {"layer_windows": [int(w) if t == "sliding_attention" else 0 for t in types]}
    return {"sliding_window": int(w)}


@register_arch("llama", "mistral", "qwen2", "phi3", "internlm")
def _llama_like(cfg) -> ArchSpec:
    mt = _get(cfg, "model_type")
    h = _get(cfg, "hidden_size")
    nh = _get(cfg, "num_attention_heads")
    return ArchSpec(
        model_type=mt, n_layers=_get(cfg, "num_hidden_layers"), hidden=h, n_heads=nh,
        n_kv_heads=_get(cfg, "num_key_value_heads", default=nh), head_dim=_get(cfg, "head_dim", default=h // nh),
        intermediate=_get(cfg, "intermediate_size"), vocab=_get(cfg, "vocab_size"), norm="rms",
        norm_eps=_get(cfg, "rms_norm_eps", default=1e-5), act=_get(cfg, "hidden_act", default="silu"), gated_mlp=True,
        pos_emb="rope", rope_theta=_rope_theta(cfg), max_positions=_get(cfg, "max_position_embeddings", default=4096),
        qkv_bias=(mt == "qwen2") or bool(_get(cfg, "attention_bias", default=False)),
        attn_out_bias=bool(_get(cfg, "attention_bias", default=False)) and mt != "qwen2",
        mlp_bias=bool(_get(cfg, "mlp_bias", default=False)),
        tie_word_embeddings=bool(_get(cfg, "tie_word_embeddings", default=False)), **_window_fields(cfg, mt))


@register_arch("opt")
def _opt(cfg) -> ArchSpec:
    h = _get(cfg, "hidden_size")
    nh = _get(cfg, "num_attention_heads")
    if _get(cfg, "word_embed_proj_dim", default=h) != h:
        raise ValueError("OPT variants with word_embed_proj_dim != hidden_size (opt-350m) are not supported")
    if not _get(cfg, "do_layer_norm_before", default=True):
        raise ValueError("post-LayerNorm OPT variants are not supported")
    return ArchSpec(
        model_type="opt", n_layers=_get(cfg, "num_hidden_layers"), hidden=h, n_heads=nh, n_kv_heads=nh,
        head_dim=h // nh, intermediate=_get(cfg, "ffn_dim"), vocab=_get(cfg, "vocab_size"), norm="layer", norm_eps=1e-5,
        act=_get(cfg, "activation_function", default="relu"), gated_mlp=False, pos_emb="learned", learned_pos_offset=2,
        max_positions=_get(cfg, "max_position_embeddings", default=2048), qkv_bias=bool(_get(cfg, "enable_bias", default=True)),
        attn_out_bias=bool(_get(cfg, "enable_bias", default=True)), mlp_bias=bool(_get(cfg, "enable_bias", default=True)),
        norm_bias=True, tie_word_embeddings=True, final_norm=True)


@register_arch("falcon")
def _falcon(cfg) -> ArchSpec:
    h = _get(cfg, "hidden_size")
    nh = _get(cfg, "num_attention_heads")
    new_arch = bool(_get(cfg, "new_decoder_architecture", default=False))
    if new_arch:
        nkv = _get(cfg, "num_kv_heads", default=nh)
    else:
        nkv = 1 if _get(cfg, "multi_query", default=True) else nh
    alibi = bool(_get(cfg, "alibi", default=False))
    return ArchSpec(
        model_type="falcon", n_layers=_get(cfg, "num_hidden_layers"), hidden=h, n_heads=nh, n_kv_heads=nkv,
        head_dim=h // nh, intermediate=_get(cfg, "ffn_hidden_size", default=4 * h), vocab=_get(cfg, "vocab_size"),
        norm="layer", norm_eps=_get(cfg, "layer_norm_epsilon", default=1e-5), act="gelu", gated_mlp=False,
        pos_emb="alibi" if alibi else "rope", alibi_scale=(h // nh) ** -0.5 if alibi else 1.0, rope_theta=_rope_theta(cfg), max_positions=_get(cfg, "max_position_embeddings", default=2048),
        qkv_bias=bool(_get(cfg, "bias", default=False)), attn_out_bias=bool(_get(cfg, "bias", default=False)),
        mlp_bias=bool(_get(cfg, "bias", default=False)), norm_bias=True,
        parallel_residual=bool(_get(cfg, "parallel_attn", default=True)), parallel_two_norms=new_arch,
        tie_word_embeddings=True, extras={"new_decoder_architecture": new_arch})


@register_arch("phi")
def _phi(cfg) -> ArchSpec:
    h = _get(cfg, "hidden_size")
    nh = _get(cfg, "num_attention_heads")
    hd = h // nh
    return ArchSpec(
        model_type="phi", n_layers=_get(cfg, "num_hidden_layers"), hidden=h, n_heads=nh,
        n_kv_heads=_get(cfg, "num_key_value_heads", default=nh), head_dim=hd, intermediate=_get(cfg, "intermediate_size"),
        vocab=_get(cfg, "vocab_size"), norm="layer", norm_eps=_get(cfg, "layer_norm_eps", default=1e-5),
        act=_get(cfg, "hidden_act", default="gelu_new"), gated_mlp=False, pos_emb="rope", rope_theta=_rope_theta(cfg),
        rotary_dim=int(hd * _get(cfg, "partial_rotary_factor", default=0.5)),
        max_positions=_get(cfg, "max_position_embeddings", default=2048), qkv_bias=True, attn_out_bias=True, mlp_bias=True,
        lm_head_bias=True, norm_bias=True, parallel_residual=True)


@register_arch("qwen")
def _qwen(cfg) -> ArchSpec:
    h = _get(cfg, "hidden_size")
    nh = _get(cfg, "num_attention_heads")
    return ArchSpec(
        model_type="qwen", n_layers=_get(cfg, "num_hidden_layers"), hidden=h, n_heads=nh, n_kv_heads=nh,
        head_dim=_get(cfg, "kv_channels", default=h // nh), intermediate=_get(cfg, "intermediate_size") // 2,
        vocab=_get(cfg, "vocab_size"), norm="rms", norm_eps=_get(cfg, "layer_norm_epsilon", default=1e-6), act="silu",
        gated_mlp=True, pos_emb="rope", rope_theta=float(_get(cfg, "rotary_emb_base", default=10000.0)),
        max_positions=_get(cfg, "seq_length", "max_position_embeddings", default=8192), qkv_bias=True)


# ---- families the reference serves only through v1 kernel injection (module_inject/containers/{gpt2,gptj,gptneox}.py).
# Here they are three more specs for the same executor, so init_inference(replace_with_kernel_inject=True) runs them
# on the sm_100a kernels with paged KV, and HCache restore works for them too.
@register_arch("gpt2")
def _gpt2(cfg) -> ArchSpec:
    h = _get(cfg, "n_embd", "hidden_size")
    nh = _get(cfg, "n_head", "num_attention_heads")
    if _get(cfg, "scale_attn_by_inverse_layer_idx", default=False) or not _get(cfg, "scale_attn_weights", default=True):
        raise ValueError("GPT-2 variants with non-standard attention scaling are not supported")
    return ArchSpec(
        model_type="gpt2", n_layers=_get(cfg, "n_layer", "num_hidden_layers"), hidden=h, n_heads=nh, n_kv_heads=nh,
        head_dim=h // nh, intermediate=_get(cfg, "n_inner", default=4 * h), vocab=_get(cfg, "vocab_size"), norm="layer",
        norm_eps=_get(cfg, "layer_norm_epsilon", default=1e-5), act=_get(cfg, "activation_function", default="gelu_new"),
        gated_mlp=False, pos_emb="learned", learned_pos_offset=0, max_positions=_get(cfg, "n_positions", default=1024),
        qkv_bias=True, attn_out_bias=True, mlp_bias=True, norm_bias=True, tie_word_embeddings=True)


@register_arch("gpt_neo")
def _gpt_neo(cfg) -> ArchSpec:
    """GPT-Neo: learned positions, UNSCALED attention scores, layers alternate between global and local (sliding-window)
    attention as listed in ``attention_layers``."""
    h = _get(cfg, "hidden_size")
    nh = _get(cfg, "num_heads", "num_attention_heads")
    n = _get(cfg, "num_layers", "num_hidden_layers")
    kinds = list(_get(cfg, "attention_layers", default=["global"] * n))
    win = int(_get(cfg, "window_size", default=256))
    return ArchSpec(
        model_type="gpt_neo", n_layers=n, hidden=h, n_heads=nh, n_kv_heads=nh, head_dim=h // nh,
        intermediate=_get(cfg, "intermediate_size", default=None) or 4 * h, vocab=_get(cfg, "vocab_size"), norm="layer",
        norm_eps=_get(cfg, "layer_norm_epsilon", default=1e-5), act=_get(cfg, "activation_function", default="gelu_new"),
        gated_mlp=False, pos_emb="learned", learned_pos_offset=0, max_positions=_get(cfg, "max_position_embeddings", default=2048),
        qkv_bias=False, attn_out_bias=True, mlp_bias=True, norm_bias=True, tie_word_embeddings=True, attn_scale=1.0,
        layer_windows=[win if k == "local" else 0 for k in kinds])


@register_arch("gptj")
def _gptj(cfg) -> ArchSpec:
    h = _get(cfg, "n_embd", "hidden_size")
    nh = _get(cfg, "n_head", "num_attention_heads")
    hd = h // nh
    return ArchSpec(
        model_type="gptj", n_layers=_get(cfg, "n_layer", "num_hidden_layers"), hidden=h, n_heads=nh, n_kv_heads=nh,
        head_dim=hd, intermediate=_get(cfg, "n_inner", default=4 * h), vocab=_get(cfg, "vocab_size"), norm="layer",
        norm_eps=_get(cfg, "layer_norm_epsilon", default=1e-5), act=_get(cfg, "activation_function", default="gelu_new"),
        gated_mlp=False, pos_emb="rope", rope_theta=10000.0, rotary_dim=_get(cfg, "rotary_dim", default=hd),
        max_positions=_get(cfg, "n_positions", default=2048), qkv_bias=False, attn_out_bias=False, mlp_bias=True,
        lm_head_bias=True, norm_bias=True, parallel_residual=True,
        tie_word_embeddings=bool(_get(cfg, "tie_word_embeddings", default=False)),
        extras={"rope_interleaved_checkpoint": True})     # rows are re-ordered once at load (families.map_gptj)


@register_arch("gpt_neox")
def _gpt_neox(cfg) -> ArchSpec:
    h = _get(cfg, "hidden_size")
    nh = _get(cfg, "num_attention_heads")
    hd = h // nh
    pct = _get(cfg, "rotary_pct", "partial_rotary_factor")
    if pct is None:
        rp = _get(cfg, "rope_parameters", "rope_scaling")
        pct = rp.get("partial_rotary_factor") if isinstance(rp, dict) else None
    pct = 0.25 if pct is None else float(pct)
    theta = _get(cfg, "rotary_emb_base")
    par = bool(_get(cfg, "use_parallel_residual", default=True))
    return ArchSpec(
        model_type="gpt_neox", n_layers=_get(cfg, "num_hidden_layers"), hidden=h, n_heads=nh, n_kv_heads=nh, head_dim=hd,
        intermediate=_get(cfg, "intermediate_size", default=4 * h), vocab=_get(cfg, "vocab_size"), norm="layer",
        norm_eps=_get(cfg, "layer_norm_eps", default=1e-5), act=_get(cfg, "hidden_act", default="gelu"), gated_mlp=False,
        pos_emb="rope", rope_theta=float(theta) if theta is not None else _rope_theta(cfg), rotary_dim=int(hd * pct),
        max_positions=_get(cfg, "max_position_embeddings", default=2048),
        qkv_bias=bool(_get(cfg, "attention_bias", default=True)), attn_out_bias=bool(_get(cfg, "attention_bias", default=True)),
        mlp_bias=True, norm_bias=True, parallel_residual=par, parallel_two_norms=par,
        tie_word_embeddings=bool(_get(cfg, "tie_word_embeddings", default=False)))


@register_arch("bloom")
def _bloom(cfg) -> ArchSpec:
    h = _get(cfg, "hidden_size", "n_embed")
    nh = _get(cfg, "n_head", "num_attention_heads")
    if _get(cfg, "apply_residual_connection_post_layernorm", default=False):
        raise ValueError("Bloom variants with the residual taken after the LayerNorm are not supported")
    return ArchSpec(
        model_type="bloom", n_layers=_get(cfg, "n_layer", "num_hidden_layers"), hidden=h, n_heads=nh, n_kv_heads=nh,
        head_dim=h // nh, intermediate=4 * h, vocab=_get(cfg, "vocab_size"), norm="layer",
        norm_eps=_get(cfg, "layer_norm_epsilon", default=1e-5), act="gelu_tanh", gated_mlp=False, pos_emb="alibi",
        max_positions=_get(cfg, "seq_length", "max_position_embeddings", default=2048), qkv_bias=True, attn_out_bias=True,
        mlp_bias=True, norm_bias=True, embed_norm=True, tie_word_embeddings=True)


@register_arch("mixtral")
def _mixtral(cfg) -> ArchSpec:
    base = _llama_like(cfg)
    return base.scaled(model_type="mixtral", n_experts=_get(cfg, "num_local_experts"), top_k=_get(cfg, "num_experts_per_tok"),
                       moe_intermediate=_get(cfg, "intermediate_size"), norm_topk_prob=True)


@register_arch("qwen2_moe")
def _qwen2_moe(cfg) -> ArchSpec:
    base = _llama_like(cfg)
    return base.scaled(model_type="qwen2_moe", qkv_bias=True, attn_out_bias=False, n_experts=_get(cfg, "num_experts"),
                       top_k=_get(cfg, "num_experts_per_tok"), moe_intermediate=_get(cfg, "moe_intermediate_size"),
                       shared_expert_intermediate=_get(cfg, "shared_expert_intermediate_size", default=0),
                       norm_topk_prob=bool(_get(cfg, "norm_topk_prob", default=False)))


@register_arch("nipolorn")
def _nipolorn(cfg) -> ArchSpec:
    """Nipolorn: every layer runs windowed attention with kept first tokens beside a Mamba-2 mixer; feed-forwards are dense
    (clamped gate) or mixtures of experts chosen by token id; norms before and after each sublayer. Everything is per layer
    in config.json (``layers``), so the scalar fields only carry the largest values."""

    def ff(m) -> Optional[FeedForwardSpec]:
        if m is None:
            return None
        if m["kind"] == "dense":
            return FeedForwardSpec(ff=int(m["ff"]), act="swiglu_clamped", limit=float(m["limit"]))
        if m["kind"] != "moe":
            raise ValueError(f"nipolorn: unknown feed-forward kind {m['kind']!r}")
        shared = m.get("shared") or {}
        return FeedForwardSpec(ff=int(m["expert"]["ff"]), act="silu", experts=int(m["router"]["experts"]), top=int(m["router"]["top"]),
                               routing="table", shared_ff=int(shared.get("ff", 0)))

    layers = []
    for lc in _get(cfg, "layers"):
        if lc["type"] != "parallel":
            raise ValueError(f"nipolorn: unknown layer type {lc['type']!r}")
        mx = lc["mixer"]
        a, r = mx["left"], mx["right"]
        layers.append(LayerSpec(
            mixer=MixerSpec(
                attn=AttentionSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                                   scale=float(a["scale"]), window=int(a["mask"]["size"]), keep_first=int(a["mask"]["keep_first"])),
                ssm=StateSpaceSpec(heads=int(r["heads"]), vdim=int(r["vdim"]), state=int(r["state"]), groups=int(r["groups"]),
                                   conv=int(r["conv"]), norm_groups=int(r["norm_groups"])),
                attn_weight=float(mx["left_scale"]), ssm_weight=float(mx["right_scale"])),
            mlp=ff(lc.get("mlp"))))
    return stack_arch("nipolorn", layers, hidden=int(_get(cfg, "width")), vocab=int(_get(cfg, "vocab")),
                      norm_eps=float(_get(cfg, "norm")["eps"]), **NIPOLORN_NORMS)


#: norms of Nipolorn: on both sides of every sublayer, weights stored as differences from one
NIPOLORN_NORMS = dict(post_norms=True, norm_weight_offset=1.0)


@register_arch("dedelorn")
def _dedelorn(cfg) -> ArchSpec:
    """Dedelorn: layers of a gated delta rule or of latent attention in any order, each beside its feed-forward (dense, or a
    mixture of experts with a corrected softmax router) on one norm; latent attention layers may share another layer's cache."""

    def ff(m) -> Optional[FeedForwardSpec]:
        if m is None:
            return None
        if m["kind"] == "dense":
            return FeedForwardSpec(ff=int(m["ff"]), act="gelu_tanh")
        if m["kind"] != "moe":
            raise ValueError(f"dedelorn: unknown feed-forward kind {m['kind']!r}")
        r = m["router"]
        return FeedForwardSpec(ff=int(m["expert"]["ff"]), act="gelu", experts=int(r["experts"]), top=int(r["top"]), routing="softmax",
                               router_scale=float(r.get("scale", 1.0)), gated=False)

    layers: List[LayerSpec] = []
    for i, lc in enumerate(_get(cfg, "layers")):
        mx = lc["mixer"]
        if lc["type"] == "delta":
            mixer = MixerSpec(delta=DeltaSpec(heads=int(mx["heads"]), kv_heads=int(mx["kv_heads"]), dim=int(mx["dim"]), vdim=int(mx["vdim"]),
                                              conv=int(mx["conv"])))
        elif lc["type"] == "latent_attention":
            rot, src = mx["rot"], mx.get("kv_from")
            a = LatentAttentionSpec(heads=int(mx["heads"]), dim=int(mx["dim"]), rot_dim=int(mx["rot_dim"]), vdim=int(mx["vdim"]),
                                    kv_rank=int(mx["kv_rank"]), scale=float(mx["scale"]), window=int((mx.get("mask") or {}).get("size", 0)),
                                    rot_base=float(rot["base"]), kv_from=None if src is None else int(src))
            if int(rot["dims"]) != a.rot_dim:
                raise ValueError("dedelorn: rot.dims must equal rot_dim")
            if src is not None:
                own = layers[a.kv_from].mixer.latent if 0 <= a.kv_from < i else None
                if own is None or own.kv_from is not None or (own.kv_rank, own.rot_dim, own.rot_base) != (a.kv_rank, a.rot_dim, a.rot_base):
                    raise ValueError(f"dedelorn: layer {i} cannot use the latents of layer {src}")
            mixer = MixerSpec(latent=a)
        else:
            raise ValueError(f"dedelorn: unknown layer type {lc['type']!r}")
        layers.append(LayerSpec(mixer=mixer, mlp=ff(lc.get("mlp"))))
    return stack_arch("dedelorn", layers, hidden=int(_get(cfg, "width")), vocab=int(_get(cfg, "vocab")),
                      norm_eps=float(_get(cfg, "norm")["eps"]), **DEDELORN_NORMS)


#: Dedelorn: one norm per layer read by both sublayers, and a norm on the embeddings
DEDELORN_NORMS = dict(parallel_residual=True, embed_norm=True)


@register_arch("lotelix")
def _lotelix(cfg) -> ArchSpec:
    """Lotelix: layers of a minGRU, of windowed attention (rotated, with sinks, an output gate and values mixed with the first such
    layer's), or of sigmoid attention beside gated linear attention, in any order; mixtures of experts with a sigmoid router."""

    def ff(m) -> Optional[FeedForwardSpec]:
        if m is None:
            return None
        if m["kind"] != "moe":
            raise ValueError(f"lotelix: unknown feed-forward kind {m['kind']!r}")
        return FeedForwardSpec(ff=int(m["expert"]["ff"]), act="relu2", experts=int(m["router"]["experts"]), top=int(m["router"]["top"]),
                               routing="sigmoid", gated=False)

    def rotation(r, adjacent) -> RotationSpec:
        sc = r.get("scaling")
        slow = {} if sc is None else dict(slow_factor=float(sc["factor"]), slow_low=float(sc["low"]), slow_high=float(sc["high"]),
                                          original=float(sc["original"]))
        return RotationSpec(dims=int(r["dims"]), base=float(r["base"]), adjacent=adjacent, **slow)

    def attention(a, adjacent, **kw) -> AttentionSpec:
        spec = AttentionSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]), scale=float(a["scale"]),
                             window=int((a.get("mask") or {}).get("size") or 0), rot=rotation(a["rot"], adjacent), **kw)
        if spec.rot.dims > spec.dim or spec.rot.dims % 2 or spec.heads % spec.kv_heads:
            raise ValueError("lotelix: rot.dims must be even and at most dim, heads a multiple of kv_heads")
        return spec

    layers: List[LayerSpec] = []
    first = None            # the layer whose values the later ones mix in
    for i, lc in enumerate(_get(cfg, "layers")):
        mx = lc["mixer"]
        if lc["type"] == "mingru":
            mixer = MixerSpec(gru=GRUSpec(width=int(mx["width"])))
        elif lc["type"] == "attention":
            a = attention(mx, False, sink=True, gate=True, v_first=first if mx.get("v_mix") else None)
            if a.v_first is not None:
                b = layers[first].mixer.attn
                if (b.kv_heads, b.vdim) != (a.kv_heads, a.vdim):
                    raise ValueError(f"lotelix: layer {i} cannot mix in the values of layer {first}")
            elif mx.get("v_mix"):
                first = i
            mixer = MixerSpec(attn=a)
        elif lc["type"] == "parallel":
            r = mx["right"]
            mixer = MixerSpec(attn=attention(mx["left"], True, weights="sigmoid", bias=True, o_bias=True, qk_norm=True),
                              linear=LinearAttentionSpec(heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]), tau=float(r["tau"])))
        else:
            raise ValueError(f"lotelix: unknown layer type {lc['type']!r}")
        layers.append(LayerSpec(mixer=mixer, mlp=ff(lc.get("mlp"))))
    width, groups = int(_get(cfg, "width")), int(_get(cfg, "norm").get("groups", 1))
    if width % groups:
        raise ValueError("lotelix: width must be a multiple of norm.groups")
    return stack_arch("lotelix", layers, hidden=width, vocab=int(_get(cfg, "vocab")), norm_eps=float(_get(cfg, "norm")["eps"]),
                      norm_groups=groups, embed_scale=float((_get(cfg, "embedding") or {}).get("scale", 1.0)))


@register_arch("relulix")
def _relulix(cfg) -> ArchSpec:
    """Relulix: layers of retention or of windowed attention (biases, partly rotated heads, bounded scores, a one more in the
    denominator; some on another layer's keys and values) in any order, each beside its feed-forward on one norm whose weight is a
    single number; mixtures of clamped gated experts weighed by the softmax over the chosen ones."""

    def ff(m) -> Optional[FeedForwardSpec]:
        if m is None:
            return None
        if m["kind"] != "moe":
            raise ValueError(f"relulix: unknown feed-forward kind {m['kind']!r}")
        f = FeedForwardSpec(ff=int(m["expert"]["ff"]), act="swiglu_clamped", limit=float(m["expert"]["limit"]),
                            experts=int(m["router"]["experts"]), top=int(m["router"]["top"]), routing="chosen")
        if not 1 <= f.top <= f.experts:
            raise ValueError("relulix: a token's experts are at least one and at most all")
        return f

    def rotation(r, dim) -> RotationSpec:
        sc = r.get("scaling")
        slow = {} if sc is None else dict(slow_factor=float(sc["factor"]), slow_low=float(sc["slow"]), slow_high=float(sc["fast"]),
                                          original=float(sc["original"]), ramp=True, amplitude=0.1 * math.log(sc["factor"]) + 1.0)
        spec = RotationSpec(dims=int(r["dims"]), base=float(r["base"]), **slow)
        if spec.dims > dim or spec.dims % 2:
            raise ValueError("relulix: rot.dims must be even and at most dim")
        return spec

    layers: List[LayerSpec] = []
    for i, lc in enumerate(_get(cfg, "layers")):
        mx = lc["mixer"]
        if lc["type"] == "retention":
            m = RetentionSpec(heads=int(mx["heads"]), dim=int(mx["dim"]), vdim=int(mx["vdim"]), decay=[float(d) for d in mx["decay"]],
                              rot=rotation(mx["rot"], int(mx["dim"])))
            if len(m.decay) != m.heads:
                raise ValueError(f"relulix: layer {i} has {m.heads} heads and {len(m.decay)} decays")
            mixer = MixerSpec(retention=m)
        elif lc["type"] == "attention":
            src = mx.get("kv_from")
            a = AttentionSpec(heads=int(mx["heads"]), kv_heads=int(mx["kv_heads"]), dim=int(mx["dim"]), vdim=int(mx["vdim"]),
                              scale=float(mx["scale"]), window=int((mx.get("mask") or {}).get("size") or 0),
                              rot=rotation(mx["rot"], int(mx["dim"])), bias=True, one_more=True, softcap=float(mx.get("softcap") or 0.0),
                              kv_from=None if src is None else int(src))
            if a.heads % a.kv_heads:
                raise ValueError("relulix: heads must be a multiple of kv_heads")
            if src is not None:
                own = layers[a.kv_from].mixer.attn if 0 <= a.kv_from < i else None
                if own is None or own.kv_from is not None or (own.kv_heads, own.dim, own.vdim, own.rot) != (a.kv_heads, a.dim, a.vdim, a.rot):
                    raise ValueError(f"relulix: layer {i} cannot use the keys and values of layer {src}")
            mixer = MixerSpec(attn=a)
        else:
            raise ValueError(f"relulix: unknown layer type {lc['type']!r}")
        layers.append(LayerSpec(mixer=mixer, mlp=ff(lc.get("mlp"))))
    return stack_arch("relulix", layers, hidden=int(_get(cfg, "width")), vocab=int(_get(cfg, "vocab")), norm_eps=float(_get(cfg, "norm")["eps"]),
                      embed_scale=float((_get(cfg, "embedding") or {}).get("scale", 1.0)), **RELULIX_NORMS)


#: Relulix: one norm per layer read by both sublayers, its weight a single number
RELULIX_NORMS = dict(parallel_residual=True, norm_scalar=True)


def stack_arch(model_type: str, layers: List[LayerSpec], hidden: int, vocab: int, norm_eps: float, **kw) -> ArchSpec:
    """ArchSpec of a stack of unlike layers; its scalar sizes are those of the layer with the widest KV pages, or the largest of any."""
    attn = [l.mixer.attn for l in layers if l.mixer.attn is not None]
    mlps = [l.mlp for l in layers if l.mlp is not None]
    latent = [l.mixer.latent for l in layers if l.mixer.latent is not None]
    geometry = [(a.kv_heads * a.page_dim, a.heads, a.kv_heads, a.page_dim) for a in attn] + [(c.page_width, 1, 1, c.page_width) for c in latent]
    _, n_heads, n_kv_heads, head_dim = max(geometry, default=(0, 1, 1, 64))
    return ArchSpec(model_type=model_type, n_layers=len(layers), hidden=hidden, n_heads=n_heads,
                    n_kv_heads=n_kv_heads, head_dim=head_dim,
                    intermediate=max((m.ff for m in mlps if not m.experts), default=0), vocab=vocab, norm="rms",
                    norm_eps=norm_eps, act="silu", gated_mlp=True, pos_emb="none",
                    sliding_window=max((a.window for a in attn + latent), default=0), max_positions=1 << 30,
                    n_experts=max((m.experts for m in mlps), default=0), top_k=max((m.top for m in mlps), default=0),
                    moe_intermediate=max((m.ff for m in mlps if m.experts), default=0),
                    shared_expert_intermediate=max((m.shared_ff for m in mlps), default=0), layers=layers, **kw)


# ---------------------------------------------------------------------------------------------------
# named configurations used by benchmarks and tests (random-init weights; shapes of the public models)
# ---------------------------------------------------------------------------------------------------
def named_arch(name: str) -> ArchSpec:
    n = name.lower().replace("_", "-")
    llama = dict(model_type="llama", norm="rms", norm_eps=1e-5, act="silu", gated_mlp=True, pos_emb="rope",
                 max_positions=4096, vocab=32000, head_dim=128)
    opt = dict(model_type="opt", norm="layer", norm_eps=1e-5, act="relu", gated_mlp=False, pos_emb="learned",
               learned_pos_offset=2, max_positions=2048, vocab=50272, qkv_bias=True, attn_out_bias=True, mlp_bias=True,
               norm_bias=True, tie_word_embeddings=True)
    table = {
        "llama-2-7b": ArchSpec(n_layers=32, hidden=4096, n_heads=32, n_kv_heads=32, intermediate=11008, **llama),
        "llama-2-13b": ArchSpec(n_layers=40, hidden=5120, n_heads=40, n_kv_heads=40, intermediate=13824, **llama),
        "llama-2-70b": ArchSpec(n_layers=80, hidden=8192, n_heads=64, n_kv_heads=8, intermediate=28672, **llama),
        "opt-125m": ArchSpec(n_layers=12, hidden=768, n_heads=12, n_kv_heads=12, head_dim=64, intermediate=3072, **opt),
        "opt-30b": ArchSpec(n_layers=48, hidden=7168, n_heads=56, n_kv_heads=56, head_dim=128, intermediate=28672, **opt),
        "tiny-llama-test": ArchSpec(n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, intermediate=512,
                                    **{**llama, "vocab": 512, "head_dim": 64}),
        "tiny-mixtral-test": ArchSpec(n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, intermediate=512,
                                      **{**llama, "vocab": 512, "head_dim": 64, "model_type": "mixtral"}, n_experts=8,
                                      top_k=2, moe_intermediate=384, norm_topk_prob=True),
        "tiny-opt-test": ArchSpec(n_layers=2, hidden=256, n_heads=4, n_kv_heads=4, intermediate=512,
                                  **{**opt, "vocab": 512, "head_dim": 64, "max_positions": 512}),
    }
    table.update(_stack_named())
    if n not in table:
        raise KeyError(f"unknown named architecture {name}; known: {sorted(table)}")
    return table[n]


def _stack_named() -> Dict[str, ArchSpec]:
    """Nipolorn, Dedelorn, Lotelix and Relulix stacks with layers of real sizes, and beside each the closest plain family at equal sizes (same
    width, heads, window and feed-forward): windowed attention with a dense MLP, or with routed experts and a shared one."""

    def nipolorn(width, heads, kv, window, keep, ssm_heads, groups, mlp):
        mixer = MixerSpec(attn=AttentionSpec(heads, kv, 128, 128, 128 ** -0.5, window, keep),
                          ssm=StateSpaceSpec(ssm_heads, 64, 128, groups, 4, groups), attn_weight=1.0, ssm_weight=0.5)
        return stack_arch("nipolorn", [LayerSpec(mixer, mlp)] * 4, hidden=width, vocab=32000, norm_eps=1e-5, **NIPOLORN_NORMS)

    def dedelorn(width, heads, rank, window, mlp):
        delta = MixerSpec(delta=DeltaSpec(heads=width // 128, kv_heads=width // 256, dim=128, vdim=128, conv=4))

        def latent(kv_from=None):
            return MixerSpec(latent=LatentAttentionSpec(heads, 96, 32, 128, rank, 128**-0.5, window, 1e4, kv_from))

        return stack_arch("dedelorn", [LayerSpec(m, mlp) for m in (delta, latent(), delta, latent(1))], hidden=width, vocab=32000,
                          norm_eps=1e-5, **DEDELORN_NORMS)

    def lotelix(width, heads, kv, window, ff):
        def attn(v_first=None):
            return MixerSpec(attn=AttentionSpec(heads, kv, 128, 128, 128**-0.5, window, rot=RotationSpec(128, 1e6, False, 8.0, 1.0, 4.0, 8192), sink=True,
                                                gate=True, v_first=v_first))

        both = MixerSpec(attn=AttentionSpec(heads, kv, 128, 128, 128**-0.5, rot=RotationSpec(128, 1e6, True), weights="sigmoid", bias=True, o_bias=True, qk_norm=True),
                         linear=LinearAttentionSpec(heads=width // 128, dim=128, vdim=128, tau=16.0, rank=16))
        mlp = FeedForwardSpec(ff=ff, act="relu2", experts=16, top=2, routing="sigmoid", gated=False)
        return stack_arch("lotelix", [LayerSpec(m, mlp) for m in (MixerSpec(gru=GRUSpec(width)), attn(), both, attn(1))], hidden=width, vocab=32000,
                          norm_eps=1e-5, norm_groups=2, embed_scale=1.0)

    def relulix(width, heads, kv, window, ff):
        rot = RotationSpec(64, 1e6, False, 4.0, 1.0, 32.0, 8192, True, 0.1 * math.log(4.0) + 1.0)

        def attn(kv_from=None):
            return MixerSpec(attn=AttentionSpec(heads, kv, 128, 128, 128**-0.5, window, rot=rot, bias=True, one_more=True, softcap=30.0, kv_from=kv_from))

        n = width // 128
        ret = MixerSpec(retention=RetentionSpec(n, 128, 128, [1.0 - 2.0**(-5.0 - 7.0 * i / n) for i in range(n)], RotationSpec(128, 1e6)))
        mlp = FeedForwardSpec(ff=ff, act="swiglu_clamped", limit=7.0, experts=16, top=2, routing="chosen")
        return stack_arch("relulix", [LayerSpec(m, mlp) for m in (ret, attn(), ret, attn(1))], hidden=width, vocab=32000, norm_eps=1e-5, embed_scale=1.0,
                          **RELULIX_NORMS)

    def plain(mt, width, heads, kv, window, **kw):
        return ArchSpec(model_type=mt, n_layers=4, hidden=width, n_heads=heads, n_kv_heads=kv, head_dim=128, vocab=32000, norm="rms",
                        norm_eps=1e-5, act="silu", gated_mlp=True, pos_emb="rope", sliding_window=window, max_positions=1 << 20, **kw)

    moe = dict(n_experts=16, top_k=2, moe_intermediate=3584, shared_expert_intermediate=3584)
    return {
        "nipolorn-2048": nipolorn(2048, 16, 4, 1024, 16, 64, 4, FeedForwardSpec(ff=8192, act="swiglu_clamped", limit=7.0)),
        "dedelorn-2048": dedelorn(2048, 16, 256, 1024, FeedForwardSpec(ff=8192, act="gelu_tanh")),
        "dedelorn-4096": dedelorn(4096, 32, 512, 4096, FeedForwardSpec(ff=14336, act="gelu_tanh")),
        "dedelorn-4096-moe": dedelorn(4096, 32, 512, 2048, FeedForwardSpec(ff=5376, act="gelu", experts=16, top=2, routing="softmax", gated=False,
                                                                            router_scale=2.5)),
        "dedelorn-2048-moe": dedelorn(2048, 16, 256, 1024, FeedForwardSpec(ff=2688, act="gelu", experts=16, top=2, routing="softmax", gated=False,
                                                                            router_scale=2.5)),
        "lotelix-2048": lotelix(2048, 16, 4, 1024, 2688),
        "lotelix-4096": lotelix(4096, 32, 8, 2048, 5376),
        "relulix-2048": relulix(2048, 16, 4, 1024, 1792),
        "relulix-4096": relulix(4096, 32, 8, 2048, 3584),
        "mistral-2048": plain("mistral", 2048, 16, 4, 1024, intermediate=8192),
        "nipolorn-4096": nipolorn(4096, 32, 8, 4096, 64, 128, 8, FeedForwardSpec(ff=14336, act="swiglu_clamped", limit=7.0)),
        "mistral-4096": plain("mistral", 4096, 32, 8, 4096, intermediate=14336),
        "nipolorn-4096-moe": nipolorn(4096, 32, 8, 2048, 64, 64, 8, FeedForwardSpec(ff=3584, experts=16, top=2, shared_ff=3584)),
        "qwen2-moe-4096": plain("qwen2_moe", 4096, 32, 8, 2048, intermediate=3584, **moe),
    }
