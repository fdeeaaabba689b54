"""Two interchangeable op back ends with one signature set.

``CudaOps``  — the sm_100a kernels (``ops/kernels.py``); used whenever tensors live on a GPU.
``CpuOps``   — the PyTorch restatements (``ops/reference.py``); used for the CPU configuration
               (``init_inference`` on CPU, CPU-only CI). Never used on a CUDA device.

The model executor (:mod:`hcache_deepspeed_b200.models.transformer`) is written once against this
interface. Both back ends write into caller-provided buffers so steady-state forwards allocate nothing
(the role of the reference's ``empty_from`` view allocator, ``deepspeed/inference/v2/allocator.py:14-28``).
"""
from __future__ import annotations

from typing import Optional

import torch

from . import reference as ref
from .fp8 import Fp8Weight, quantize_rows_reference


def _fp8_emulate(a, w):
    """CPU restatement of the W8A8 path: fp8-round the activations per token, de-quantise both operands to fp32."""
    if not isinstance(w, Fp8Weight):
        return a, w
    q, s = quantize_rows_reference(a)
    return q.view(torch.float8_e4m3fn).float() * s[:, None], w.dequantize()


def windowed_len(n_keys: int, window: int, keep_first: int = 0) -> int:
    """Keys a work item really reads under a sliding window with kept first tokens (one tile of slack at both edges)."""
    return min(n_keys, window + 256 + (keep_first + 127) // 128 * 128) if window else n_keys


def padded_head_norm(m, eps: float):
    """(eps, factor) that make a norm over the zero-padded rows of retention's heads one over their own values."""
    r = m.vwidth / m.vdim
    return eps / r, r**-0.5


class CpuOps:
    name = "cpu-reference"

    # ---- linear ---------------------------------------------------------------------------------
    def gemm(self, a, w, out, bias=None, act=0, gated=False, workspace=None, comm=None, tp_wait=False, tp_signal=False, limit=0.0):
        a, w = _fp8_emulate(a, w)
        out.copy_(ref.gemm(a, w, bias=bias, act=act, gated=gated, out_dtype=out.dtype, limit=limit))
        return out

    def gemm_accum(self, a, w, accum, bias=None, comm=None, tp_signal=False):
        a, w = _fp8_emulate(a, w)
        accum += ref.gemm(a, w, bias=bias, out_dtype=torch.float32)

    def reserve_fp8(self, max_tokens, ks, device) -> None:
        pass

    # ---- norm -----------------------------------------------------------------------------------
    def norm(self, x, gamma, out, beta=None, delta=None, zero_delta=False, res_out=None, eps=1e-5, layer_norm=False,
             comm=None, zero_buf=None, scatter_rows=None):
        if delta is not None:
            s = (x.float() + delta.float()).to(x.dtype)
            if zero_delta and delta.dtype == torch.float32:
                delta.zero_()
            if res_out is not None:
                res_out.copy_(s)
            x = s
        out.copy_(ref.norm(x, gamma, beta, eps, layer_norm))
        return out

    # ---- attention-side -------------------------------------------------------------------------------
    def qkv_rope_kv_append(self, x, w_qkv, b_qkv, qkv_buf, q_out, kv_layer, tok_pos, tok_slot, inv_freq, n_q, n_kv, d,
                           rot_dim, block_size, workspace=None, comm=None, tp_wait=False):
        T = x.shape[0]
        dt = x.dtype
        x, w_qkv = _fp8_emulate(x, w_qkv)
        qkv = ref.gemm(x, w_qkv, bias=b_qkv, out_dtype=dt)
        q, k, v = qkv.split([n_q * d, n_kv * d, n_kv * d], dim=1)
        q, k, v = q.reshape(T, n_q, d), k.reshape(T, n_kv, d), v.reshape(T, n_kv, d)
        if inv_freq is not None:
            q = ref.rope_rotate_half(q, tok_pos, inv_freq, rot_dim)
            k = ref.rope_rotate_half(k, tok_pos, inv_freq, rot_dim)
        q_out.copy_(q.reshape(T, n_q * d))
        ref.kv_append(kv_layer, k, v, tok_slot)

    def restore_kv_proj(self, latents, w_kv, b_kv, kv_layer, tok_pos, tok_slot, inv_freq, n_kv, d, rot_dim, block_size,
                        scratch=None):
        T = latents.shape[0]
        dt = latents.dtype
        latents, w_kv = _fp8_emulate(latents, w_kv)
        kv = ref.gemm(latents, w_kv, bias=b_kv, out_dtype=dt)
        k, v = kv[:, :n_kv * d].reshape(T, n_kv, d), kv[:, n_kv * d:].reshape(T, n_kv, d)
        if inv_freq is not None:
            k = ref.rope_rotate_half(k, tok_pos, inv_freq, rot_dim)
        ref.kv_append(kv_layer, k, v, tok_slot)

    def attention(self, q, out, kv_layer, batch, n_q, n_kv, d, scale, ws_small=None, ws_large=None, alibi=None, window=0,
                  keep_first=0, sink=None, sigmoid_bias=None, gate=None, softcap=0.0):
        T = q.shape[0]
        q3, o3 = q.view(T, n_q, d), out.view(T, n_q, d)
        for items in (batch.items_small(), batch.items_large()):
            if items.shape[0]:
                ref.paged_attention(q3, kv_layer, batch.block_tables(), items, n_q, n_kv, scale, out=o3, alibi=alibi,
                                    window=window, keep_first=keep_first, sink=sink, sigmoid_bias=sigmoid_bias, gate=gate, softcap=softcap)

    # ---- stacks of unlike layers ----------------------------------------------------------------------
    def embed_f32(self, ids, weight, out, gamma=None, cols=None, eps=1e-5, scale=1.0):
        x = ref.embed(ids, weight).float() * scale
        out.copy_(x if gamma is None else x * torch.rsqrt((x * x).sum(-1, keepdim=True) / cols + eps) * gamma)
        return out

    def norm_residual(self, resid, gamma, out, delta=None, factor=1.0, post=None, cols=None, eps=1e-5, store_resid=True, groups=1,
                      delta2=None, post2=None):
        x, y = ref.norm_residual(resid, gamma, delta, factor, post, cols, eps, groups, delta2, post2)
        for d in (delta, delta2):
            if d is not None and d.dtype == torch.float32:
                d.zero_()
        if store_resid:
            resid.copy_(x)
        out.copy_(y)
        return out

    def mixer_in_proj(self, x, lw, a, proj, q_out, kv_layer, first, tok_pos, tok_slot, block_size, eps, workspace=None):
        self.gemm(x, lw.w_qkv, proj[:, :lw.w_qkv.shape[0]], bias=lw.b_qkv)
        self.attention_append(proj, lw, a, q_out, kv_layer, first, tok_pos, tok_slot, block_size, eps)

    def attention_append(self, proj, lw, a, q_out, kv_layer, first, tok_pos, tok_slot, block_size, eps):
        q = ref.attention_append(proj, kv_layer, tok_pos, tok_slot, a.heads if q_out is not None else 0, a.cached_heads, lw.rot_freq,
                                 lw.q_norm, lw.k_norm, a.heads * a.dim, a.kv_heads * a.dim, eps, first, lw.v_mix, lw.rot_amp, a.page_dim)
        if q_out is not None:
            q_out.copy_(q)

    def state_space(self, proj, lw, m, ssm_state, conv_state, spans, n_single, conv_buf, dt_buf, out):
        for row0, n, seen, slot in spans.tolist():
            u = proj[row0:row0 + n]
            if seen == 0:
                ssm_state[slot].zero_()
            xbc = ref.short_conv(u[:, m.inner:m.inner + m.conv_dim], conv_state[slot], lw.ssm_conv_w, lw.ssm_conv_b, seen)
            xbc = xbc.to(proj.dtype).float()
            GN = m.groups * m.state
            dt = torch.nn.functional.softplus(u[:, m.inner + m.conv_dim:].float() + lw.ssm_dt_bias)
            y = ref.selective_scan(xbc[:, :m.inner].reshape(n, m.heads, m.vdim), xbc[:, m.inner:m.inner + GN].reshape(n, m.groups, m.state),
                                   xbc[:, m.inner + GN:].reshape(n, m.groups, m.state), dt, lw.ssm_a, lw.ssm_d, ssm_state[slot])
            out[row0:row0 + n] = y.reshape(n, m.inner)
        return out

    def delta_rule(self, proj, lw, m, state, conv_state, spans, n_single, conv_buf, dt_buf, y, out, eps, workspace):
        C, GN = m.conv_dim, m.groups * m.state
        for row0, n, seen, slot in spans.tolist():
            u = proj[row0:row0 + n]
            if seen == 0:
                state[slot].zero_()
            vkq = ref.short_conv(u[:, m.inner:m.inner + C], conv_state[slot], lw.ssm_conv_w, lw.ssm_conv_b, seen).to(proj.dtype).float()
            decay, beta = u[:, m.inner + C:m.inner + C + m.heads].float(), u[:, m.inner + C + m.heads:m.in_dim].float()
            decay = torch.exp(lw.ssm_a * torch.nn.functional.softplus(decay + lw.ssm_dt_bias))
            v, k, q = vkq.split([m.inner, GN, GN], 1)
            o = ref.delta_scan(q.reshape(n, m.groups, m.state), k.reshape(n, m.groups, m.state), v.reshape(n, m.heads, m.vdim), decay,
                               torch.sigmoid(beta), state[slot])
            y[row0:row0 + n] = o.reshape(n, m.inner)
        if out is not None:
            out.copy_(ref.gated_norm(y, proj[:, :m.inner], lw.ssm_norm, m.heads, eps, gate_after=True))
        return y

    def gru(self, proj, lw, m, state, spans, n_single, out, workspace):
        C = m.inner
        for row0, n, seen, slot in spans.tolist():
            u, S = proj[row0:row0 + n].float(), state[slot].view(-1)
            if seen == 0:
                S.zero_()
            y = ref.gru_scan(u[:, :C] + lw.gru_bias[:C], u[:, C:2 * C] + lw.gru_bias[C:], S)
            if out is not None:
                out[row0:row0 + n] = y * torch.nn.functional.silu(u[:, 2 * C:3 * C])

    def linear_attention(self, q, k, v, gate, z, lw, m, state, spans, n_single, y, out, eps, workspace):
        NK, NV = m.heads * m.dim, m.heads * m.vdim
        for row0, n, seen, slot in spans.tolist():
            if seen == 0:
                state[slot].zero_()
            rows = slice(row0, row0 + n)
            decay = ref.linear_decay(z[rows, :NK].float() + lw.decay_bias, m.tau)
            split = lambda t, w: t[rows, :w].reshape(n, m.heads, w // m.heads)  # noqa: E731
            y[rows, :NV] = ref.linear_scan(split(q, NK), split(k, NK), split(v, NV), decay.view(n, m.heads, m.dim), state[slot]).reshape(n, NV)
        if out is not None:
            out.zero_()
            out[:, :NV] = ref.gated_norm(y[:, :NV], gate[:, :NV], lw.ssm_norm, m.heads, eps, gate_after=True)

    def retention_in_proj(self, x, lw, m, proj, qk, tok_pos, prompts, workspace=None):
        self.gemm(x, lw.w_qkv, proj)
        return (*proj.split([m.keys, m.keys, m.inner, m.inner], 1), False)

    def retention(self, q, k, v, gate, lw, m, turned, state, spans, n_single, y, out, eps, workspace):
        for row0, n, seen, slot in spans.tolist():
            if seen == 0:
                state[slot].zero_()
            pos = torch.arange(seen, seen + n)
            turned = lambda t: ref.rotate_halves(t[row0:row0 + n].reshape(n, m.heads, m.width), pos, lw.rot_freq, lw.rot_amp)  # noqa: E731
            y[row0:row0 + n] = ref.retention_scan(turned(q), turned(k), v[row0:row0 + n].reshape(n, m.heads, m.vwidth), lw.ret_decay, m.dim**-0.5,
                                                  state[slot]).reshape(n, m.inner)
        if out is not None:
            head_eps, scale = padded_head_norm(m, eps)
            out.copy_(ref.gated_norm(y, gate, lw.ssm_norm, m.heads, head_eps, scale, gate_after=True))

    def latent_append(self, proj, q_out, pages, tok_pos, tok_slot, c, lw, eps):
        n_q = c.heads * c.head_width
        if q_out is not None:
            q = proj[:, :n_q].reshape(-1, c.heads, c.head_width).clone()
            q[..., c.dim:c.dim + c.rot_dim] = ref.rotate_pairs(q[..., c.dim:c.dim + c.rot_dim], tok_pos, lw.rot_freq).to(q.dtype)
            q_out.copy_(q.reshape(q_out.shape))
        if pages is not None:
            rows = ref.latent_rows(proj[:, n_q:n_q + c.kv_rank + c.rot_dim], tok_pos, c.kv_rank, lw.rot_freq, lw.latent_norm, eps, c.page_width)
            pages[:, 0, 0].view(-1, c.page_width)[tok_slot.long()] = rows.to(pages.dtype)

    def latent_attention(self, q, out, pages, batch, c, lw, bufs, ws_large=None):
        q3 = q.view(-1, c.heads, c.head_width)
        lat = torch.cat([torch.einsum("thd,hdr->thr", q3[..., :c.dim].float(), lw.w_uk.float()), q3[..., c.dim:c.dim + c.rot_dim].float()], 2)
        mean = torch.zeros(q3.shape[0], c.heads, c.kv_rank)
        for items in (batch.items_small(), batch.items_large()):
            if items.shape[0]:
                ref.paged_latent_attention(lat, pages, batch.block_tables(), items, c.kv_rank, abs(c.scale) or 1.0, c.window, out=mean)
        v = torch.einsum("thr,hrv->thv", mean, lw.w_uv.float())
        out.copy_(torch.nn.functional.pad(v, (0, c.head_width - c.vdim)).reshape(out.shape))

    def gated_norm(self, y, z, weight, out, groups, eps, scale=1.0):
        out.copy_(ref.gated_norm(y, z, weight, groups, eps, scale))
        return out

    def table_route(self, ids, lw, f, bufs):
        self._picked = lw.moe_table[ids.long()].long()
        self._scores = torch.full(self._picked.shape, 1.0 / f.top)

    def softmax_route(self, x, lw, f, bufs):
        s = torch.softmax(ref.gemm(x, lw.w_router, out_dtype=torch.float32)[:, :f.experts], -1)
        self._picked = torch.topk(s + lw.router_bias, f.top, -1).indices
        self._scores = s.gather(-1, self._picked) * f.router_scale

    def sigmoid_route(self, x, lw, f, bufs):
        s = torch.sigmoid(ref.gemm(x, lw.w_router, out_dtype=torch.float32)[:, :f.experts])
        self._scores, self._picked = torch.topk(s, f.top, -1)

    def chosen_route(self, x, lw, f, bufs):
        z, self._picked = torch.topk(ref.gemm(x, lw.w_router, out_dtype=torch.float32)[:, :f.experts] + lw.router_bias, f.top, -1)
        self._scores = torch.softmax(z, -1)

    def routed_experts(self, x, ids, lw, f, act, base, out, bufs):
        """``out`` = ``base`` (None, or ``out`` itself) + the chosen experts' weighted outputs (the outputs of weighted inputs,
        where the routing says so)."""
        picked, inputs = self._picked, f.weighs_inputs
        acc = torch.zeros_like(out) if base is None else base.float().clone()
        for e, ew in enumerate(lw.experts):
            rows, place = (picked == e).nonzero(as_tuple=True)
            if rows.numel():
                xs, s = x.index_select(0, rows), self._scores[rows, place][:, None]
                h = ref.gemm((xs.float() * s).to(x.dtype) if inputs else xs, ew.w_up, act=act, gated=f.gated, limit=f.limit)
                acc.index_add_(0, rows, ref.gemm(h, ew.w_down).float() * (1.0 if inputs else s))
        out.copy_(acc)
        return out

    def table_moe(self, x, ids, lw, f, act, shared, out, bufs):
        self.table_route(ids, lw, f, bufs)
        return self.routed_experts(x, ids, lw, f, act, shared, out, bufs)

    # ---- misc ---------------------------------------------------------------------------------------
    def embed(self, ids, weight, out, pos_weight=None, tok_pos=None, pos_offset=0):
        out.copy_(ref.embed(ids, weight, pos_weight, tok_pos, pos_offset))
        return out

    def gather_rows(self, x, row_idx, out):
        out.copy_(x[row_idx.long()])
        return out

    def argmax(self, logits):
        return logits.float().argmax(-1).to(torch.int32)


class CudaOps:
    name = "sm_100a"

    #: at or below this many tokens the QKV projection runs as split-K GEMM + RoPE/append kernel (fills all
    #: SMs while streaming weights); above it the RoPE/KV epilogue is fused into the tcgen05 GEMM
    FUSED_QKV_MIN_TOKENS = 129

    def __init__(self):
        from . import kernels
        self.k = kernels

    def _fp8_act(self, a):
        """Per-token E4M3 quantisation of ``a`` into persistent buffers (no allocation in steady state)."""
        T, K = a.shape
        bufs = self.__dict__.setdefault("_fp8_bufs", {})
        q, s = bufs.get(K, (None, None))
        if q is None or q.shape[0] < T or q.device != a.device:
            cap = max(T, 0 if q is None else 2 * q.shape[0], 64)
            q = torch.empty(cap, K, dtype=torch.uint8, device=a.device)
            s = torch.empty(cap, dtype=torch.float32, device=a.device)
            bufs[K] = (q, s)
        return self.k.quantize_fp8_rows(a, q[:T], s[:T])

    def reserve_fp8(self, max_tokens: int, ks, device) -> None:
        """Size the activation-quantisation buffers up front (before any CUDA-graph capture)."""
        bufs = self.__dict__.setdefault("_fp8_bufs", {})
        for K in ks:
            bufs[K] = (torch.empty(max_tokens, K, dtype=torch.uint8, device=device),
                       torch.empty(max_tokens, dtype=torch.float32, device=device))

    def gemm(self, a, w, out, bias=None, act=0, gated=False, workspace=None, comm=None, tp_wait=False, tp_signal=False, limit=0.0):
        """``tp_wait``: ``a`` was all-gathered into this GPU's buffer by the peers' norm kernels — the first kernel that
        reads it acquires their flags. ``tp_signal``: the GEMM's last CTA releases ``out`` to the peers."""
        if isinstance(w, Fp8Weight):
            if tp_wait:
                comm.arm(wait=True)          # consumed by the activation quantiser, the first reader of `a`
            aq, a_s = self._fp8_act(a)
            if tp_signal:
                comm.arm(signal=True)
            return self.k.gemm_fp8(aq, a_s, w.q, w.scale, out, bias=bias, act=act, gated=gated,
                                   workspace=workspace if a.shape[0] <= 64 else None, w_fmt=w.fmt_code)
        if tp_wait or tp_signal:
            comm.arm(wait=tp_wait, signal=tp_signal)
        return self.k.gemm(a, w, bias=bias, act=act, gated=gated, out=out,
                           workspace=workspace if a.shape[0] <= 128 else None, limit=limit)

    def gemm_accum(self, a, w, accum, bias=None, comm=None, tp_signal=False):
        """``accum (fp32) += a @ w.T``. ``tp_signal`` (tensor parallel): the kernel's last CTA releases the partial sums
        to the peers; the reduction itself happens in ``norm_tp``."""
        if isinstance(w, Fp8Weight):
            if a.shape[0] > 64:
                raise NotImplementedError("fp8 weights: above 64 tokens the executor routes reducing GEMMs through the "
                                          "16-bit partial-sum buffer")
            aq, a_s = self._fp8_act(a)
            if tp_signal:
                comm.arm(signal=True)
            self.k.gemm_fp8_accum(aq, a_s, w.q, w.scale, accum, bias=bias, out_dtype=a.dtype, w_fmt=w.fmt_code)
            return
        if tp_signal:
            comm.arm(signal=True)
        self.k.gemm_accum(a, w, accum, bias=bias)

    def norm(self, x, gamma, out, beta=None, delta=None, zero_delta=False, res_out=None, eps=1e-5, layer_norm=False,
             comm=None, zero_buf=None, scatter_rows=None):
        """``comm`` set: ``delta`` is this rank's partial-sum buffer of a row-parallel GEMM (fp32 or 16-bit, symmetric
        memory) and the kernel performs the collective (see ``hds_norm_tp``). ``scatter_rows = (row0, n_rows)`` selects
        the reduce-scatter + all-gather shape: ``out`` (symmetric) is written on every rank and the kernel signals."""
        if comm is not None and delta is not None:
            comm.pre_wait()
            kw = {}
            if scatter_rows is not None:
                mc = comm.multicast_ptr(out, "st")
                kw = dict(row0=scatter_rows[0], n_rows=scatter_rows[1], signal=not comm.debug_nosync, out_mc=mc,
                          out_ptrs=None if mc else comm.peer_ptrs_raw(out))
            return self.k.norm_tp(comm.ctx, x, gamma, out, comm.peer_ptrs_raw(delta), src_mc=comm.multicast_ptr(delta, "ld"),
                                  partial_16bit=delta.dtype != torch.float32, zero_buf=zero_buf, beta=beta, res_out=res_out,
                                  eps=eps, layer_norm=layer_norm, wait=not comm.debug_nosync, **kw)
        return self.k.norm(x, gamma, out, beta=beta, delta=delta, zero_delta=zero_delta, res_out=res_out, eps=eps,
                           layer_norm=layer_norm)

    def qkv_rope_kv_append(self, x, w_qkv, b_qkv, qkv_buf, q_out, kv_layer, tok_pos, tok_slot, inv_freq, n_q, n_kv, d,
                           rot_dim, block_size, workspace=None, comm=None, tp_wait=False):
        T = x.shape[0]
        fusable = d in (64, 128) and (inv_freq is None or rot_dim == d)
        if isinstance(w_qkv, Fp8Weight):
            self.gemm(x, w_qkv, qkv_buf, bias=b_qkv, comm=comm, tp_wait=tp_wait)
            self.k.rope_kv_append(qkv_buf, q_out, kv_layer, tok_pos, tok_slot, inv_freq, n_q, n_kv, d, rot_dim, block_size)
        elif fusable and T >= self.FUSED_QKV_MIN_TOKENS:
            if tp_wait:
                comm.arm(wait=True)
            self.k.qkv_rope_proj(x, w_qkv, q_out, kv_layer, tok_pos, tok_slot, inv_freq, n_q, n_kv, d, block_size,
                                 bias_qkv=b_qkv)
        else:
            if tp_wait:
                comm.arm(wait=True)
            self.k.gemm(x, w_qkv, bias=b_qkv, out=qkv_buf, workspace=workspace if T <= 128 else None)
            self.k.rope_kv_append(qkv_buf, q_out, kv_layer, tok_pos, tok_slot, inv_freq, n_q, n_kv, d, rot_dim, block_size)

    def restore_kv_proj(self, latents, w_kv, b_kv, kv_layer, tok_pos, tok_slot, inv_freq, n_kv, d, rot_dim, block_size,
                        scratch=None):
        if isinstance(w_kv, Fp8Weight):
            if scratch is None or scratch.shape[0] < latents.shape[0]:
                scratch = torch.empty(latents.shape[0], w_kv.shape[0], dtype=latents.dtype, device=latents.device)
            scratch = scratch[:latents.shape[0]]
            self.gemm(latents, w_kv, scratch, bias=b_kv)
            self.k.rope_kv_append(scratch, scratch, kv_layer, tok_pos, tok_slot, inv_freq, 0, n_kv, d, rot_dim, block_size)
        elif latents.dtype == torch.float32:
            self.k.gemm(latents, w_kv, out=scratch)
            self.k.kv_append_generic(scratch, scratch, kv_layer, tok_slot, 0, n_kv, d, block_size)
        elif d in (64, 128) and (inv_freq is None or rot_dim == d):
            self.k.restore_kv_proj(latents, w_kv, kv_layer, tok_pos, tok_slot, inv_freq, n_kv, d, block_size, bias_kv=b_kv)
        else:
            # head sizes the fused epilogue does not cover: plain GEMM into scratch, then RoPE/append with zero
            # query heads (scratch: [T, 2 * n_kv * d])
            self.k.gemm(latents, w_kv, bias=b_kv, out=scratch)
            self.k.rope_kv_append(scratch, scratch, kv_layer, tok_pos, tok_slot, inv_freq, 0, n_kv, d, rot_dim, block_size)

    def attention(self, q, out, kv_layer, batch, n_q, n_kv, d, scale, ws_small=None, ws_large=None, alibi=None, window=0,
                  keep_first=0, sink=None, sigmoid_bias=None, gate=None, softcap=0.0):
        k = self.k
        bs = batch.block_size
        if q.dtype == torch.float32 or d not in (64, 128):
            k.paged_attention_generic(q, out, kv_layer, batch.block_tables(), batch.tokens_to_seq(), batch.tok_pos(), n_q, n_kv, d, bs,
                                      scale, window=window, keep_first=keep_first, sink=sink, sigmoid_bias=sigmoid_bias, gate=gate, softcap=softcap)
            return
        # with a sliding window an item reads at most window + one tile of keys: size the KV split for that
        seen = lambda n_kv_tokens: windowed_len(n_kv_tokens, window, keep_first)  # noqa: E731
        opts = dict(alibi=alibi, window=window, keep_first=keep_first, sink=sink, sigmoid_bias=sigmoid_bias, gate=gate, softcap=softcap)
        if batch.n_items_small:
            n = batch.n_items_small
            if use_packed_decode(n_q, n_kv, d):
                # grouped-query decode: the group's query heads share one pass over the KV pages, on the tensor cores
                splits = pick_packed_splits(n, n_kv, seen(batch.max_kv_len_small))
                k.paged_attention_prefill(q, out, kv_layer, batch.block_tables(), batch.items_small(), n, n_q, n_kv, d, bs,
                                          scale, n_splits=splits, workspace=ws_large if splits > 1 else None, packed=True, **opts)
            else:
                splits = pick_decode_splits(n, n_kv, seen(batch.max_kv_len_small))
                k.paged_attention_splitkv(q, out, kv_layer, batch.block_tables(), batch.items_small(), n,
                                          batch.rows_per_small_item, n_q, n_kv, d, bs, splits, scale, ws_small, **opts)
        if batch.n_items_large:
            n = batch.n_items_large
            splits = pick_prefill_splits(n, n_q, seen(batch.max_kv_len_large))
            k.paged_attention_prefill(q, out, kv_layer, batch.block_tables(), batch.items_large(), n, n_q, n_kv, d, bs,
                                      scale, n_splits=splits, workspace=ws_large if splits > 1 else None, **opts)

    # ---- stacks of unlike layers ----------------------------------------------------------------------
    def embed_f32(self, ids, weight, out, **kw):
        return self.k.embed_f32(ids, weight, out, **kw)

    def norm_residual(self, resid, gamma, out, **kw):
        return self.k.norm_residual(resid, gamma, out, **kw)

    def mixer_in_proj(self, x, lw, a, proj, q_out, kv_layer, first, tok_pos, tok_slot, block_size, eps, workspace=None):
        """Every projection that reads the layer's input: Q to ``q_out``, K / V to their pages, the rest to ``proj``'s columns
        behind those of the attention. Decode-size batches stream all weights in ONE GEMM; larger ones keep the QKV rows' fused
        rotating and paged epilogue (where no norm comes before it) and run the others as a second GEMM. ``first``: pages of the
        layer whose values are mixed in."""
        k, T, d, w_in, b = self.k, x.shape[0], a.page_dim, lw.w_qkv, lw.b_qkv
        n_in, n_attn, n_kv = w_in.shape[0], (a.heads + 2 * a.cached_heads) * d, a.cached_heads
        if x.dtype != torch.float32 and d in (64, 128) and T >= self.FUSED_QKV_MIN_TOKENS and not a.qk_norm:
            k.qkv_rope_proj(x, w_in[:n_attn], q_out, kv_layer, tok_pos, tok_slot, lw.rot_freq, a.heads, n_kv, d, block_size,
                            bias_qkv=None if b is None else b[:n_attn], amp=lw.rot_amp)
            if n_in > n_attn:
                k.gemm(x, w_in[n_attn:], out=proj[:, n_attn:n_in], bias=None if b is None else b[n_attn:])
            if first is not None:
                k.mix_cached_values(kv_layer, first, tok_slot, lw.v_mix, a.kv_heads, d, block_size)
            return
        self.gemm(x, w_in, proj[:, :n_in], bias=b, workspace=workspace)
        self.attention_append(proj, lw, a, q_out, kv_layer, first, tok_pos, tok_slot, block_size, eps)

    def attention_append(self, proj, lw, a, q_out, kv_layer, first, tok_pos, tok_slot, block_size, eps):
        """Projected rows [q | k | v] -> rotated (and normed) queries and page rows. ``q_out`` None: keys and values only."""
        k, d, n_q = self.k, a.page_dim, a.heads if q_out is not None else 0
        q_out = proj if q_out is None else q_out
        if a.rot is not None or a.qk_norm or first is not None or a.kv_from is not None:
            k.attention_append(proj, q_out, kv_layer, tok_pos, tok_slot, n_q, a.cached_heads, d, block_size, lw.rot_freq, lw.q_norm, lw.k_norm,
                               a.heads * a.dim, a.kv_heads * a.dim, eps, first, lw.v_mix, lw.rot_amp)
        elif proj.dtype == torch.float32:
            k.kv_append_generic(proj, q_out, kv_layer, tok_slot, n_q, a.kv_heads, d, block_size)
        else:
            k.rope_kv_append(proj, q_out, kv_layer, tok_pos, tok_slot, None, n_q, a.kv_heads, d, d, block_size)

    def gru(self, proj, lw, m, state, spans, n_single, out, workspace):
        self.k.gru(proj, lw.gru_bias, state, spans, n_single, out, workspace)

    def linear_attention(self, q, k, v, gate, z, lw, m, state, spans, n_single, y, out, eps, workspace):
        self.k.linear_attention(q, k, v, gate, z, lw.decay_bias, 1.0 / m.tau, state, spans, n_single, y, out, lw.ssm_norm, eps, workspace)

    def retention_in_proj(self, x, lw, m, proj, qk, tok_pos, prompts, workspace=None):
        """q, k, v, gate of retention, and whether q and k have been turned: in the epilogue of batches with ``prompts`` that are large
        enough, for the chunked kernels (which take them so); else the recurrence does it in fp32."""
        k, nk, nv = self.k, m.keys, m.inner
        if prompts and x.dtype == torch.bfloat16 and m.width in (64, 128) and x.shape[0] >= self.FUSED_QKV_MIN_TOKENS:
            k.qkv_rope_proj(x, lw.w_qkv[:2 * nk], qk, None, tok_pos, tok_pos, lw.rot_freq, 2 * m.heads, 0, m.width, 1, amp=lw.rot_amp)
            k.gemm(x, lw.w_qkv[2 * nk:], out=proj[:, 2 * nk:])
            return qk[:, :nk], qk[:, nk:], proj[:, 2 * nk:2 * nk + nv], proj[:, 2 * nk + nv:], True
        self.gemm(x, lw.w_qkv, proj, workspace=workspace)
        return (*proj.split([nk, nk, nv, nv], 1), False)

    def retention(self, q, k, v, gate, lw, m, turned, state, spans, n_single, y, out, eps, workspace):
        self.k.retention(q, k, v, gate, lw.ret_decay, None if turned else lw.rot_freq, lw.rot_amp, m.dim**-0.5, m.vdim, state, spans, n_single, y, out, lw.ssm_norm, eps,
                         workspace)

    def state_space(self, proj, lw, m, ssm_state, conv_state, spans, n_single, conv_buf, dt_buf, out):
        return self.k.state_space(proj, lw.ssm_conv_w, lw.ssm_conv_b, lw.ssm_dt_bias, lw.ssm_a, lw.ssm_d, ssm_state, conv_state, spans,
                                  n_single, m.groups, conv_buf, dt_buf, out)

    def gated_norm(self, y, z, weight, out, groups, eps, scale=1.0):
        return self.k.gated_norm(y, z, weight, out, groups, eps, scale)

    def table_route(self, ids, lw, f, bufs):
        """Experts by token id."""
        T = ids.numel()
        self.k.moe_table_route(ids, lw.moe_table, f.experts, bufs["scores"][:T], bufs["expert_ids"][:T], bufs["offsets"][:T], bufs["counts"])

    def softmax_route(self, x, lw, f, bufs):
        """Experts by router: fp32 scores (the product accumulates in fp32 and is never rounded), corrected choice."""
        k, T = self.k, x.shape[0]
        logits = bufs["logits"][:T]             # zero between calls: the gating kernel clears what it has read
        k.gemm_accum(x, lw.w_router, logits)
        k.moe_topk_gating(logits[:, :f.experts], f.top, False, bufs["scores"][:T], bufs["expert_ids"][:T], bufs["offsets"][:T], bufs["counts"],
                          bias=lw.router_bias, scale=f.router_scale, clear=True)

    def sigmoid_route(self, x, lw, f, bufs):
        """Experts by router: the largest sigmoids of fp32 logits."""
        k, T = self.k, x.shape[0]
        logits = bufs["logits"][:T]
        k.gemm_accum(x, lw.w_router, logits)
        k.moe_topk_gating(logits[:, :f.experts], f.top, False, bufs["scores"][:T], bufs["expert_ids"][:T], bufs["offsets"][:T], bufs["counts"],
                          clear=True, sigmoid=True)

    def chosen_route(self, x, lw, f, bufs):
        """Experts by router: the largest fp32 logits, bias included, weighed by the softmax over them."""
        k, T = self.k, x.shape[0]
        logits = bufs["logits"][:T]
        k.gemm_accum(x, lw.w_router, logits)
        k.moe_topk_gating(logits[:, :f.experts], f.top, True, bufs["scores"][:T], bufs["expert_ids"][:T], bufs["offsets"][:T], bufs["counts"],
                          bias=lw.router_bias, clear=True, biased=True)

    def routed_experts(self, x, ids, lw, f, act, base, out, bufs):
        """Routed tokens: scatter -> grouped GEMM -> grouped GEMM -> weighted sum, added to ``base`` (``out`` itself: in place)."""
        k, T, E = self.k, x.shape[0], f.experts
        rows = k.moe_padded_rows(T, E, f.top)
        xs, hs, ys = bufs["xs"][:rows], bufs["hs"][:rows], bufs["ys"][:rows]
        ids_e, off, slots = bufs["expert_ids"][:T], bufs["offsets"][:T], bufs["mapped_slots"][:T]
        scores = bufs["scores"][:T]
        k.moe_scatter(x, xs, ids_e, off, bufs["counts"], bufs["pad_off"], slots, f.top, scores if f.weighs_inputs else None)
        k.moe_gemm(xs, lw.moe_up, bufs["pad_off"], E, hs, act=act, gated=f.gated, limit=f.limit)
        k.moe_gemm(hs, lw.moe_down, bufs["pad_off"], E, ys)
        return k.moe_combine(ys, slots, None if f.weighs_inputs else scores, base, out)

    def table_moe(self, x, ids, lw, f, act, shared, out, bufs):
        self.table_route(ids, lw, f, bufs)
        return self.routed_experts(x, ids, lw, f, act, shared, out, bufs)

    # ---- latent attention -----------------------------------------------------------------------------
    def latent_append(self, proj, q_out, pages, tok_pos, tok_slot, c, lw, eps):
        self.k.latent_append(proj, q_out, pages, tok_pos, tok_slot, c.heads, c.dim, c.rot_dim, c.head_width, c.kv_rank, lw.rot_freq,
                             lw.latent_norm, eps)

    def latent_attention(self, q, out, pages, batch, c, lw, bufs, ws_large=None):
        """Decode steps and short portions in the latent space; prompts on K / V pages projected from the cached rows they see (as
        long as those fit the scratch pages)."""
        k, T, bs, D = self.k, q.shape[0], batch.block_size, c.head_width
        plan, scale = None, abs(c.scale) or 1.0
        if lw.w_kv is not None and batch.n_items_large and T > batch.current_sequences:
            plan = batch.visible_pages(c.window, bufs.blocks)
        generic = q.dtype == torch.float32 or not k.latent_attention_supported(c.kv_rank, c.page_width)
        limit = batch.small_item_tokens if plan is not None else 1 << 30     # sequences with more new tokens take the other path
        if generic or batch.n_items_small or plan is None:
            lat, mean = bufs.queries(T, c), bufs.means(T, c)
            k.head_matmul(q, lw.w_uk, lat, batch.tokens_to_seq(), batch.spans(), limit, in_width=D, out_width=c.page_width, copy=c.rot_dim)
            if generic:
                k.paged_attention_generic(lat, mean, pages, batch.block_tables(), batch.tokens_to_seq(), batch.tok_pos(), c.heads, 1,
                                          c.page_width, bs, scale, window=c.window, value_dim=c.kv_rank, spans=batch.spans(), limit=limit)
            else:
                for items, n, tokens, splits in latent_launches(batch, c.heads, c.kv_rank, c.page_width, c.window, plan is None):
                    k.paged_attention_latent(lat, mean, pages, batch.block_tables(), batch.items_small() if items == "small" else
                                             batch.items_large(), n, tokens, c.heads, c.kv_rank, bs, splits, scale, bufs.workspace, c.window)
            k.head_matmul(mean, lw.w_uv, out, batch.tokens_to_seq(), batch.spans(), limit, in_width=c.kv_rank, out_width=D, copy=0)
        if plan is not None:
            ids, tables = plan
            n = ids.numel()
            k.kv_blocks_copy(pages[None], bufs.rows[:n], ids, to_staging=True)
            kv = bufs.kv_pages(n, c)
            k.restore_kv_proj(bufs.rows.view(-1)[:n * bs * c.page_width].view(n * bs, c.page_width), lw.w_kv, kv, bufs.slots[:n * bs],
                              bufs.slots[:n * bs], None, c.heads, D, bs)
            n_items = batch.n_items_large
            splits = pick_prefill_splits(n_items, c.heads, windowed_len(batch.max_kv_len_large, c.window))
            k.paged_attention_prefill(q, out, kv, tables, batch.items_large(), n_items, c.heads, c.heads, D, bs, scale, n_splits=splits,
                                      workspace=ws_large if splits > 1 else None, window=c.window)

    # ---- gated delta rule -----------------------------------------------------------------------------
    def delta_rule(self, proj, lw, m, state, conv_state, spans, n_single, conv_buf, dt_buf, y, out, eps, workspace):
        return self.k.delta_rule(proj, lw.ssm_conv_w, lw.ssm_conv_b, lw.ssm_dt_bias, lw.ssm_a, state, conv_state, spans, n_single, m.groups,
                                 conv_buf, dt_buf, y, out, lw.ssm_norm, eps, workspace)

    def embed(self, ids, weight, out, pos_weight=None, tok_pos=None, pos_offset=0):
        return self.k.embed(ids, weight, out, pos_weight=pos_weight, tok_pos=tok_pos, pos_offset=pos_offset)

    def gather_rows(self, x, row_idx, out):
        return self.k.gather_rows(x, row_idx, out)

    def argmax(self, logits):
        return self.k.argmax(logits)


N_SM = 148
MAX_DECODE_SPLITS = 16
MAX_PREFILL_SPLITS = 16


def pick_decode_splits(n_items: int, n_kv_heads: int, max_kv_len: int) -> int:
    """KV splits for the split-KV kernel. Up to one CTA per SM: split until (items x kv heads x splits) fills the SMs —
    measured (profiles/kernel_bench_attn_warps.txt): 32 CTAs -> 4 splits, 64 -> 2. Up to the 2 x 148 resident slots of
    the 4-warp configuration: one wave, no split. Beyond that a second, mostly empty wave would cost up to half the
    bandwidth (320 CTAs: 3.8 TB/s unsplit vs 5.1 TB/s with 4 splits, profiles/kernel_bench_attn_waves.txt): take the
    smallest split count whose waves are at least 85 % full. Each split keeps at least 2 tiles (256 keys)."""
    ctas = max(1, n_items * n_kv_heads)
    tiles = max(1, (max_kv_len + 127) // 128)
    cap = max(1, min(MAX_DECODE_SPLITS, tiles // 2 if tiles >= 2 else 1))
    slots = 2 * N_SM
    if ctas <= N_SM:
        want = max(1, N_SM // ctas)
    elif ctas <= slots:
        want = 1
    else:
        want, best = 1, 0.0
        for s in range(1, min(cap, 8) + 1):
            eff = ctas * s / (slots * -(-ctas * s // slots))
            if eff >= 0.85:
                want = s
                break
            if eff > best:
                want, best = s, eff
    return int(max(1, min(want, cap)))


#: grouped-query decode goes to the tensor-core kernel from this group size on (HDS_GQA_PACKED=0 keeps the SIMT kernel)
PACKED_MIN_GROUP = 4


def use_packed_decode(n_q_heads: int, n_kv_heads: int, head_dim: int) -> bool:
    import os
    G = n_q_heads // max(1, n_kv_heads)
    return (head_dim == 128 and G >= PACKED_MIN_GROUP and 128 % G == 0 and os.environ.get("HDS_GQA_PACKED", "1") != "0")


def pick_packed_splits(n_items: int, n_kv_heads: int, max_kv_len: int) -> int:
    """KV splits of the head-packed decode kernel (one CTA per SM): as many as keep (items x KV heads x splits) within
    one wave of CTAs; each split keeps at least 2 tiles of 128 keys."""
    ctas = max(1, n_items * n_kv_heads)
    tiles = max(1, (max_kv_len + 127) // 128)
    cap = max(1, min(MAX_PREFILL_SPLITS, tiles // 2 if tiles >= 2 else 1))
    return int(max(1, min(cap, N_SM // ctas)))


def pick_prefill_splits(n_items: int, n_q_heads: int, max_kv_len: int) -> int:
    """KV splits for the tensor-core kernel: one CTA per SM when (items x heads) alone cannot fill the GPU."""
    ctas = max(1, n_items * n_q_heads)
    if ctas >= N_SM:
        return 1
    want = (N_SM + ctas - 1) // ctas
    tiles = max(1, (max_kv_len + 127) // 128)
    return int(max(1, min(want, MAX_PREFILL_SPLITS, tiles // 2 if tiles >= 2 else 1)))


def latent_launches(batch, heads: int, rank: int, width: int, window: int, with_large: bool):
    """Launches of the latent attention kernel for a batch: (item list, items, tokens per item at most, KV splits)."""
    out = []
    if batch.n_items_small:
        out.append(("small", batch.n_items_small, batch.rows_per_small_item // batch.group, batch.max_kv_len_small))
    if with_large and batch.n_items_large:
        out.append(("large", batch.n_items_large, batch.max_large_item_tokens, batch.max_kv_len_large))
    launches = []
    for kind, n, tokens, kv_len in out:
        launches.append((kind, n, tokens, latent_splits(n, tokens, heads, rank, width, kv_len, window)))
    return tuple(launches)


def latent_splits(n_items: int, item_tokens: int, heads: int, rank: int, width: int, max_kv_len: int, window: int) -> int:
    """KV splits of the latent attention kernel: one wave of CTAs at most, at least one tile each."""
    from .kernels import latent_attention_ctas
    ctas, tile = latent_attention_ctas(item_tokens, heads, rank, width)
    tiles = max(1, -(-(min(max_kv_len, window) if window else max_kv_len) // tile))
    return int(max(1, min(MAX_PREFILL_SPLITS, N_SM // (n_items * ctas), tiles)))


class LatentBuffers:
    """Scratch of latent attention, shared by all layers: queries and results in the latent space, and the pages that prompts
    project their context to. ``blocks``: pages that scratch holds (a batch that sees more attends in the latent space)."""

    def __init__(self, layers, state_config, block_size: int, dtype: torch.dtype, device: torch.device) -> None:
        T, S, W = state_config.max_ragged_batch_size, state_config.max_ragged_sequence_count, max(c.page_width for c in layers)
        self._dtype, self._device, self._bs = dtype, device, block_size
        self._flat = {}
        expanding = [c for c in layers if c.head_width <= 128] if dtype != torch.float32 else []
        self.blocks = 0
        if expanding:
            seen = max(min(c.window or state_config.max_context, state_config.max_context) for c in expanding)
            per_block = max(2 * c.heads * c.head_width for c in expanding) * block_size * 2
            want = -(-T // block_size) + min(S, 8) * (-(-seen // block_size) + 3)
            self.blocks = max(1, min(want, (2 << 30) // per_block))
            self.rows = torch.zeros(self.blocks, 1, 1, 1, block_size, W, dtype=dtype, device=device)
            self._kv = torch.zeros(self.blocks * per_block // 2, dtype=dtype, device=device)
            self.slots = torch.arange(self.blocks * block_size, dtype=torch.int32, device=device)
        self.workspace = None
        if dtype != torch.float32:
            from . import kernels
            self.workspace = torch.zeros(kernels.latent_attention_workspace_bytes(), dtype=torch.uint8, device=device)
        for c in layers:       # decode steps find their buffers in place (a graph cannot allocate them)
            self.queries(min(T, 8 * S), c)
            self.means(min(T, 8 * S), c)

    def _get(self, name: str, n: int) -> torch.Tensor:
        t = self._flat.get(name)
        if t is None or t.numel() < n:
            t = self._flat[name] = torch.zeros(n, dtype=self._dtype, device=self._device)
        return t[:n]

    def queries(self, T: int, c) -> torch.Tensor:
        return self._get("queries", T * c.heads * c.page_width).view(T, c.heads * c.page_width)

    def means(self, T: int, c) -> torch.Tensor:
        return self._get("means", T * c.heads * c.kv_rank).view(T, c.heads * c.kv_rank)

    def kv_pages(self, n: int, c) -> torch.Tensor:
        size = 2 * c.heads * self._bs * c.head_width
        return self._kv[:n * size].view(n, 2, c.heads, self._bs, c.head_width)


def get_ops(device: torch.device):
    return CudaOps() if device.type == "cuda" else CpuOps()
