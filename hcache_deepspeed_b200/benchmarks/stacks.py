"""Throughput of stacks that mix attention with recurrent state, beside the closest families at equal sizes.

``bench.py --stacks``. Four layers of each size, random weights, through the public engine: one 4096-token prompt, and decode steps
of 8 and 64 sequences at 4096 tokens of context. Then the kernels that only such stacks use, each next to its counterpart in a
plain family: CUDA-event medians with an L2-sized flush between launches, as fractions of the measured peaks.
"""
from __future__ import annotations

import json
import os
import statistics
from typing import Callable, Dict, Optional

import torch

GROUPS = [("dedelorn-2048", "nipolorn-2048", "mistral-2048"), ("dedelorn-4096", "nipolorn-4096", "mistral-4096"),
          ("relulix-2048", "lotelix-2048", "dedelorn-2048-moe"), ("relulix-4096", "lotelix-4096", "dedelorn-4096-moe", "nipolorn-4096-moe", "qwen2-moe-4096")]
PROMPT = 4096


def peaks() -> Dict[str, float]:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    out = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    if os.path.exists(path):
        with open(path) as f:
            out.update({k: v for k, v in json.load(f).items() if k in out})
    return out


def _time(fn: Callable[[], None], iters: int, warmup: int, before: Optional[Callable[[], None]] = None) -> float:
    """Median milliseconds of ``fn`` on the device; ``before`` runs untimed in front of every iteration."""
    times = []
    for i in range(warmup + iters):
        if before is not None:
            before()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        b.synchronize()
        if i >= warmup:
            times.append(a.elapsed_time(b))
    return statistics.median(times)


def bench_engine(name: str, steps: int, warmup: int) -> Dict[str, float]:
    from ..inference.v2 import RaggedInferenceEngineConfig, build_engine_from_arch
    from ..models.arch import named_arch
    spec = named_arch(name)
    eng = build_engine_from_arch(spec, RaggedInferenceEngineConfig(
        state_manager={"max_tracked_sequences": 66, "max_ragged_batch_size": PROMPT, "max_ragged_sequence_count": 64, "max_context": PROMPT + 256,
                       "memory_config": {"mode": "tokens", "size": 66 * (PROMPT + 256)}, "max_state_slots": 66},
        hcache={"enabled": False, "capture": "off"}), seed=1, dtype=torch.bfloat16, device=torch.device("cuda"))
    g = torch.Generator().manual_seed(0)
    prompt = torch.randint(0, spec.vocab, (PROMPT, ), generator=g)
    out = {}
    ms = _time(lambda: eng.put([999], [prompt]), steps, warmup, before=lambda: eng.flush(999) if eng.state_manager.get_sequence(999) else None)
    eng.flush(999)
    out["prefill_ms"], out["prefill_tokens_per_s"] = round(ms, 3), round(PROMPT / ms * 1e3)
    for uid in range(64):
        eng.put([uid], [prompt])
    for n in (8, 64):
        uids = list(range(n))
        cur = [torch.randint(0, spec.vocab, (1, ), generator=g) for _ in uids]
        ms = _time(lambda: eng.put(uids, cur), 4 * steps, warmup + 4)
        out[f"decode{n}_ms"], out[f"decode{n}_tokens_per_s"] = round(ms, 4), round(n / ms * 1e3)
    out["weights_MiB"] = round(eng.model().w.n_bytes() / 2**20)
    return out


def _rnd(*shape, dtype=torch.bfloat16, scale=1.0):
    return (torch.randn(shape, device="cuda") * scale).to(dtype)


def _reporter(p: Dict[str, float], iters: int, warmup: int):
    flush = torch.empty(512 << 20, dtype=torch.uint8, device="cuda")

    def report(op, kernel, fn, bytes_=0.0, flops=0.0):
        ms = _time(fn, iters, warmup, before=flush.zero_)
        need = max(bytes_ / (p["hbm_gbs"] * 1e6), flops / (p["bf16_tflops"] * 1e9))     # ms at the measured peaks
        print(json.dumps({"op": op, "kernel": kernel, "us": round(ms * 1e3, 1), "roofline_us": round(need * 1e3, 1),
                          "bound": "memory" if bytes_ / (p["hbm_gbs"] * 1e6) >= flops / (p["bf16_tflops"] * 1e9) else "math",
                          "of_measured_peak": round(need / ms, 3)}), flush=True)

    return report


def bench_kernels(p: Dict[str, float], iters: int, warmup: int) -> None:
    """Kernels of a stack next to the like kernel of a plain family (``like``), with bytes or flops that the operation itself
    needs. Sizes: width 4096, 32 / 8 attention heads of 128, 128 state-space heads of 64 x 128 in 8 groups."""
    from ..ops import kernels as K
    dev, bf, rnd, report = "cuda", torch.bfloat16, _rnd, _reporter(p, iters, warmup)
    W, T = 4096, PROMPT

    for rows in (T, 64):
        x32, x16, d16, out = rnd(rows, W, dtype=torch.float32), rnd(rows, W), rnd(rows, W), rnd(rows, W)
        g32, g16 = torch.ones(W, device=dev), torch.ones(W, device=dev, dtype=bf)
        report(f"norm {rows}x{W}", "norm_residual", lambda: K.norm_residual(x32, g32, out, delta=d16, post=g32, eps=1e-5), rows * W * (4 + 4 + 2 + 2))
        report(f"norm {rows}x{W}", "norm (like)", lambda: K.norm(x16, g16, out, delta=d16, res_out=x16, eps=1e-5), rows * W * (2 + 2 + 2 + 2))
    heads, P, N, G = 128, 64, 128, 8
    inner, C = heads * P, heads * P + 2 * G * N
    ld = 2 * inner + 2 * G * N + heads
    vec = lambda n: torch.randn(n, device=dev) * 0.5  # noqa: E731
    cw, cb, db, a, d = torch.randn(4, C, device=dev) * 0.5, vec(C), vec(heads) - 3, -torch.exp(vec(heads)), vec(heads)
    for rows, seqs in ((T, 1), (T, 4), (64, 64), (8, 8)):
        n = rows // seqs
        proj = rnd(rows, ld)
        state, ring = torch.zeros(seqs, heads, P, N, device=dev), torch.zeros(seqs, 4, C, device=dev)
        spans = torch.tensor([[i * n, n, 128, i] for i in range(seqs)], dtype=torch.int32, device=dev)
        u, dt, y = torch.zeros(rows, C, dtype=bf, device=dev), torch.zeros(rows, heads, device=dev), torch.zeros(rows, inner, device=dev)
        single = seqs if n == 1 else 0
        # algorithmic bytes: projections in, y out, the states in and out
        need = rows * (C * 2 + heads * 2 + inner * 4) + 2 * seqs * (heads * P * N + 4 * C) * 4
        report(f"state space {seqs}x{n}", "conv + chunked scan" if n > 1 else "step", lambda: K.state_space(
            proj, cw, cb, db, a, d, state, ring, spans, single, G, u, dt, y), need)
        mix, w = rnd(rows, inner), torch.ones(inner, device=dev)
        report(f"gated norm {rows}x{inner}", "gated_norm", lambda: K.gated_norm(y, proj[:, :inner], w, mix, G, 1e-5, 0.5), rows * inner * (4 + 2 + 2))
    from ..ops.backend import latent_splits, pick_packed_splits, windowed_len
    nq, nkv, D, page = 32, 8, 128, 64
    ws = torch.zeros(256 << 20, dtype=torch.uint8, device=dev)
    for window, keep in ((0, 0), (1024, 0), (1024, 64), (4096, 64)):
        cache = rnd(T // page + 1, 2, nkv, page, D)
        table = torch.randperm(T // page, device=dev).to(torch.int32)[None].contiguous()
        q, o = rnd(T, nq * D), rnd(T, nq * D)
        items = torch.tensor([[0, i, 128, i] for i in range(0, T, 128)], dtype=torch.int32, device=dev)
        pairs = sum(i + 1 if not window else min(i + 1, window + max(0, min(keep, i + 1 - window))) for i in range(T))
        report(f"attention prefill {T} window {window} keep {keep}", "paged_attention_prefill" + ("" if window or keep else " (like)"), lambda:
               K.paged_attention_prefill(q, o, cache, table, items, T // 128, nq, nkv, D, page, 0.09, window=window, keep_first=keep),
               flops=4.0 * pairs * nq * D)
    B = 64
    for window, keep in ((0, 0), (1024, 0), (1024, 64)):
        cache = rnd(B * T // page, 2, nkv, page, D)
        tables = torch.randperm(B * T // page, device=dev).to(torch.int32).view(B, T // page).contiguous()
        q, o = rnd(B, nq * D), rnd(B, nq * D)
        items = torch.tensor([[i, i, 1, T - 1] for i in range(B)], dtype=torch.int32, device=dev)
        keys = T if not window else min(T, window + keep)
        sp = pick_packed_splits(B, nkv, windowed_len(T, window, keep))
        report(f"attention decode {B}x{T} window {window} keep {keep}", "paged_attention_packed" + ("" if window or keep else " (like)"), lambda:
               K.paged_attention_prefill(q, o, cache, tables, items, B, nq, nkv, D, page, 0.09, n_splits=sp, workspace=ws, packed=True,
                                         window=window, keep_first=keep), B * keys * 2 * nkv * D * 2)
    del cache
    # gated delta rule: 32 heads of 128 x 128, 16 groups; norm and gate behind it included
    heads, P, N, G = 32, 128, 128, 16
    inner, C = heads * P, heads * P + 2 * G * N
    cw, cb, db, a = torch.randn(4, C, device=dev) * 0.5, torch.zeros(C, device=dev), vec(heads) - 3, -torch.exp(vec(heads))
    for rows, seqs in ((T, 1), (T, 4), (64, 64), (8, 8)):
        n = rows // seqs
        proj = rnd(rows, inner + C + 2 * heads)
        state, ring = torch.zeros(seqs, heads, P, N, device=dev), torch.zeros(seqs, 4, C, device=dev)
        spans = torch.tensor([[i * n, n, 128, i] for i in range(seqs)], dtype=torch.int32, device=dev)
        u, dt, y = torch.zeros(rows, C, dtype=bf, device=dev), torch.zeros(rows, heads, device=dev), torch.zeros(rows, inner, device=dev)
        mix, w = rnd(rows, inner), torch.ones(inner, device=dev)
        dws = torch.empty(K.delta_workspace_bytes(rows, seqs, heads, G), dtype=torch.uint8, device=dev) if n > 1 else None
        moved = 2 * seqs * (heads * P * N + 4 * C) * 4
        if n > 1:
            report(f"delta rule {seqs}x{n}", "conv + chunked delta rule", lambda: K.delta_rule(
                proj, cw, cb, db, a, state, ring, spans, 0, G, u, dt, y, None, w, 1e-5, dws), rows * (C * 2 + 2 * heads * 2 + inner * 4) + moved)
            report(f"norm + gate {rows}x{inner}", "gated_norm", lambda: K.gated_norm(y, proj[:, :inner], w, mix, heads, 1e-5, gate_after=True),
                   rows * inner * (4 + 2 + 2))
        else:
            report(f"delta rule {seqs}x{n}", "step with norm and gate", lambda: K.delta_rule(
                proj, cw, cb, db, a, state, ring, spans, seqs, G, u, dt, y, mix, w, 1e-5), rows * (C * 2 + 2 * heads * 2 + inner * 4) + moved)
    # latent attention: 32 heads of 96 + 32 rotated, values of 128, latents of 512
    nh, dim, rot, rank, hw, width = 32, 96, 32, 512, 128, 576
    from ..models.hybrid import rotation_frequencies
    freq, gl = rotation_frequencies(rot, 1e4).to(dev), torch.ones(rank, device=dev)
    for rows in (T, 64):
        proj, q = rnd(rows, nh * hw + rank + rot), rnd(rows, nh * hw)
        pages = rnd(rows // page + 1, 1, 1, page, width)
        pos = torch.arange(rows, dtype=torch.int32, device=dev)
        report(f"latent append {rows}", "latent_append", lambda: K.latent_append(proj, q, pages, pos, pos, nh, dim, rot, hw, rank, freq, gl, 1e-5),
               rows * (2 * nh * hw + 2 * rank + rot + width) * 2)
        qkv, cache = rnd(rows, (nh + 16) * 128), rnd(rows // page + 1, 2, 8, page, 128)
        report(f"latent append {rows}", "rope_kv_append (like)", lambda: K.rope_kv_append(qkv, q, cache, pos, pos, torch.ones(64, device=dev), 32, 8, 128,
                                                                                        128, page), rows * 2 * (nh + 16) * 128 * 2)
    lws = torch.zeros(K.latent_attention_workspace_bytes(), dtype=torch.uint8, device=dev)
    for B, window in ((64, 0), (64, 1024), (8, 1024)):
        pages = rnd(B * T // page, 1, 1, page, width)
        tables = torch.randperm(B * T // page, device=dev).to(torch.int32).view(B, T // page).contiguous()
        lat, mean = rnd(B, nh * width, scale=0.1), rnd(B, nh * rank)
        items = torch.tensor([[i, i, 1, T - 1] for i in range(B)], dtype=torch.int32, device=dev)
        sp = latent_splits(B, 1, nh, rank, width, T, window)
        keys = T if not window else min(T, window)
        report(f"latent attention decode {B}x{T} window {window}", "paged_attention_latent", lambda: K.paged_attention_latent(
            lat, mean, pages, tables, items, B, 1, nh, rank, page, sp, 0.09, lws, window), B * keys * (rank + rot) * 2)
    del pages
    seq, spans = torch.arange(64, dtype=torch.int32, device=dev), torch.ones(64, 4, dtype=torch.int32, device=dev)
    wk, wv = rnd(nh, dim, rank, scale=0.02), rnd(nh, rank, 128, scale=0.02)
    for B in (64, 8):
        q, lat, mean, o = rnd(B, nh * hw), rnd(B, nh * width), rnd(B, nh * rank), rnd(B, nh * 128)
        report(f"queries to latents {B}", "head_matmul", lambda: K.head_matmul(q, wk, lat, seq, spans, 8, hw, width, rot),
               (wk.numel() + q.numel() + lat.numel()) * 2)
        report(f"latents to values {B}", "head_matmul", lambda: K.head_matmul(mean, wv, o, seq, spans, 8, rank, 128), (wv.numel() + mean.numel() + o.numel()) * 2)
    rows16, w_kv = rnd(T, width), rnd(2 * nh * hw, width, scale=0.02)
    kv = rnd(T // page, 2, nh, page, hw)
    slot = torch.arange(T, dtype=torch.int32, device=dev)
    report(f"latents to K / V pages {T}", "restore_kv_proj", lambda: K.restore_kv_proj(rows16, w_kv, kv, slot, slot, None, nh, hw, page),
           bytes_=(rows16.numel() + w_kv.numel() + kv.numel()) * 2, flops=2.0 * T * w_kv.numel())
    q, o = rnd(T, nh * hw), rnd(T, nh * hw)
    table = torch.arange(T // page, dtype=torch.int32, device=dev)[None].contiguous()
    items = torch.tensor([[0, i, 128, i] for i in range(0, T, 128)], dtype=torch.int32, device=dev)
    for window in (0, 1024):
        pairs = sum(min(i + 1, window or T) for i in range(T))
        report(f"latent attention prefill {T} window {window}", "paged_attention_prefill on projected pages", lambda: K.paged_attention_prefill(
            q, o, kv, table, items, T // 128, nh, nh, hw, page, 0.09, window=window), flops=2.0 * pairs * nh * (dim + rot + 128))
    del kv, q, o
    ff = 14336
    w_up = rnd(2 * ff, W, scale=0.02)
    wsg = torch.zeros(K.gemm_splitk_workspace_bytes(128, 2 * ff), dtype=torch.uint8, device=dev)
    for rows in (T, 64, 8):
        x, h = rnd(rows, W), rnd(rows, ff)
        for act, tag in ((5, "gated GEMM, clamped"), (4, "gated GEMM, gelu"), (3, "gated GEMM, silu (like)")):
            report(f"mlp up {rows}x{2 * ff}x{W}", tag, lambda: K.gemm(x, w_up, out=h, act=act, gated=True, limit=7.0,
                                                                       workspace=wsg if rows <= 128 else None),
                   2 * (2 * ff * W + rows * (W + ff)), 2.0 * rows * 2 * ff * W)
    E, top, V = 16, 2, 32000
    i32 = lambda *s: torch.zeros(s, dtype=torch.int32, device=dev)  # noqa: E731
    table = torch.stack([torch.randperm(E, device=dev)[:top] for _ in range(256)]).int().repeat(V // 256, 1).contiguous()
    for rows in (T, 64):
        scores, e, off, slots, counts, pad = torch.zeros(rows, top, device=dev), i32(rows, top), i32(rows, top), i32(rows, top), i32(E), i32(E + 1)
        R = K.moe_padded_rows(rows, E, top)
        x, xs, ys, base, out, lg = rnd(rows, W), rnd(R, W), rnd(R, W), rnd(rows, W), torch.zeros(rows, W, device=dev), rnd(rows, E)
        ids = torch.randint(0, V, (rows, ), device=dev).int()

        def by_table():
            K.moe_table_route(ids, table, E, scores, e, off, counts)
            K.moe_scatter(x, xs, e, off, counts, pad, slots, top)

        def by_gate():
            K.moe_topk_gating(lg, top, True, scores, e, off, counts)
            K.moe_scatter(x, xs, e, off, counts, pad, slots, top)

        report(f"route + scatter {rows}", "table", by_table, rows * W * 2 * (1 + top))
        report(f"route + scatter {rows}", "top-k gate (like)", by_gate, rows * W * 2 * (1 + top))
        wr, lg32, bias = rnd(E, W, scale=0.02), torch.zeros(rows, E, device=dev), torch.zeros(E, device=dev)

        def by_corrected_gate():
            K.gemm_accum(x, wr, lg32)
            K.moe_topk_gating(lg32, top, False, scores, e, off, counts, bias=bias, scale=2.5, clear=True)
            K.moe_scatter(x, xs, e, off, counts, pad, slots, top)

        report(f"router + route + scatter {rows}", "fp32 scores, corrected top-k gate", by_corrected_gate, rows * W * 2 * (2 + top))

        def by_gate_too():
            K.gemm(x, wr, out=lg)
            by_gate()

        report(f"router + route + scatter {rows}", "16-bit router, top-k gate (like)", by_gate_too, rows * W * 2 * (2 + top))
        report(f"combine {rows}", "moe_combine + shared", lambda: K.moe_combine(ys, slots, scores, base, out), rows * W * (2 * top + 2 + 4))
        report(f"combine {rows}", "moe_gather (like)", lambda: K.moe_gather(ys, slots, scores, out), rows * W * (2 * top + 4 + 4))


def bench_lotelix_kernels(p: Dict[str, float], iters: int, warmup: int) -> None:
    """The same for what Lotelix adds: minGRU, gated linear attention (32 heads of 128 x 128), sinks, sigmoid weights, gates, normed and
    rotated inputs, mixed values, grouped norms, weighted expert inputs."""
    from ..ops import kernels as K
    from ..ops.backend import pick_packed_splits, windowed_len
    dev, bf, f32, rnd, report = "cuda", torch.bfloat16, torch.float32, _rnd, _reporter(p, iters, warmup)
    W, T = 4096, PROMPT
    for rows in (T, 64):
        x, g, g2, out = rnd(rows, W, dtype=f32), torch.ones(W, device=dev), torch.ones(W, device=dev), rnd(rows, W)
        a, b, h = rnd(rows, W), rnd(rows, W), rnd(rows, W)
        report(f"norm {rows}x{W}", "norm_residual, 2 groups", lambda: K.norm_residual(x, g, out, delta=a, eps=1e-5, groups=2), rows * W * (4 + 4 + 2 + 2))
        report(f"norm {rows}x{W}", "norm_residual, two normed outputs", lambda: K.norm_residual(
            x, g, out, delta=a, post=g, eps=1e-5, groups=2, delta2=b, post2=g2), rows * W * (4 + 4 + 2 + 2 + 2))
        report(f"norm {rows}x{W}", "norm (like)", lambda: K.norm(h, g.to(bf), out, delta=a, res_out=h, eps=1e-5), rows * W * (2 + 2 + 2 + 2))
    bias = rnd(2 * W, dtype=f32)
    heads, N, P = 32, 128, 128
    for rows, seqs in ((T, 1), (T, 4), (64, 64), (8, 8)):
        n = rows // seqs
        single = seqs if n == 1 else 0
        spans = torch.tensor([[i * n, n, 128, i] for i in range(seqs)], dtype=torch.int32, device=dev)
        proj, state, mix = rnd(rows, 3 * W), torch.zeros(seqs, W, device=dev), rnd(rows, W)
        ws = torch.empty(K.gru_workspace_bytes(rows, seqs, W), dtype=torch.uint8, device=dev)
        report(f"minGRU {seqs}x{n}", "chunks" if n > 1 else "step", lambda: K.gru(proj, bias, state, spans, single, mix, ws), rows * W * 8 + 8 * seqs * W)
        proj, z, state = rnd(rows, 4 * heads * N), rnd(rows, heads * N), torch.zeros(seqs, heads, P, N, device=dev)
        q, k, v, gate = proj.split(heads * N, 1)
        b, w, y = torch.ones(heads * N, device=dev), torch.ones(heads * P, device=dev), torch.zeros(rows, heads * P, device=dev)
        lws = torch.empty(K.linear_attention_workspace_bytes(rows, seqs, heads, P, N), dtype=torch.uint8, device=dev)
        report(f"linear attention {seqs}x{n}", "chunks, norm and gate" if n > 1 else "step, norm and gate", lambda: K.linear_attention(
            q, k, v, gate, z, b, 1 / 16, state, spans, single, y, mix, w, 1e-5, lws), rows * heads * N * 2 * 6 + 2 * seqs * heads * P * N * 4)
        del lws
    nq, nkv, D, page = 32, 8, 128, 64
    ws = torch.zeros(256 << 20, dtype=torch.uint8, device=dev)
    sink, sbias = torch.zeros(nq, device=dev), torch.full((nq, ), -6.0, device=dev)
    cache = rnd(T // page + 1, 2, nkv, page, D)
    table = torch.randperm(T // page, device=dev).to(torch.int32)[None].contiguous()
    q, o, gate = rnd(T, nq * D), rnd(T, nq * D), rnd(T, nq * D)
    items = torch.tensor([[0, i, 128, i] for i in range(0, T, 128)], dtype=torch.int32, device=dev)
    cases = [("softmax (like)", 0, {}), ("sigmoid weights", 0, {"sigmoid_bias": sbias}), ("softmax (like)", 2048, {}),
             ("sink and gate", 2048, {"sink": sink, "gate": gate})]
    for tag, window, opts in cases:
        pairs = sum(min(i + 1, window or T) for i in range(T))
        report(f"attention prefill {T} window {window}", tag, lambda: K.paged_attention_prefill(
            q, o, cache, table, items, T // 128, nq, nkv, D, page, 0.09, window=window, **opts), flops=4.0 * pairs * nq * D)
    B = 64
    cache = rnd(B * T // page, 2, nkv, page, D)
    tables = torch.randperm(B * T // page, device=dev).to(torch.int32).view(B, T // page).contiguous()
    items = torch.tensor([[i, i, 1, T - 1] for i in range(B)], dtype=torch.int32, device=dev)
    qd, od, gd = rnd(B, nq * D), rnd(B, nq * D), rnd(B, nq * D)
    for tag, window, opts in cases:
        sp = pick_packed_splits(B, nkv, windowed_len(T, window))
        opts = dict(opts, gate=gd) if "gate" in opts else opts
        report(f"attention decode {B}x{T} window {window}", tag, lambda: K.paged_attention_prefill(
            qd, od, cache, tables, items, B, nq, nkv, D, page, 0.09, n_splits=sp, workspace=ws, packed=True, window=window, **opts),
               B * min(T, window or T) * 2 * nkv * D * 2)
    del cache, q, o, gate
    freq, qn, kn, share = torch.ones(64, device=dev), torch.ones(nq * D, device=dev), torch.ones(nkv * D, device=dev), torch.ones(1, device=dev)
    for rows in (T, 64):
        qkv, q, pages, first = rnd(rows, (nq + 2 * nkv) * D), rnd(rows, nq * D), rnd(rows // page + 1, 2, nkv, page, D), rnd(rows // page + 1, 2, nkv, page, D)
        pos = torch.arange(rows, dtype=torch.int32, device=dev)
        need = rows * 2 * (nq + 2 * nkv) * D * 2
        report(f"attention inputs {rows}", "norms, rotation, pages", lambda: K.attention_append(
            qkv, q, pages, pos, pos, nq, nkv, D, page, freq, qn, kn, nq * D, nkv * D, 1e-5), need)
        report(f"attention inputs {rows}", "rotation, pages, mixed values", lambda: K.attention_append(
            qkv, q, pages, pos, pos, nq, nkv, D, page, freq, first=first, share=share), need + rows * nkv * D * 2)
        report(f"attention inputs {rows}", "rope_kv_append (like)", lambda: K.rope_kv_append(qkv, q, pages, pos, pos, freq, nq, nkv, D, D, page), need)
        report(f"mix values {rows}", "mix_cached_values", lambda: K.mix_cached_values(pages, first, pos, share, nkv, D, page), rows * 3 * nkv * D * 2)
    E, top, ff = 16, 2, 5376
    i32 = lambda *s: torch.zeros(s, dtype=torch.int32, device=dev)  # noqa: E731
    for rows in (T, 64):
        scores, e, off, slots, counts, pad = torch.zeros(rows, top, device=dev), i32(rows, top), i32(rows, top), i32(rows, top), i32(E), i32(E + 1)
        R = K.moe_padded_rows(rows, E, top)
        x, xs, ys, out, wr, lg = rnd(rows, W), rnd(R, W), rnd(R, W), torch.zeros(rows, W, device=dev), rnd(E, W, scale=0.02), torch.zeros(rows, E, device=dev)
        hs, wu, wd = rnd(R, ff), rnd(E * ff, W, scale=0.02), rnd(E * W, ff, scale=0.02)

        def route(sigmoid):
            K.gemm_accum(x, wr, lg)
            K.moe_topk_gating(lg, top, False, scores, e, off, counts, clear=True, sigmoid=sigmoid)
            K.moe_scatter(x, xs, e, off, counts, pad, slots, top, scores if sigmoid else None)

        for tag, sigmoid in (("sigmoid scores, weighted rows", True), ("softmax scores (like)", False)):
            report(f"router + route + scatter {rows}", tag, lambda: route(sigmoid), rows * W * 2 * (2 + top))
        for tag, act in (("grouped GEMM, squared relu", 6), ("grouped GEMM, gelu (like)", 1)):
            report(f"experts up {rows}", tag, lambda: K.moe_gemm(xs, wu, pad, E, hs, act=act), 2 * (wu.numel() + rows * top * (W + ff)), 2.0 * rows * top * W * ff)
        report(f"experts down {rows}", "grouped GEMM", lambda: K.moe_gemm(hs, wd, pad, E, ys), 2 * (wd.numel() + rows * top * (W + ff)), 2.0 * rows * top * W * ff)
        report(f"combine {rows}", "moe_combine, plain sum", lambda: K.moe_combine(ys, slots, None, None, out), rows * W * (2 * top + 4))
        report(f"combine {rows}", "moe_combine, weighted (like)", lambda: K.moe_combine(ys, slots, scores, None, out), rows * W * (2 * top + 4))


def bench_relulix_kernels(p: Dict[str, float], iters: int, warmup: int) -> None:
    """The same for what Relulix adds: retention (32 heads of 128 x 128 and of 64 x 128), bounded scores with a one more, rotation with amplitudes,
    queries alone, experts weighed among the chosen, clamped gated experts."""
    from ..ops import kernels as K
    from ..ops.backend import pick_packed_splits, windowed_len
    dev, rnd, report = "cuda", _rnd, _reporter(p, iters, warmup)
    W, T, heads, P = 4096, PROMPT, 32, 128
    i32 = lambda *s: torch.zeros(s, dtype=torch.int32, device=dev)  # noqa: E731
    for N in (128, 64):
        decay = torch.linspace(-0.05, -1e-3, heads, device=dev)
        for rows, seqs in ((T, 1), (T, 4), (64, 64), (8, 8)):
            n = rows // seqs
            single = seqs if n == 1 else 0
            spans = torch.tensor([[i * n, n, 128, i] for i in range(seqs)], dtype=torch.int32, device=dev)
            proj, z, state, mix = rnd(rows, 2 * heads * (N + P)), rnd(rows, heads * N), torch.zeros(seqs, heads, P, N, device=dev), rnd(rows, heads * P)
            q, k, v, gate = proj.split([heads * N, heads * N, heads * P, heads * P], 1)
            b, w, y = torch.ones(heads * N, device=dev), torch.ones(heads * P, device=dev), torch.zeros(rows, heads * P, device=dev)
            moved = rows * heads * (2 * N + 3 * P) * 2 + 2 * seqs * heads * P * N * 4
            tag = "chunks, norm and gate" if n > 1 else "step, norm and gate"
            ws = torch.empty(K.retention_workspace_bytes(rows, seqs, heads, P, N), dtype=torch.uint8, device=dev)
            report(f"retention {seqs}x{n}, heads {N}x{P}", tag, lambda: K.retention(
                q, k, v, gate, decay, None, None, N**-0.5, P, state, spans, single, y, mix, w, 1e-5, ws), moved)
            ws = torch.empty(K.linear_attention_workspace_bytes(rows, seqs, heads, P, N), dtype=torch.uint8, device=dev)
            report(f"retention {seqs}x{n}, heads {N}x{P}", "linear attention, norm and gate (like)", lambda: K.linear_attention(
                q, k, v, gate, z, b, 1 / 16, state, spans, single, y, mix, w, 1e-5, ws), moved + rows * heads * N * 2)
            del ws
    nq, nkv, D, page, window = 32, 8, 128, 64, 2048
    ws = torch.zeros(256 << 20, dtype=torch.uint8, device=dev)
    sink = torch.zeros(nq, device=dev)
    cases = [("softmax (like)", {}), ("sink (like)", {"sink": sink}), ("bounded, one more", {"sink": sink, "softcap": 30.0})]
    cache, q, o = rnd(T // page + 1, 2, nkv, page, D), rnd(T, nq * D), rnd(T, nq * D)
    table = torch.randperm(T // page, device=dev).to(torch.int32)[None].contiguous()
    items = torch.tensor([[0, i, 128, i] for i in range(0, T, 128)], dtype=torch.int32, device=dev)
    pairs = sum(min(i + 1, window) for i in range(T))
    for tag, opts in cases:
        report(f"attention prefill {T} window {window}", tag, lambda: K.paged_attention_prefill(
            q, o, cache, table, items, T // 128, nq, nkv, D, page, 0.09, window=window, **opts), flops=4.0 * pairs * nq * D)
    B = 64
    for kvh in (nkv, nq):         # head-packed on the tensor cores, and one query head per key head
        cache = rnd(B * T // page // (kvh // nkv), 2, kvh, page, D)
        tables = torch.arange(cache.shape[0], device=dev).to(torch.int32).view(-1, T // page).contiguous()
        n = tables.shape[0]
        items = torch.tensor([[i, i, 1, T - 1] for i in range(n)], dtype=torch.int32, device=dev)
        qd, od = rnd(n, nq * D), rnd(n, nq * D)
        for tag, opts in cases:
            need = n * window * 2 * kvh * D * 2
            if kvh == nkv:
                sp = pick_packed_splits(n, kvh, windowed_len(T, window))
                report(f"attention decode {n}x{T} window {window}, {nq} / {kvh} heads", tag, lambda: K.paged_attention_prefill(
                    qd, od, cache, tables, items, n, nq, kvh, D, page, 0.09, n_splits=sp, workspace=ws, packed=True, window=window, **opts), need)
            else:
                report(f"attention decode {n}x{T} window {window}, {nq} / {kvh} heads", tag, lambda: K.paged_attention_splitkv(
                    qd, od, cache, tables, items, n, 1, nq, kvh, D, page, 1, 0.09, ws, window=window, **opts), need)
    del cache
    freq, amp = 1e4**(-torch.arange(64, device=dev) / 64), torch.full((64, ), 1.1, device=dev)
    x, w, b = rnd(T, W), rnd((nq + 2 * nkv) * D, W, scale=0.02), rnd((nq + 2 * nkv) * D)
    pages, pos = rnd(T // page, 2, nkv, page, D), torch.arange(T, dtype=torch.int32, device=dev)
    for tag, n, kw in (("biases, rotation with amplitudes, pages", nkv, {"bias_qkv": b, "amp": amp}), ("the same, queries alone", 0, {"bias_qkv": b, "amp": amp}),
                       ("rotation, pages (like)", nkv, {})):
        rows = (nq + 2 * n) * D
        report(f"q, k, v of {T}", tag, lambda: K.qkv_rope_proj(x, w[:rows], q, pages, pos, pos, freq, nq, n, D, page, **kw), flops=2.0 * T * rows * W)
    for rows in (64, ):
        qkv, n_all = rnd(rows, (nq + 2 * nkv) * D), (nq + 2 * nkv) * D
        for tag, n, kw in (("rotation with amplitudes, pages", nkv, {"amp": amp}), ("the same, queries alone", 0, {"amp": amp})):
            report(f"attention inputs {rows}", tag, lambda: K.attention_append(qkv, q, pages, pos, pos, nq, n, D, page, freq, **kw), rows * 4 * (nq + 2 * n) * D)
        report(f"attention inputs {rows}", "rope_kv_append (like)", lambda: K.rope_kv_append(qkv, q, pages, pos, pos, freq, nq, nkv, D, D, page), rows * 4 * n_all)
    del x, w, pages
    E, top, ff = 16, 2, 3584
    for rows in (T, 64):
        scores, e, off, slots, counts, pad = torch.zeros(rows, top, device=dev), i32(rows, top), i32(rows, top), i32(rows, top), i32(E), i32(E + 1)
        R = K.moe_padded_rows(rows, E, top)
        x, xs, wr, lg, bias = rnd(rows, W), rnd(R, W), rnd(E, W, scale=0.02), torch.zeros(rows, E, device=dev), torch.zeros(E, device=dev)
        hs, wu = rnd(R, ff), rnd(E * 2 * ff, W, scale=0.02)

        def route(**kw):
            K.gemm_accum(x, wr, lg)
            K.moe_topk_gating(lg, top, bool(kw), scores, e, off, counts, clear=True, **kw)
            K.moe_scatter(x, xs, e, off, counts, pad, slots, top)

        for tag, kw in (("logits with a bias choose", {"bias": bias, "biased": True}), ("softmax scores (like)", {})):
            report(f"router + route + scatter {rows}", tag, lambda: route(**kw), rows * W * 2 * (2 + top))
        for tag, act in (("grouped GEMM, clamped gate", 5), ("grouped GEMM, silu gate (like)", 3)):
            report(f"experts up {rows}", tag, lambda: K.moe_gemm(xs, wu, pad, E, hs, act=act, gated=True, limit=7.0),
                   2 * (wu.numel() + rows * top * (W + ff)), 2.0 * rows * top * W * 2 * ff)
        ys, d32, out = rnd(R, W), torch.zeros(rows, W, device=dev), torch.zeros(rows, W, device=dev)
        report(f"combine {rows}", "moe_combine onto the mixer's output", lambda: K.moe_combine(ys, slots, scores, d32, d32), rows * W * (2 * top + 8))
        report(f"combine {rows}", "moe_combine (like)", lambda: K.moe_combine(ys, slots, scores, None, out), rows * W * (2 * top + 4))


def main(steps: int = 5, warmup: int = 3, only: str = "") -> None:
    p = peaks()
    for group in GROUPS:
        for name in group if not only or any(n.startswith(only) for n in group) else ():
            print(json.dumps({"stack": name, "layers": 4, "prompt": PROMPT, "dtype": "bf16", "data": "random weights, synthetic tokens",
                              **bench_engine(name, steps, warmup)}), flush=True)
            torch.cuda.empty_cache()
    for prefix, kernels in (("", bench_kernels), ("lotelix", bench_lotelix_kernels), ("relulix", bench_relulix_kernels)):
        if not only or only == prefix:
            kernels(p, max(steps, 10), warmup)
            torch.cuda.empty_cache()


if __name__ == "__main__":
    main()
