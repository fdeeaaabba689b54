"""Nipolorn on the GPU: each kernel against its fp32 restatement, then whole models against the plain oracle."""
import pytest
import torch

from hcache_deepspeed_b200.ops import reference as ref

from . import nipolorn_helper as H
from . import nipolorn_oracle as oracle

pytestmark = [pytest.mark.gpu, pytest.mark.timeout(600)]
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16


def k():
    from hcache_deepspeed_b200.ops import kernels
    return kernels


def rnd(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed + sum(shape))) * scale).to(dtype).cuda()


# ---- attention: one planted key among empty ones ---------------------------------------------------------------------
def attend(kind, q, cache, table, pos0, d, n_q, n_kv, window, keep, page, out=None):
    """q [n, n_q, d] at positions pos0.. of one sequence whose keys are all in the cache already."""
    n = q.shape[0]
    qd = q.reshape(n, n_q * d).contiguous()
    out = torch.zeros_like(qd) if out is None else out
    tables = table[None].cuda()
    ws = torch.zeros(64 << 20, dtype=torch.uint8, device="cuda")
    item = lambda r0, m: torch.tensor([[0, r0, m, pos0 + r0]], dtype=torch.int32, device="cuda")  # noqa: E731
    if kind == "generic":
        k().paged_attention_generic(qd, out, cache, tables, torch.zeros(n, dtype=torch.int32, device="cuda"),
                                    torch.arange(pos0, pos0 + n, dtype=torch.int32, device="cuda"), n_q, n_kv, d, page, 1.0, window, keep)
    elif kind.startswith("split"):
        per = 8 // (n_q // n_kv)
        for r in range(0, n, per):
            m = min(per, n - r)
            k().paged_attention_splitkv(qd, out, cache, tables, item(r, m), 1, m * (n_q // n_kv), n_q, n_kv, d, page, int(kind[5:]), 1.0, ws,
                                        window=window, keep_first=keep)
    else:
        packed = kind.startswith("packed")
        step = 128 // (n_q // n_kv) if packed else 128
        for r in range(0, n, step):
            k().paged_attention_prefill(qd, out, cache, tables, item(r, min(step, n - r)), 1, n_q, n_kv, d, page, 1.0, n_splits=int(kind[6:]),
                                        workspace=ws, packed=packed, window=window, keep_first=keep)
    return out.view(n, n_q, d) if out.is_contiguous() else out.unflatten(1, (n_q, d))


KINDS = [("split1", 64, 2, 2), ("split3", 64, 4, 2), ("split2", 128, 3, 1), ("packed1", 128, 4, 1), ("packed3", 128, 8, 2),
         ("prefil1", 64, 4, 1), ("prefil2", 128, 6, 2), ("generic", 128, 4, 2), ("generic", 160, 2, 1)]


@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
@pytest.mark.parametrize("window,keep", [(48, 5), (1, 1), (128, 0), (200, 130), (300, 64), (64, 300)])
def test_planted_key_is_seen_exactly_inside_its_window(kind, d, n_q, n_kv, window, keep):
    """A key of huge score is planted at one position; its value shows in the output of exactly the queries that see it:
    positions at the window's and the kept range's edges, at page borders, far back and first of all."""
    dtype, page, n_keys = BF16, 64, 700
    n = 2 if kind.startswith("split") or kind.startswith("packed") else 150
    cache0, table = H.attention_case(d, n_q, n_kv, page, dtype, "cuda", n_keys)
    q = torch.zeros(n, n_q, d, dtype=dtype, device="cuda")
    q[..., 0] = 8.0
    for pos0 in (n_keys - n, 447, 130):
        pos0 = min(pos0, n_keys - n)
        last = pos0 + n - 1
        places = {0, keep - 1, keep, pos0 - window, pos0 - window + 1, last - window, last - window + 1, pos0, last, 63, 64, 128}
        for j in sorted(p for p in places if 0 <= p <= last):
            cache = cache0.clone()
            cache[int(table[j // page]), 0, :, j % page, 0] = 8.0
            cache[int(table[j // page]), 1, :, j % page] = 1.0
            got = attend(kind, q, cache.cuda(), table, pos0, d, n_q, n_kv, window, keep, page).float()
            i = torch.arange(pos0, pos0 + n, device="cuda")
            sees = (j <= i) & ((i - j < window) | (j < keep))
            assert ((got.amin((1, 2)) > 0.9) == sees).all() and ((got.amax((1, 2)) < 0.1) == ~sees).all(), (j, pos0)


@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
def test_attention_against_reference_and_strided_rows(kind, d, n_q, n_kv):
    page, n_keys, window, keep = 64, 500, 90, 70
    n = 2 if kind.startswith("split") or kind.startswith("packed") else 200
    cache, table = H.attention_case(d, n_q, n_kv, page, BF16, "cuda", n_keys)
    cache = torch.randn(cache.shape, generator=torch.Generator().manual_seed(1)).to(BF16).cuda()
    q = rnd(n, n_q, d, dtype=BF16, scale=0.2)
    items = torch.tensor([[0, 0, n, n_keys - n]], dtype=torch.int32)
    want = ref.paged_attention(q.cpu(), cache.cpu(), table[None], items, n_q, n_kv, 1.0, window=window, keep_first=keep).float()
    wide = torch.full((n, n_q * d + 24), 7.0, dtype=BF16, device="cuda")
    got = attend(kind, q, cache, table, n_keys - n, d, n_q, n_kv, window, keep, page, out=wide[:, :n_q * d])
    torch.testing.assert_close(got.float().cpu(), want, rtol=3e-2, atol=3e-2)
    assert (wide[:, n_q * d:] == 7.0).all()


def test_split_scratch_serves_changing_batch_sizes():
    """Arrival counters of a large launch must not land on partial sums that a smaller one left in the same scratch."""
    d, n_kv, page, keys = 64, 16, 64, 640
    g = torch.Generator().manual_seed(0)
    cache = torch.randn(16, 2, n_kv, page, d, generator=g).to(BF16).cuda()
    ws = torch.zeros(64 << 20, dtype=torch.uint8, device="cuda")
    for n in (2, 24, 3, 40, 24):
        q = rnd(n, n_kv * d, seed=n, dtype=BF16, scale=0.2)
        tables = torch.stack([torch.randperm(16, generator=g)[:10] for _ in range(n)]).to(torch.int32)
        items = torch.tensor([[i, i, 1, keys - 1] for i in range(n)], dtype=torch.int32)
        out = torch.zeros_like(q)
        k().paged_attention_splitkv(q, out, cache, tables.cuda(), items.cuda(), n, 1, n_kv, n_kv, d, page, 3, 1.0, ws)
        want = ref.paged_attention(q.cpu().view(n, n_kv, d), cache.cpu(), tables, items, n_kv, n_kv, 1.0)
        torch.testing.assert_close(out.cpu().view(n, n_kv, d).float(), want.float(), rtol=3e-2, atol=3e-2)


# ---- state-space mixer -------------------------------------------------------------------------------------------------
SSM = [(6, 20, 12, 3, 3), (4, 64, 128, 1, 4), (8, 32, 64, 2, 4), (3, 17, 9, 3, 1), (2, 128, 128, 2, 4), (2, 48, 32, 1, 4), (2, 5, 300, 1, 6)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("heads,P,N,groups,taps", SSM)
@pytest.mark.parametrize("method", [0, 1])
def test_state_space_against_reference(heads, P, N, groups, taps, dtype, method):
    """Three sequences with their own slots over several launches: long and short portions, single tokens, a slot used again."""
    inner, C = heads * P, heads * P + 2 * groups * N
    slots = 4
    mk = lambda *s, **kw: rnd(*s, **kw)  # noqa: E731
    cw, cb, db = mk(taps, C, scale=0.6), mk(C, seed=1, scale=0.2), mk(heads, seed=2) - 1
    a, dsk = -torch.exp(mk(heads, seed=3, scale=0.7)), mk(heads, seed=4)
    state, ring = mk(slots, heads, P, N, seed=5), mk(slots, taps, C, seed=6)
    st_ref, ring_ref = state.cpu().clone(), ring.cpu().clone()
    tol = dict(rtol=2e-4, atol=2e-4) if dtype == F32 else dict(rtol=1e-2, atol=1e-2)
    seen = {}
    for step, plan in enumerate([[(0, 150), (2, 2)], [(0, 1), (2, 1), (3, 1)], [(3, 40), (0, 129), (2, 1)], [(1, 257)], [(1, 1)], [(0, 3), (1, 128)]]):
        if step == 5:
            seen[0] = 0      # slot 0 handed to another sequence
        T = sum(n for _, n in plan)
        ld = 8 * ((2 * inner + 2 * groups * N + heads + 8) // 8) + 8
        proj = mk(T, ld, seed=10 + step, dtype=dtype)
        spans, row = [], 0
        for s, n in plan:
            spans.append([row, n, seen.get(s, 0), s])
            row += n
            seen[s] = seen.get(s, 0) + n
        sp = torch.tensor(spans, dtype=torch.int32)
        u = torch.zeros(T, 8 * ((C + 7) // 8), dtype=dtype, device="cuda")
        dt, y = torch.zeros(T, heads, device="cuda"), torch.zeros(T, inner, device="cuda")
        k().state_space(proj, cw, cb, db, a, dsk, state, ring, sp.cuda(), sum(n == 1 for _, n in plan), groups, u, dt, y, method=method)
        for r0, n, at, s in spans:
            p = proj[r0:r0 + n].cpu()
            if at == 0:
                st_ref[s].zero_()
            xbc = ref.short_conv(p[:, inner:inner + C], ring_ref[s], cw.cpu(), cb.cpu(), at).to(dtype).float()
            dts = torch.nn.functional.softplus(p[:, inner + C:inner + C + heads].float() + db.cpu())
            want = ref.selective_scan(xbc[:, :inner].reshape(n, heads, P), xbc[:, inner:inner + groups * N].reshape(n, groups, N),
                                      xbc[:, inner + groups * N:].reshape(n, groups, N), dts, a.cpu(), dsk.cpu(), st_ref[s])
            scale = float(want.abs().max())
            torch.testing.assert_close(y[r0:r0 + n].cpu().view(n, heads, P) / scale, want / scale, **tol)
            torch.testing.assert_close(state[s].cpu() / st_ref[s].abs().max(), st_ref[s] / st_ref[s].abs().max(), **tol)
            filled = [q % taps for q in range(max(0, at + n - taps), at + n)]
            torch.testing.assert_close(ring[s].cpu()[filled], ring_ref[s][filled])


@pytest.mark.parametrize("heads,P,N,groups", [(4, 64, 128, 2), (3, 48, 32, 1), (2, 128, 64, 1), (2, 8, 16, 2), (6, 40, 96, 3)])
def test_chunked_scan_against_token_scan(heads, P, N, groups):
    """The tensor-core scan keeps 16 bits of every fp32 operand: far closer to the fp32 scan than 16-bit rounding would be.
    Lengths around the chunk borders, with and without carried state, fast and slow decays."""
    inner, C, taps = heads * P, heads * P + 2 * groups * N, 4
    cw, cb, db = rnd(taps, C, scale=0.6), rnd(C, seed=1, scale=0.2), rnd(heads, seed=2) - 1
    a, dsk = -torch.exp(rnd(heads, seed=3, scale=2.0)), rnd(heads, seed=4)
    for lens in ([2], [128, 127], [129, 3, 300], [64, 256, 2]):
        T = sum(lens)
        proj = rnd(T, 8 * ((2 * inner + 2 * groups * N + heads + 7) // 8), seed=T, dtype=BF16)
        spans, row = [], 0
        for i, n in enumerate(lens):
            spans.append([row, n, 5 if i % 2 else 0, len(lens) - 1 - i])
            row += n
        outs = []
        for method in (1, 2):
            state, ring = rnd(len(lens), heads, P, N, seed=5), rnd(len(lens), taps, C, seed=6)
            u = torch.zeros(T, 8 * ((C + 7) // 8), dtype=BF16, device="cuda")
            dt, y = torch.zeros(T, heads, device="cuda"), torch.zeros(T, inner, device="cuda")
            k().state_space(proj, cw, cb, db, a, dsk, state, ring, torch.tensor(spans, dtype=torch.int32, device="cuda"), 0, groups, u, dt, y,
                            method=method)
            outs.append((y, state, ring))
        for got, want in zip(outs[1], outs[0]):
            torch.testing.assert_close(got / want.abs().max(), want / want.abs().max(), rtol=0, atol=5e-5)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cols,groups", [(120, 5), (256, 1), (4096, 8), (51, 3)])
def test_gated_norm(cols, groups, dtype):
    y, z, w = rnd(33, cols), rnd(33, cols + 8, dtype=dtype), rnd(cols)
    out = torch.full((33, cols + 8), 3.0, dtype=dtype, device="cuda")
    k().gated_norm(y, z[:, :cols], w, out[:, :cols], groups, 1e-5, 0.7)
    want = ref.gated_norm(y, z[:, :cols], w, groups, 1e-5, 0.7)
    tol = 1e-5 if dtype == F32 else 1e-2
    torch.testing.assert_close(out[:, :cols].float(), want, rtol=tol, atol=tol)
    assert (out[:, cols:] == 3.0).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,pad", [(88, 88), (75, 80), (4096, 4096), (9001, 9008)])
@pytest.mark.parametrize("delta", [None, "f32", "same"])
def test_norm_residual(H, pad, delta, dtype):
    z = lambda t: torch.nn.functional.pad(t, (0, pad - H))  # noqa: E731
    x, g, p = z(rnd(7, H)), z(rnd(H, seed=1)), z(rnd(H, seed=2))
    d = None if delta is None else z(rnd(7, H, seed=3, scale=0.1)).to(F32 if delta == "f32" else dtype)
    wx, wo = ref.norm_residual(x, g, d, 1.7, p, H, 1e-5)
    out = torch.empty(7, pad, dtype=dtype, device="cuda")
    for store in (False, True):
        x1, d1 = x.clone(), None if d is None else d.clone()
        k().norm_residual(x1, g, out, delta=d1, factor=1.7, post=p, cols=H, eps=1e-5, store_resid=store)
        tol = 2e-5 if dtype == F32 else 1e-2
        torch.testing.assert_close(out.float(), wo, rtol=tol, atol=tol)
        torch.testing.assert_close(x1, wx if store and d is not None else x, rtol=2e-5, atol=2e-5)
        if delta == "f32" or (d is not None and dtype == F32):
            assert not d1.any()


# ---- matrix products -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,ff,K", [(1, 72, 88), (9, 8192, 256), (40, 96, 128), (300, 200, 192), (2300, 2048, 128)])
def test_clamped_gate_epilogue(M, ff, K, dtype):
    from hcache_deepspeed_b200.models.weights import interleave_gate_up
    x = rnd(M, K, dtype=dtype)
    w = interleave_gate_up(rnd(ff, K, dtype=dtype, scale=0.2), rnd(ff, K, seed=1, dtype=dtype, scale=0.2))
    ws = torch.zeros(k().gemm_splitk_workspace_bytes(128, 2 * ff), dtype=torch.uint8, device="cuda")
    for limit in (0.8, 3.0):
        got = k().gemm(x, w, act=5, gated=True, limit=limit, workspace=ws if M <= 128 else None)
        want = ref.gemm(x, w, act=5, gated=True, limit=limit, out_dtype=F32)
        tol = 1e-4 if dtype == F32 else 3e-2
        torch.testing.assert_close(got.float(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("E,top,shared", [(5, 2, True), (12, 1, True), (9, 3, False)])
def test_table_moe(E, top, shared, dtype):
    from hcache_deepspeed_b200.models.arch import FeedForwardSpec
    from hcache_deepspeed_b200.models.weights import ExpertWeights, LayerWeights
    from hcache_deepspeed_b200.ops.backend import CpuOps, CudaOps
    W, ff, V, T = 64, 32, 50, 270
    ex = [ExpertWeights(rnd(2 * ff, W, seed=e, dtype=dtype, scale=0.2), rnd(W, ff, seed=e, dtype=dtype, scale=0.2)) for e in range(E)]
    g = torch.Generator().manual_seed(0)
    lw = LayerWeights(experts=ex, moe_table=torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(V)]).int().cuda())
    lw.stack_experts()
    f = FeedForwardSpec(ff=ff, experts=E, top=top)
    rows = k().moe_padded_rows(T, E, top)
    i32 = lambda *s: torch.zeros(s, dtype=torch.int32, device="cuda")  # noqa: E731
    bufs = dict(scores=torch.zeros(T, top, device="cuda"), expert_ids=i32(T, top), offsets=i32(T, top), mapped_slots=i32(T, top), counts=i32(E),
                pad_off=i32(E + 1), xs=torch.zeros(rows, W, dtype=dtype, device="cuda"), hs=torch.zeros(rows, ff, dtype=dtype, device="cuda"),
                ys=torch.zeros(rows, W, dtype=dtype, device="cuda"))
    for n in (T, 3, 140):
        x, ids = rnd(n, W, seed=n, dtype=dtype), torch.randint(0, V, (n, ), generator=g).int()
        base = rnd(n, W, seed=n + 1, dtype=dtype) if shared else None
        out = torch.full((n, W), 5.0, device="cuda")
        CudaOps().table_moe(x, ids.cuda(), lw, f, 3, base, out, bufs)
        cl = LayerWeights(experts=[ExpertWeights(e.w_up.cpu(), e.w_down.cpu()) for e in lw.experts], moe_table=lw.moe_table.cpu())
        want = CpuOps().table_moe(x.cpu(), ids, cl, f, 3, None if base is None else base.cpu(), torch.zeros(n, W), None)
        tol = 1e-4 if dtype == F32 else 3e-2
        torch.testing.assert_close(out.cpu(), want, rtol=tol, atol=tol)


# ---- whole models ----------------------------------------------------------------------------------------------------------
MODELS = {"mixed": H.MIXED, "odd": H.ODD, "wide": H.WIDE, "tiled": H.TILED}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_and_portions(name, dtype):
    H.check_whole_and_portions(MODELS[name], dtype, "cuda", n=400 if name == "tiled" else 190)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "tiled"])
def test_mixed_batches_reuse_pages_and_slots(name, dtype):
    H.check_mixed_batches(MODELS[name], dtype, "cuda")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decode(dtype):
    H.check_long_decode(H.MIXED, dtype, "cuda")


@pytest.mark.parametrize("name,dtype", [("mixed", F32), ("mixed", BF16), ("tiled", BF16)])
def test_restore_from_hidden_states(name, dtype):
    H.check_restore(MODELS[name], dtype, "cuda")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_greedy_generation(dtype, tmp_path):
    H.check_greedy(H.MIXED, dtype, True, tmp_path / "m")


def test_decode_runs_as_a_graph_and_fp16_is_served():
    cfg = H.TILED
    w, t = H.weights(cfg, seed=2), H.tokens(cfg, 60)
    eng = H.engine(cfg, w, F16, "cuda")
    assert H.error(H.run(eng, 0, t, [20]), H.expected(cfg, w, t)) < H.TOLERANCE[F16]
    assert eng.graph_replays > 20
