"""Lotelix on the GPU: each kernel against its fp32 restatement, then whole models against the plain oracle."""
import pytest
import torch

from hcache_deepspeed_b200.ops import reference as ref

from . import lotelix_helper as H

pytestmark = [pytest.mark.gpu, pytest.mark.timeout(600)]
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16


def k():
    from hcache_deepspeed_b200.ops import kernels
    return kernels


def rnd(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed + sum(shape))) * scale).to(dtype).cuda()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def close(got, want, dtype, fine=1e-4, coarse=2e-2):
    tol = fine if dtype == F32 else coarse
    torch.testing.assert_close(got.float().cpu(), want.float().cpu(), rtol=tol, atol=tol)


# ---- attention with sinks, sigmoid weights and gates --------------------------------------------------------------------
def attend(kind, q, cache, table, pos0, n_kv, window=0, out=None, **opts):
    """q [n, n_q, d] at positions pos0.. of one sequence whose keys are all in the cache already."""
    n, n_q, d = q.shape
    page = cache.shape[3]
    qd = q.reshape(n, n_q * d).contiguous()
    out = torch.zeros_like(qd) if out is None else out
    tables = table[None].cuda()
    ws = torch.zeros(64 << 20, dtype=torch.uint8, device="cuda")
    items = lambda per: i32([[0, r, min(per, n - r), pos0 + r] for r in range(0, n, per)])  # noqa: E731
    if kind == "generic":
        k().paged_attention_generic(qd, out, cache, tables, i32([0] * n), torch.arange(pos0, pos0 + n, dtype=torch.int32, device="cuda"), n_q, n_kv, d, page,
                                    1.0, window, **opts)
    elif kind.startswith("split"):
        per = 8 // (n_q // n_kv)
        it = items(per)
        k().paged_attention_splitkv(qd, out, cache, tables, it, it.shape[0], per * (n_q // n_kv), n_q, n_kv, d, page, int(kind[5:]), 1.0, ws, window=window,
                                    **opts)
    else:
        packed = kind.startswith("packed")
        it = items(128 // (n_q // n_kv) if packed else 128)
        k().paged_attention_prefill(qd, out, cache, tables, it, it.shape[0], n_q, n_kv, d, page, 1.0, n_splits=int(kind[6:]), workspace=ws, packed=packed,
                                    window=window, **opts)
    return out.view(n, n_q, d) if out.is_contiguous() else out.unflatten(1, (n_q, d))


KINDS = [("split1", 64, 2, 2), ("split3", 64, 4, 2), ("split2", 128, 3, 1), ("split1", 64, 8, 1), ("packed1", 128, 4, 1), ("packed3", 128, 8, 2),
         ("prefil1", 64, 4, 1), ("prefil2", 128, 6, 2), ("prefil3", 64, 3, 3), ("generic", 128, 4, 2), ("generic", 160, 2, 1)]


def options(mode, n, n_q, d, dtype):
    opts = {"sink": rnd(n_q, seed=3, scale=2.0)} if "sink" in mode else {}
    if "sigmoid" in mode:
        opts["sigmoid_bias"] = rnd(n_q, seed=4) - 3
    if "gate" in mode:
        opts["gate"] = rnd(n, n_q * d + 16, seed=5, dtype=dtype)[:, 8:8 + n_q * d]
    return opts


@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
@pytest.mark.parametrize("mode", ["sink", "sink+gate", "sigmoid", "sigmoid+gate", "gate"])
@pytest.mark.parametrize("window", [0, 90])
def test_attention_against_reference(kind, d, n_q, n_kv, mode, window):
    page, n_keys = 64, 500
    n = 150 if kind.startswith("prefil") else 5
    for dtype in ([BF16, F16] if kind != "generic" else [BF16, F32]):
        cache, table = H.attention_case(d, n_q, n_kv, page, dtype, "cuda", n_keys)
        cache = torch.randn(cache.shape, generator=torch.Generator().manual_seed(1)).to(dtype).cuda()
        q = rnd(n, n_q, d, dtype=dtype, scale=0.2)
        opts = options(mode, n, n_q, d, dtype)
        items = torch.tensor([[0, 0, n, n_keys - n]], dtype=torch.int32)
        cpu = {a: b.float().cpu() for a, b in opts.items()}
        want = ref.paged_attention(q.cpu().float(), cache.cpu(), table[None], items, n_q, n_kv, 1.0, window=window, **cpu)
        wide = torch.full((n, n_q * d + 24), 7.0, dtype=dtype, device="cuda")
        got = attend(kind, q, cache, table, n_keys - n, n_kv, window, wide[:, :n_q * d], **opts)
        assert (got.float().cpu() - want).abs().max() < (1e-4 if dtype == F32 else 1e-2) * want.abs().max()
        assert (wide[:, n_q * d:] == 7.0).all()


@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
@pytest.mark.parametrize("mode", ["sink", "sigmoid"])
@pytest.mark.parametrize("window", [1, 48, 128, 300, 0])
def test_planted_key_is_seen_exactly_inside_its_window(kind, d, n_q, n_kv, mode, window):
    """A key of huge score is planted at one position; its value shows in the output of exactly the queries that see it: positions at
    the window's edges, at page borders, far back and first of all."""
    page, n_keys = 64, 700
    n = 150 if kind.startswith("prefil") else 2
    cache0, table = H.attention_case(d, n_q, n_kv, page, BF16, "cuda", n_keys)
    q = torch.zeros(n, n_q, d, dtype=BF16, device="cuda")
    q[..., 0] = 8.0
    opts = {"sink": torch.full((n_q, ), 9.0, device="cuda")} if mode == "sink" else {"sigmoid_bias": torch.full((n_q, ), -20.0, device="cuda")}
    for pos0 in (n_keys - n, 447, 130):
        pos0 = min(pos0, n_keys - n)
        last = pos0 + n - 1
        places = {0, 1, pos0 - window, pos0 - window + 1, last - window, last - window + 1, pos0, last, 63, 64, 128}
        for j in sorted(p for p in places if 0 <= p <= last):
            cache = cache0.clone()
            cache[int(table[j // page]), 0, :, j % page, 0] = 8.0
            cache[int(table[j // page]), 1, :, j % page] = 1.0
            got = attend(kind, q, cache.cuda(), table, pos0, n_kv, window, **opts).float()
            i = torch.arange(pos0, pos0 + n, device="cuda")
            sees = (j <= i) & ((i - j < window) if window else True)
            assert ((got.amin((1, 2)) > 0.9) == sees).all() and ((got.amax((1, 2)) < 0.1) == ~sees).all(), (j, pos0)


@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
def test_sinks_and_sums_over_equal_keys(kind, d, n_q, n_kv):
    """n equal keys leave n / (n + exp(sink)) of their value; sigmoid weights add up to n times one of them. The first tokens of a
    sequence, where a sink takes the most."""
    page = 64
    cache, table = H.attention_case(d, n_q, n_kv, page, BF16, "cuda", 700)
    cache[:, 1] = 1.0
    sink = torch.linspace(-3, 4, n_q, device="cuda")
    for pos0, n in ((0, 5), (0, 1), (600, 2)):
        q, count = torch.zeros(n, n_q, d, dtype=BF16, device="cuda"), torch.arange(pos0 + 1, pos0 + n + 1, device="cuda").float()[:, None]
        got = attend(kind, q, cache.cuda(), table, pos0, n_kv, sink=sink)
        torch.testing.assert_close(got.float().mean(-1), count / (count + sink.exp()), rtol=1e-2, atol=1e-3)
        got = attend(kind, q, cache.cuda(), table, pos0, n_kv, sigmoid_bias=sink)
        torch.testing.assert_close(got.float().mean(-1), count * torch.sigmoid(sink), rtol=1e-2, atol=1e-3)


def test_options_last_for_one_launch():
    d, n_kv, page = 64, 2, 64
    cache, table = H.attention_case(d, n_kv, n_kv, page, BF16, "cuda", 100)
    cache[:, 1] = 1.0
    q = torch.zeros(2, n_kv, d, dtype=BF16, device="cuda")
    for kind in ("split1", "prefil1", "generic"):
        assert attend(kind, q, cache.cuda(), table, 50, n_kv, sink=torch.full((n_kv, ), 9.0, device="cuda")).max() < 0.1
        assert (attend(kind, q, cache.cuda(), table, 50, n_kv).float() - 1).abs().max() < 1e-2


# ---- what enters attention -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("n_q,n_kv,D,D1", [(6, 2, 64, 64), (8, 8, 128, 64), (3, 1, 136, 136), (4, 2, 64, 128)])
@pytest.mark.parametrize("normed", [False, True])
@pytest.mark.parametrize("mixed", [False, True])
def test_attention_append(n_q, n_kv, D, D1, normed, mixed, dtype):
    T, page, blocks = 37, 64, 4
    proj = rnd(T, (n_q + 2 * n_kv) * D + 16, dtype=dtype)[:, :(n_q + 2 * n_kv) * D]
    pos = torch.randint(0, 3000, (T, ), generator=torch.Generator().manual_seed(0)).int()
    slot = torch.randperm(blocks * page, generator=torch.Generator().manual_seed(1))[:T].int()
    slot[5] = -1
    freq = torch.cat([500.0**(-torch.arange(D // 4) / (D // 4)), torch.zeros(D // 2 - D // 4)]).float()
    qn, kn = (1 + rnd(n_q * D, scale=0.2), 1 + rnd(n_kv * D, scale=0.2)) if normed else (None, None)
    first, share = (rnd(blocks, 2, n_kv, page, D1, dtype=dtype), torch.tensor([0.7], device="cuda")) if mixed else (None, None)
    cache, q = torch.full((blocks, 2, n_kv, page, D), 3.0, dtype=dtype, device="cuda"), torch.zeros(T, n_q * D, dtype=dtype, device="cuda")
    cols = (n_q * D - 11, n_kv * D - 3)
    k().attention_append(proj, q, cache, pos.cuda(), slot.cuda(), n_q, n_kv, D, page, freq.cuda(), qn, kn, *cols, 1e-3, first, share)
    cpu = lambda t: None if t is None else t.float().cpu()  # noqa: E731
    want = torch.full((blocks, 2, n_kv, page, D), 3.0)
    want_q = ref.attention_append(cpu(proj), want, pos, slot, n_q, n_kv, freq, cpu(qn), cpu(kn), *cols, 1e-3, cpu(first), cpu(share))
    close(q, want_q, dtype, fine=1e-3)
    close(cache, want, dtype, fine=1e-3)
    again = torch.full((blocks, 2, n_kv, page, D), 3.0, dtype=dtype, device="cuda")      # keys and values alone
    part = proj[:, n_q * D:]
    k().attention_append(part, part, again, pos.cuda(), slot.cuda(), 0, n_kv, D, page, freq.cuda(), None, kn, *cols, 1e-3, first, share)
    close(again, cache, dtype, fine=1e-5)
    if mixed:
        plain = torch.full((blocks, 2, n_kv, page, D), 3.0, dtype=dtype, device="cuda")
        k().attention_append(proj, q, plain, pos.cuda(), slot.cuda(), n_q, n_kv, D, page, freq.cuda(), qn, kn, *cols, 1e-3)
        k().mix_cached_values(plain, first, slot.cuda(), share, n_kv, D, page)
        close(plain, want, dtype, fine=1e-3)


# ---- recurrences -----------------------------------------------------------------------------------------------------------
#: launches over four slots: long and short portions (chunk borders among them), single tokens, a slot used again by another sequence
PLANS = [[(0, 150), (2, 2)], [(0, 1), (2, 1), (3, 1)], [(3, 40), (0, 64), (2, 1)], [(1, 257)], [(1, 1)], [(0, 3), (1, 128), (2, 65), (3, 63)]]


def batches():
    seen = {}
    for step, plan in enumerate(PLANS):
        if step == 5:
            seen[0] = 0
        spans, row = [], 0
        for s, n in plan:
            spans.append([row, n, seen.get(s, 0), s])
            row += n
            seen[s] = seen.get(s, 0) + n
        yield step, row, spans, sum(n == 1 for _, n in plan)


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("C", [8, 40, 520, 1032])
def test_gru_against_reference(C, dtype):
    state = rnd(4, 1, C, 1, seed=5)
    st, bias = state.cpu().clone(), rnd(2 * C, seed=6)
    ws = torch.empty(k().gru_workspace_bytes(300, 4, C), dtype=torch.uint8, device="cuda")
    for step, T, spans, single in batches():
        proj = rnd(T, 3 * C, seed=step, dtype=dtype, scale=2.0)
        proj[0, C:2 * C] = -bias[C:].to(dtype)
        out = torch.full((T, C + 8), 4.0, dtype=dtype, device="cuda")
        other = state.clone()
        k().gru(proj, bias, state, i32(spans), single, out[:, :C], ws)
        k().gru(proj, bias, other, i32(spans), single, None, ws)
        assert torch.equal(state, other) and (out[:, C:] == 4.0).all()
        for r0, n, at, s in spans:
            p, S = proj[r0:r0 + n].cpu().float(), st[s].view(-1)
            if at == 0:
                S.zero_()
            y = ref.gru_scan(p[:, :C] + bias[:C].cpu(), p[:, C:2 * C] + bias[C:].cpu(), S)
            close(out[r0:r0 + n, :C], y * torch.nn.functional.silu(p[:, 2 * C:]), dtype)
            torch.testing.assert_close(state[s].cpu(), st[s], rtol=1e-4, atol=1e-4)


def linear_case(T, heads, N, P, dtype, seed, decay=1.0):
    nk, nv = -(-heads * N // 8) * 8, -(-heads * P // 8) * 8
    proj = rnd(T, 2 * nk + 2 * nv + 16, seed=seed, dtype=dtype)
    z = rnd(T, nk, seed=seed + 1, dtype=dtype, scale=2 * decay)
    return (proj[:, :nk], proj[:, nk:2 * nk], proj[:, 2 * nk:2 * nk + nv], proj[:, 2 * nk + nv:2 * nk + 2 * nv], z)


LINEAR = [(2, 10, 18), (3, 24, 40), (4, 64, 128), (2, 128, 48), (3, 7, 9), (1, 272, 150), (2, 256, 64), (2, 16, 16), (2, 96, 144), (1, 530, 16), (2, 48, 256)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("heads,N,P", LINEAR)
@pytest.mark.parametrize("method", [0, 1])
def test_linear_attention_against_reference(heads, N, P, method, dtype):
    nk, nv, tau, eps = heads * N, heads * P, 3.0, 1e-4
    state = rnd(4, heads, P, N, seed=5)
    st, bias, w = state.cpu().clone(), rnd(nk, seed=6) + 1, 1 + rnd(P, seed=7, scale=0.2).repeat(heads)
    n_ws = k().linear_attention_workspace_bytes(300, 4, heads, P, N)
    ws = torch.empty(n_ws, dtype=torch.uint8, device="cuda") if n_ws else None
    for step, T, spans, single in batches():
        q, kk, v, g, z = linear_case(T, heads, N, P, dtype, 10 * step)
        y = torch.zeros(T, -(-nv // 8) * 8, device="cuda")
        out = torch.full((T, -(-nv // 8) * 8 + 8), 4.0, dtype=dtype, device="cuda")
        other = state.clone()
        k().linear_attention(q, kk, v, g, z, bias, 1 / tau, state, i32(spans), single, y, out[:, :nv], w, eps, ws, method)
        k().linear_attention(q, kk, v, g, z, bias, 1 / tau, other, i32(spans), single, y, None, w, eps, ws, method)
        assert torch.equal(state, other) and (out[:, nv:] == 4.0).all()
        for r0, n, at, s in spans:
            if at == 0:
                st[s].zero_()
            f = lambda t, d: t[r0:r0 + n, :heads * d].cpu().float().reshape(n, heads, d)  # noqa: E731
            decay = ref.linear_decay(f(z, N) + bias.cpu().view(heads, N), tau)
            o = ref.linear_scan(f(q, N), f(kk, N), f(v, P), decay, st[s]).reshape(n, nv)
            want = ref.gated_norm(o, g[r0:r0 + n, :nv].cpu(), w.cpu(), heads, eps, gate_after=True)
            close(out[r0:r0 + n, :nv], want, dtype, fine=5e-4, coarse=3e-2)
            top = st[s].abs().max()
            torch.testing.assert_close(state[s].cpu() / top, st[s] / top, rtol=0, atol=1e-4)


@pytest.mark.parametrize("heads,N,P", [(4, 128, 128), (3, 64, 48), (2, 256, 144), (5, 16, 32)])
@pytest.mark.parametrize("decay,tau", [(0.5, 16.0), (3.0, 1.0), (20.0, 1.0), (200.0, 0.25)])
@pytest.mark.parametrize("cells", [0, 3])
def test_chunked_linear_attention_against_token_scan(heads, N, P, decay, tau, cells):
    """The tensor-core form keeps 16 bits of every fp32 operand: far closer to the fp32 scan than 16-bit rounding would be. Lengths around
    the chunk borders, slow decays and ones that wipe a channel within a token, scratch for a few chunks only."""
    for lens in ([2], [64, 63], [65, 3, 300], [200, 1, 129, 2]):
        T, nv = sum(lens), heads * P
        q, kk, v, g, z = linear_case(T, heads, N, P, BF16, T, decay)
        spans, row = [], 0
        for i, n in enumerate(lens):
            spans.append([row, n, 5 if i % 2 else 0, len(lens) - 1 - i])
            row += n
        single = sum(n == 1 for n in lens)
        n_ws = k().linear_attention_workspace_bytes(T, len(lens), heads, P, N) if not cells else cells * heads * N * (P + 64) * 4
        ws = torch.empty(n_ws, dtype=torch.uint8, device="cuda")
        res = []
        for method in (1, 2):
            state = rnd(len(lens), heads, P, N, seed=5, scale=0.3)
            y, out = torch.zeros(T, nv, device="cuda"), torch.zeros(T, nv, dtype=BF16, device="cuda")
            k().linear_attention(q, kk, v, g, z, torch.zeros(heads * N, device="cuda"), 1 / tau, state, i32(spans), single, y, out,
                                 torch.ones(nv, device="cuda"), 1e-5, ws, method)
            res.append((out.float(), state))
        assert torch.isfinite(res[1][0]).all()
        atol = 5e-4 if decay > 100 else 1e-4            # (running sums of thousands: their last fp32 bit is a share of a decay)
        torch.testing.assert_close(res[1][1] / res[0][1].abs().max(), res[0][1] / res[0][1].abs().max(), rtol=0, atol=atol)
        torch.testing.assert_close(res[1][0], res[0][0], rtol=1e-2, atol=2e-3)


# ---- norms, router, experts ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cols,groups", [(75, 5), (75, 75), (256, 2), (4096, 1), (4096, 8), (2048, 4), (12288, 3)])
@pytest.mark.parametrize("delta", [None, "f32", "same"])
@pytest.mark.parametrize("two", [False, True])
def test_grouped_norm_of_the_stream(cols, groups, delta, two, dtype):
    pad = -(-cols // 8) * 8
    z = lambda t: torch.nn.functional.pad(t, (0, pad - cols))  # noqa: E731
    x, g = z(rnd(7, cols)), z(rnd(cols, seed=1))
    kind = F32 if delta == "f32" else dtype
    d = None if delta is None else z(rnd(7, cols, seed=3)).to(kind)
    d2, p, p2 = (z(rnd(7, cols, seed=4)).to(kind), z(rnd(cols, seed=5)), z(rnd(cols, seed=6))) if two and d is not None else (None, None, None)
    wx, wo = ref.norm_residual(x, g, d, 1.3, p, cols, 1e-3, groups, d2, p2)
    out = torch.empty(7, pad, dtype=dtype, device="cuda")
    k().norm_residual(x, g, out, delta=d, factor=1.3, post=p, cols=cols, eps=1e-3, groups=groups, delta2=d2, post2=p2)
    close(out, wo, dtype, fine=5e-5)
    torch.testing.assert_close(x, wx, rtol=2e-5, atol=2e-5)
    for t in (d, d2):
        assert t is None or t.dtype != F32 or not t.any()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_embedding_factor(dtype):
    w, ids = rnd(50, 80, dtype=dtype), i32([3, 49, -1, 0, 3])
    got = k().embed_f32(ids, w, torch.empty(5, 80, device="cuda"), scale=2.5)
    torch.testing.assert_close(got, w.float()[[3, 49, 0, 0, 3]] * torch.tensor([2.5, 2.5, 0, 2.5, 2.5], device="cuda")[:, None])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,N,K", [(5, 48, 40), (300, 72, 64), (130, 520, 192)])
def test_squared_relu_and_bias(M, N, K, dtype):
    x, w, b = rnd(M, K, dtype=dtype, scale=0.3), rnd(N, K, dtype=dtype, scale=0.3), rnd(N, dtype=dtype)
    close(k().gemm(x, w, bias=b), ref.gemm(x.cpu(), w.cpu(), bias=b.cpu()), dtype)
    close(k().gemm(x, w, act=6), ref.gemm(x.cpu(), w.cpu(), act=6), dtype)
    acc = rnd(M, N, seed=1)
    want = acc.cpu() + ref.gemm(x.cpu(), w.cpu(), bias=b.cpu(), out_dtype=F32)
    k().gemm_accum(x, w, acc, bias=b)
    close(acc, want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("E,top", [(7, 3), (12, 1), (40, 12), (9, 9)])
def test_sigmoid_router_and_weighted_inputs(E, top, dtype):
    from hcache_deepspeed_b200.models.arch import FeedForwardSpec
    from hcache_deepspeed_b200.models.weights import ExpertWeights, LayerWeights
    from hcache_deepspeed_b200.ops.backend import CpuOps, CudaOps
    W, ff, T = 64, 32, 270
    E8 = -(-E // 8) * 8
    ex = [ExpertWeights(rnd(ff, W, seed=e, dtype=dtype, scale=0.2), rnd(W, ff, seed=e, dtype=dtype, scale=0.2)) for e in range(E)]
    router = torch.nn.functional.pad(rnd(E, W, seed=99, scale=0.3), (0, 0, 0, E8 - E)).to(dtype)
    lw = LayerWeights(experts=ex, w_router=router)
    lw.stack_experts()
    f = FeedForwardSpec(ff=ff, act="relu2", experts=E, top=top, routing="sigmoid", gated=False)
    rows = k().moe_padded_rows(T, E, top)
    z = lambda *s, dt=torch.int32: torch.zeros(s, dtype=dt, device="cuda")  # noqa: E731
    bufs = dict(scores=z(T, top, dt=F32), expert_ids=z(T, top), offsets=z(T, top), mapped_slots=z(T, top), counts=z(E), pad_off=z(E + 1),
                logits=z(T, E8, dt=F32), xs=z(rows, W, dt=dtype), hs=z(rows, ff, dt=dtype), ys=z(rows, W, dt=dtype))
    cl = LayerWeights(experts=[ExpertWeights(e.w_up.cpu(), e.w_down.cpu()) for e in lw.experts], w_router=router.cpu())
    gpu, cpu = CudaOps(), CpuOps()
    for n in (T, 3, 140):
        x = rnd(n, W, seed=n, dtype=dtype)
        cpu.sigmoid_route(x.cpu(), cl, f, None)
        want = cpu.routed_experts(x.cpu(), None, cl, f, 6, None, torch.zeros(n, W), None)
        gpu.sigmoid_route(x, lw, f, bufs)
        assert not bufs["logits"].any()
        ids, order = bufs["expert_ids"][:n].cpu().long().sort(-1)
        same = (ids == cpu._picked.sort(-1).values).all(-1)
        assert same.float().mean() > 0.99           # (a close call may fall either way)
        got = gpu.routed_experts(x, None, lw, f, 6, None, torch.full((n, W), 9.0, device="cuda"), bufs).cpu()
        close(got[same], want[same], dtype, coarse=3e-2)


def test_saturated_sigmoids_still_choose_the_largest():
    T, E = 4, 8
    logits = torch.full((T, E), 30.0, device="cuda")
    logits[:, 5], logits[:, 2] = 60.0, 50.0
    scores, ids, off, counts = torch.zeros(T, 2, device="cuda"), *(torch.zeros(s, dtype=torch.int32, device="cuda") for s in ((T, 2), (T, 2), (E, )))
    k().moe_topk_gating(logits, 2, False, scores, ids, off, counts, sigmoid=True)
    assert (ids == i32([5, 2])).all() and (scores == 1.0).all()


# ---- whole models ----------------------------------------------------------------------------------------------------------
MODELS = {"mixed": H.MIXED, "odd": H.ODD, "wide": H.WIDE, "tiled": H.TILED}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_and_portions(name, dtype):
    H.check_whole_and_portions(MODELS[name], dtype, "cuda", n=400 if name == "tiled" else 190)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "tiled", "wide"])
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
    w, t = H.weights(cfg, seed=2, run_in=F16), H.tokens(cfg, 60)
    eng = H.engine(cfg, w, F16, "cuda")
    assert H.error(H.run(eng, 0, t, [20]), H.expected(cfg, w, t)) < H.TOLERANCE[F16]
    assert eng.graph_replays > 20


def test_scales_that_are_not_positive():
    for scale in (0.0, -0.3):
        cfg = H.config([(H.attention(dim=64, vdim=64, rot=64, scale=scale), None), (H.parallel(heads=4, kv=2, dim=64, vdim=64, rot=32, scale=scale), None)])
        for dtype in (F32, BF16):
            w, t = H.weights(cfg, run_in=dtype), H.tokens(cfg, 170)
            assert H.error(H.run(H.engine(cfg, w, dtype, "cuda"), 0, t, [150, 2]), H.expected(cfg, w, t)) < H.TOLERANCE[dtype]
