"""Relulix on the GPU: each kernel against its fp32 restatement, then whole models against the plain oracle."""
import math

import pytest
import torch

from hcache_deepspeed_b200.ops import reference as ref

from . import relulix_helper as H
from . import relulix_oracle as oracle
from .test_gpu_lotelix import KINDS, attend, batches, close, i32, k, rnd

pytestmark = [pytest.mark.gpu, pytest.mark.timeout(600)]
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16


# ---- attention with bounded scores ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
@pytest.mark.parametrize("cap,size", [(5.0, 1.0), (30.0, 0.2), (1.0, 3.0)])
@pytest.mark.parametrize("window", [0, 90])
def test_attention_against_reference(kind, d, n_q, n_kv, cap, size, window):
    """Scores far below the bound, around it and far above it; with and without a one more in the denominator."""
    page, n_keys = 64, 500
    n = 150 if kind.startswith("prefil") else 5
    for dtype in ([BF16, F16] if kind != "generic" else [BF16, F32]):
        cache, table = H.attention_case(d, n_q, n_kv, page, dtype, "cuda", n_keys)
        cache = torch.randn(cache.shape, generator=torch.Generator().manual_seed(1)).to(dtype).cuda()
        q = rnd(n, n_q, d, dtype=dtype, scale=size)
        items = torch.tensor([[0, 0, n, n_keys - n]], dtype=torch.int32)
        for sink in (None, torch.zeros(n_q)):
            want = ref.paged_attention(q.cpu().float(), cache.cpu(), table[None], items, n_q, n_kv, 1.0, window=window, softcap=cap, sink=sink)
            got = attend(kind, q, cache, table, n_keys - n, n_kv, window, softcap=cap, sink=None if sink is None else sink.cuda())
            assert (got.float().cpu() - want).abs().max() < (1e-4 if dtype == F32 else 1e-2) * want.abs().max()


@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
@pytest.mark.parametrize("window", [1, 48, 128, 300, 0])
def test_planted_key_is_seen_exactly_inside_its_window(kind, d, n_q, n_kv, window):
    """A key whose bounded score still stands out: its value shows in the output of exactly the queries that see it, at the window's
    edges, at page borders, far back and first of all; unseen, the one more in the denominator keeps the rest small."""
    page, n_keys = 64, 700
    n = 150 if kind.startswith("prefil") else 2
    cache0, table = H.attention_case(d, n_q, n_kv, page, BF16, "cuda", n_keys)
    q = torch.zeros(n, n_q, d, dtype=BF16, device="cuda")
    q[..., 0] = 8.0
    sink = torch.zeros(n_q, device="cuda")
    for pos0 in (n_keys - n, 447, 130):
        pos0 = min(pos0, n_keys - n)
        last = pos0 + n - 1
        places = {0, 1, pos0 - window, pos0 - window + 1, last - window, last - window + 1, pos0, last, 63, 64, 128}
        for j in sorted(p for p in places if 0 <= p <= last):
            cache = cache0.clone()
            cache[int(table[j // page]), 0, :, j % page, 0] = 8.0
            cache[int(table[j // page]), 1, :, j % page] = 1.0
            got = attend(kind, q, cache.cuda(), table, pos0, n_kv, window, softcap=20.0, sink=sink).float()
            i = torch.arange(pos0, pos0 + n, device="cuda")
            sees = (j <= i) & ((i - j < window) if window else True)
            assert ((got.amin((1, 2)) > 0.9) == sees).all() and ((got.amax((1, 2)) < 0.1) == ~sees).all(), (j, pos0)


@pytest.mark.parametrize("kind,d,n_q,n_kv", KINDS)
def test_weights_of_equal_scores(kind, d, n_q, n_kv):
    """n keys of one score s weigh n e^c / (1 + n e^c) together, c the bounded score: also where e^c is far from one, of either sign, and
    for the first tokens of a sequence."""
    page, cap = 64, 6.0
    for s in (-40.0, -3.0, 0.0, 2.0, 40.0):
        cache, table = H.attention_case(d, n_q, n_kv, page, BF16, "cuda", 700)
        cache[:, 1] = 1.0
        cache[:, 0, ..., 0] = s
        e = math.exp(cap * math.tanh(s / cap))
        for pos0, n in ((0, 5), (0, 1), (600, 2)):
            q = torch.zeros(n, n_q, d, dtype=BF16, device="cuda")
            q[..., 0] = 1.0
            count = torch.arange(pos0 + 1, pos0 + n + 1, device="cuda").float()[:, None].expand(n, n_q)
            got = attend(kind, q, cache.cuda(), table, pos0, n_kv, sink=torch.zeros(n_q, device="cuda"), softcap=cap)
            torch.testing.assert_close(got.float().mean(-1), count * e / (1 + count * e), rtol=1e-2, atol=1e-4)


def test_the_bound_lasts_for_one_launch():
    d, n_kv, page = 64, 2, 64
    cache, table = H.attention_case(d, n_kv, n_kv, page, BF16, "cuda", 100)
    cache[int(table[0]), 0, :, 7, 0], cache[int(table[0]), 1, :, 7] = 8.0, 1.0
    q = torch.zeros(2, n_kv, d, dtype=BF16, device="cuda")
    q[..., 0] = 8.0
    for kind in ("split1", "prefil1", "generic"):
        assert attend(kind, q, cache.cuda(), table, 50, n_kv, softcap=0.5).max() < 0.1
        assert (attend(kind, q, cache.cuda(), table, 50, n_kv).float() - 1).abs().max() < 1e-2


# ---- rotation ------------------------------------------------------------------------------------------------------------
def rotated_case(T, n_q, n_kv, D, dtype):
    proj = rnd(T, (n_q + 2 * n_kv) * D + 16, dtype=dtype)[:, :(n_q + 2 * n_kv) * D]
    pos = torch.randint(0, 3000, (T, ), generator=torch.Generator().manual_seed(0)).int()
    slot = torch.randperm(4 * 64, generator=torch.Generator().manual_seed(1))[:T].int()
    freq = torch.cat([500.0**(-torch.arange(D // 4) / (D // 4)), torch.zeros(D // 2 - D // 4)]).float()
    amp = torch.cat([torch.full((D // 4, ), 1.3), torch.ones(D // 2 - D // 4)])
    return proj, pos, slot, freq, amp


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("n_q,n_kv,D", [(6, 2, 64), (8, 8, 128), (3, 1, 136)])
def test_append_with_amplitudes_and_queries_alone(n_q, n_kv, D, dtype):
    T, page = 37, 64
    proj, pos, slot, freq, amp = rotated_case(T, n_q, n_kv, D, dtype)
    slot[5] = -1
    cache, q = torch.full((4, 2, n_kv, page, D), 3.0, dtype=dtype, device="cuda"), torch.zeros(T, n_q * D, dtype=dtype, device="cuda")
    k().attention_append(proj, q, cache, pos.cuda(), slot.cuda(), n_q, n_kv, D, page, freq.cuda(), amp=amp.cuda())
    want = torch.full((4, 2, n_kv, page, D), 3.0)
    want_q = ref.attention_append(proj.float().cpu(), want, pos, slot, n_q, n_kv, freq, None, None, 0, 0, 0.0, None, None, amp)
    close(q, want_q, dtype, fine=1e-3)
    close(cache, want, dtype, fine=1e-3)
    alone = torch.zeros_like(q)
    k().attention_append(proj[:, :n_q * D], alone, None, pos.cuda(), slot.cuda(), n_q, 0, D, page, freq.cuda(), amp=amp.cuda())
    assert torch.equal(alone, q)


@pytest.mark.parametrize("T,n_q,n_kv,D", [(140, 4, 2, 64), (300, 6, 2, 128), (2100, 32, 8, 128)])
@pytest.mark.parametrize("own", [True, False])
def test_fused_projection_with_amplitudes_and_queries_alone(T, n_q, n_kv, D, own):
    page, W, n_kv = 64, 64, n_kv if own else 0
    rows = (n_q + 2 * n_kv) * D
    x, w, b = rnd(T, W, dtype=BF16, scale=0.3), rnd(rows, W, dtype=BF16, scale=0.3), rnd(rows, dtype=BF16)
    _, _, _, freq, amp = rotated_case(8, n_q, max(n_kv, 1), D, BF16)
    blocks = -(-T // page)
    pos, slot = (torch.arange(T) + 11).int(), torch.randperm(blocks * page)[:T].int()
    cache = torch.full((blocks, 2, max(n_kv, 1), page, D), 3.0, dtype=BF16, device="cuda")
    q = torch.zeros(T, n_q * D, dtype=BF16, device="cuda")
    k().qkv_rope_proj(x, w, q, cache, pos.cuda(), slot.cuda(), freq.cuda(), n_q, n_kv, D, page, bias_qkv=b, amp=amp.cuda())
    y = ref.gemm(x.cpu(), w.cpu(), bias=b.cpu(), out_dtype=F32)
    want = torch.full(cache.shape, 3.0)
    want_q = ref.attention_append(y, want, pos, slot, n_q, n_kv, freq, None, None, 0, 0, 0.0, None, None, amp, D)
    close(q, want_q, BF16)
    close(cache, want, BF16)


# ---- retention -------------------------------------------------------------------------------------------------------------
def retention_case(T, heads, N, P, dtype, seed):
    proj = rnd(T, 2 * heads * N + 2 * heads * P + 16, seed=seed, dtype=dtype)
    return proj[:, :heads * N], proj[:, heads * N:2 * heads * N], proj[:, 2 * heads * N:heads * (2 * N + P)], proj[:, heads * (2 * N + P):2 * heads * (N + P)]


def turning(N, dims=None, base=300.0, amplitude=None):
    n = (N if dims is None else dims) // 2
    freq = torch.cat([base**(-torch.arange(n) / max(n, 1)), torch.zeros(N // 2 - n)]).float().cuda()
    return freq, None if amplitude is None else torch.cat([torch.full((n, ), amplitude), torch.ones(N // 2 - n)]).float().cuda()


def workspace(T, seqs, heads, P, N, cells=0):
    n = cells * heads * P * N * 4 if cells else k().retention_workspace_bytes(T, seqs, heads, P, N)
    return torch.empty(n, dtype=torch.uint8, device="cuda") if n else None


RETENTION = [(2, 64, 16), (3, 48, 48), (4, 64, 128), (2, 128, 64), (3, 64, 112), (1, 272, 150), (2, 256, 64), (2, 128, 144), (1, 128, 256), (5, 64, 48), (1, 2, 1)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("heads,N,P", RETENTION)
@pytest.mark.parametrize("turned", [False, True])
def test_retention_against_reference(heads, N, P, turned, dtype):
    eps, scale = 1e-4, 0.7 * N**-0.5
    cols = max(1, P - 3)                                 # (the last three values are padding)
    state = rnd(4, heads, P, N, seed=5)
    state[:, :, cols:] = 0
    st = state.cpu().clone()
    decay = torch.tensor([0.0, -0.02, -0.5, -5.0, -200.0][:heads])
    freq, amp = turning(N, N // 2 // 2 * 2, amplitude=1.2 if P % 2 else None)
    ws = workspace(300, 4, heads, P, N)
    for step, T, spans, single in batches():
        q, kk, v, g = retention_case(T, heads, N, P, dtype, 10 * step)
        v.view(T, heads, P)[..., cols:] = 0
        y = torch.zeros(T, -(-heads * P // 8) * 8, device="cuda")
        out = torch.full((T, -(-heads * P // 8) * 8 + 8), 4.0, dtype=dtype, device="cuda")
        other = state.clone()
        args = (q, kk, v, g, decay.cuda(), None if turned else freq, amp, scale, cols)
        k().retention(*args, state, i32(spans), single, y, out[:, :heads * P], torch.ones(heads * P, device="cuda"), eps, ws)
        k().retention(*args, other, i32(spans), single, y, None, torch.ones(heads * P, device="cuda"), eps, ws)
        assert torch.equal(state, other) and (out[:, heads * P:] == 4.0).all()
        for r0, n, at, s in spans:
            if at == 0:
                st[s].zero_()
            f = lambda t, d: t[r0:r0 + n].cpu().float().reshape(n, heads, d)  # noqa: E731
            qk = [f(t, N) if turned else ref.rotate_halves(f(t, N), torch.arange(at, at + n), freq.cpu(), None if amp is None else amp.cpu()) for t in (q, kk)]
            o = ref.retention_scan(*qk, f(v, P), decay, scale, st[s])
            want = oracle.rms(o[..., :cols], eps).reshape(n, heads, cols) * oracle.silu(f(g, P)[..., :cols])
            close(out[r0:r0 + n, :heads * P].reshape(n, heads, P)[..., :cols], want, dtype, fine=5e-4, coarse=3e-2)
            top = st[s].abs().max()
            torch.testing.assert_close(state[s].cpu() / top, st[s] / top, rtol=0, atol=1e-4)
    assert not k().retention_stuck()


@pytest.mark.parametrize("heads,N,P", [(4, 128, 128), (3, 64, 48), (2, 64, 128), (2, 128, 144), (5, 64, 32), (2, 64, 256), (1, 128, 112), (40, 64, 64), (24, 128, 128)])
@pytest.mark.parametrize("cells", [0, 3])
def test_chunked_retention_against_token_scan(heads, N, P, cells):
    """The tensor-core form keeps 16 bits of every fp32 operand: far closer to the fp32 scan than 16-bit rounding would be. Lengths around the
    chunk borders, decays from none to ones that forget within a token, carried states, scratch for a few chunks, more work than blocks."""
    decay = torch.tensor(([-0.001, 0.0, -0.3, -30.0, -200.0] * heads)[:heads], device="cuda")
    for lens in ([2], [128, 127], [129, 3, 400], [300, 1, 257, 2], [1500]):
        T = sum(lens)
        q, kk, v, g = retention_case(T, heads, N, P, BF16, T)
        spans, row = [], 0
        for i, n in enumerate(lens):
            spans.append([row, n, 5000 if i % 2 else 0, len(lens) - 1 - i])
            row += n
        single = sum(n == 1 for n in lens)
        ws = workspace(T, len(lens), heads, P, N, cells)
        res = []
        for method in (1, 2):
            state = rnd(len(lens), heads, P, N, seed=5, scale=0.3)
            y, out = torch.zeros(T, heads * P, device="cuda"), torch.zeros(T, heads * P, dtype=BF16, device="cuda")
            k().retention(q, kk, v, g, decay, None, None, N**-0.5, P, state, i32(spans), single, y, out, torch.ones(heads * P, device="cuda"), 1e-5, ws, method)
            res.append((out.float(), state))
        assert not k().retention_stuck() and torch.isfinite(res[1][0]).all()
        top = res[0][1].abs().amax((0, 2, 3), keepdim=True)
        torch.testing.assert_close(res[1][1] / top, res[0][1] / top, rtol=0, atol=1e-4)
        torch.testing.assert_close(res[1][0], res[0][0], rtol=1e-2, atol=3e-3)


def test_a_key_far_back_is_still_there():
    """One key among hundreds of others: with a slow decay what it left is read at a distance, across chunks, decode steps and launches."""
    heads, N, P, n = 2, 64, 64, 700
    freq, _ = turning(N, 0)
    decay = torch.tensor([-0.002, -4.0], device="cuda")
    q = torch.zeros(n, heads * N, dtype=BF16, device="cuda")
    kk, v = q.clone(), torch.zeros(n, heads * P, dtype=BF16, device="cuda")
    proj = torch.cat([q, kk, v, v], 1)
    at = 5
    proj[at, heads * N::N][:heads] = 1.0          # k: channel 0 of both heads
    proj[at, 2 * heads * N:2 * heads * N + heads * P] = 1.0
    proj[:, :heads * N:N] = 1.0                   # every query asks for channel 0
    cut = lambda a, b: (proj[a:b, :heads * N], proj[a:b, heads * N:2 * heads * N], proj[a:b, 2 * heads * N:2 * heads * N + heads * P],  # noqa: E731
                        proj[a:b, 2 * heads * N + heads * P:])
    state, ws, got, p0 = torch.zeros(1, heads, P, N, device="cuda"), workspace(n, 1, heads, P, N), [], 0
    for m in (3, 200, 1, 128, 129, 2, 1, 236):
        y = torch.zeros(m, heads * P, device="cuda")
        turned = m > 128        # (all angles are zero: either form may come)
        k().retention(*cut(p0, p0 + m), decay, None if turned else freq, None, 1.0, P, state, i32([[0, m, p0, 0]]), int(m == 1), y, None,
                      torch.ones(heads * P, device="cuda"), 1e-5, ws)
        p0 += m
        got.append(state[0, :, 0, 0].clone())
        since = p0 - 1 - at
        want = torch.exp2(decay * since) if since >= 0 else torch.zeros_like(decay)
        torch.testing.assert_close(got[-1], want, rtol=1e-4, atol=1e-7)
    assert p0 == n


# ---- router and experts --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("E,top", [(7, 3), (12, 1), (40, 12), (9, 9), (1, 1)])
def test_router_with_bias_weighs_the_chosen(E, top, dtype):
    from hcache_deepspeed_b200.models.arch import FeedForwardSpec
    from hcache_deepspeed_b200.models.weights import ExpertWeights, LayerWeights
    from hcache_deepspeed_b200.ops.backend import CpuOps, CudaOps
    W, ff, T = 64, 32, 270
    E8 = -(-E // 8) * 8
    ex = [ExpertWeights(rnd(2 * ff, W, seed=e, dtype=dtype, scale=0.3), rnd(W, ff, seed=e, dtype=dtype, scale=0.3)) for e in range(E)]
    router = torch.nn.functional.pad(rnd(E, W, seed=99, scale=0.3), (0, 0, 0, E8 - E)).to(dtype)
    lw = LayerWeights(experts=ex, w_router=router, router_bias=rnd(E, seed=7, scale=2.0))
    lw.stack_experts()
    f = FeedForwardSpec(ff=ff, act="swiglu_clamped", limit=0.8, experts=E, top=top, routing="chosen")
    rows = k().moe_padded_rows(T, E, top)
    z = lambda *s, dt=torch.int32: torch.zeros(s, dtype=dt, device="cuda")  # noqa: E731
    bufs = dict(scores=z(T, top, dt=F32), expert_ids=z(T, top), offsets=z(T, top), mapped_slots=z(T, top), counts=z(E), pad_off=z(E + 1),
                logits=z(T, E8, dt=F32), xs=z(rows, W, dt=dtype), hs=z(rows, ff, dt=dtype), ys=z(rows, W, dt=dtype))
    cl = LayerWeights(experts=[ExpertWeights(e.w_up.cpu(), e.w_down.cpu()) for e in lw.experts], w_router=router.cpu(), router_bias=lw.router_bias.cpu())
    gpu, cpu = CudaOps(), CpuOps()
    for n in (T, 3, 140):
        x = rnd(n, W, seed=n, dtype=dtype)
        cpu.chosen_route(x.cpu(), cl, f, None)
        want = cpu.routed_experts(x.cpu(), None, cl, f, 5, None, torch.zeros(n, W), None)
        gpu.chosen_route(x, lw, f, bufs)
        assert not bufs["logits"].any()
        ids, order = bufs["expert_ids"][:n].cpu().long().sort(-1)
        same = (ids == cpu._picked.sort(-1).values).all(-1)
        assert same.float().mean() > 0.99           # (a close call may fall either way)
        torch.testing.assert_close(bufs["scores"][:n].cpu().sum(-1), torch.ones(n))
        base = rnd(n, W, seed=2)
        got = gpu.routed_experts(x, None, lw, f, 5, base, base, bufs).cpu()
        close(got[same], want[same] + rnd(n, W, seed=2).cpu()[same], dtype, coarse=3e-2)


def test_far_apart_logits_still_choose_the_largest():
    T, E = 4, 8
    logits = torch.full((T, E), -300.0, device="cuda")
    logits[:, 5], logits[:, 2], logits[:, 6] = 60.0, -150.0, -151.0
    bias = torch.zeros(E, device="cuda")
    bias[6] = 2.0
    scores, ids, off, counts = torch.zeros(T, 2, device="cuda"), *(torch.zeros(s, dtype=torch.int32, device="cuda") for s in ((T, 2), (T, 2), (E, )))
    k().moe_topk_gating(logits, 2, True, scores, ids, off, counts, bias=bias, biased=True)
    assert (ids == i32([5, 6])).all() and (scores == torch.tensor([1.0, 0.0], device="cuda")).all()


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
        cfg = H.config([(H.attention(dim=64, vdim=64, rot=64, scale=scale), None), (H.attention(dim=64, vdim=64, rot=64, size=40, scale=-scale, kv_from=0), None)])
        for dtype in (F32, BF16):
            w, t = H.weights(cfg, run_in=dtype), H.tokens(cfg, 170)
            assert H.error(H.run(H.engine(cfg, w, dtype, "cuda"), 0, t, [150, 2]), H.expected(cfg, w, t)) < H.TOLERANCE[dtype]
