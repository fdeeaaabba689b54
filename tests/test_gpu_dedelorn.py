"""Dedelorn on the GPU: each kernel against its fp32 restatement, then whole models against the plain oracle."""
import pytest
import torch

from hcache_deepspeed_b200.ops import reference as ref

from . import dedelorn_helper as H

pytestmark = [pytest.mark.gpu, pytest.mark.timeout(600)]
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16


def k():
    from hcache_deepspeed_b200.ops import kernels
    return kernels


def rnd(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed + sum(shape))) * scale).to(dtype).cuda()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# ---- latent attention ------------------------------------------------------------------------------------------------
def attend(q, pages, table, pos0, rank, window, splits, item_tokens=128):
    """q [n, heads, width] at positions pos0.. of one sequence whose rows are all cached already; splits 0: the generic kernel."""
    n, heads, width = q.shape
    qd, out = q.reshape(n, heads * width).contiguous(), torch.full((n, heads * rank), 5.0, dtype=q.dtype, device="cuda")
    page = pages.shape[3]
    if splits == 0:
        k().paged_attention_generic(qd, out, pages, table[None].cuda(), i32([0] * n), torch.arange(pos0, pos0 + n, dtype=torch.int32, device="cuda"),
                                    heads, 1, width, page, 1.0, window, value_dim=rank)
    else:
        ws = torch.zeros(k().latent_attention_workspace_bytes(), dtype=torch.uint8, device="cuda")
        items = i32([[0, r, min(item_tokens, n - r), pos0 + r] for r in range(0, n, item_tokens)])
        k().paged_attention_latent(qd, out, pages, table[None].cuda(), items, items.shape[0], min(n, item_tokens), heads, rank, page, splits, 1.0,
                                   ws, window)
    return out.view(n, heads, rank)


#: (splits, heads, rank, rotated, new tokens): widths of one panel up to nine, several value blocks, rows of several tokens
LATENT = [(1, 6, 112, 16, 2), (3, 5, 20, 10, 3), (1, 16, 200, 56, 40), (2, 40, 256, 32, 3), (1, 128, 512, 64, 2), (3, 7, 300, 20, 1), (1, 20, 64, 64, 130),
          (0, 3, 104, 24, 20), (0, 2, 600, 40, 3)]


@pytest.mark.parametrize("splits,heads,rank,rot,n", LATENT)
@pytest.mark.parametrize("window", [0, 1, 48, 128, 200])
def test_planted_row_is_seen_exactly_inside_its_window(splits, heads, rank, rot, n, window):
    page, n_keys = 64, 500
    width = -(-(rank + rot) // 64) * 64
    blocks = -(-n_keys // page)
    table = torch.randperm(blocks + 3, generator=torch.Generator().manual_seed(0))[:blocks].to(torch.int32)
    q = torch.zeros(n, heads, width, dtype=BF16, device="cuda")
    q[..., rank] = 8.0                       # the score comes from the rotated part, the value from the latent
    for pos0 in (n_keys - n, 190, 0):
        last = pos0 + n - 1
        places = {0, pos0 - window, pos0 - window + 1, last - window, last - window + 1, pos0, last, 63, 64, 128}
        for j in sorted(p for p in places if 0 <= p <= last):
            pages = torch.zeros(blocks + 3, 1, 1, page, width, dtype=BF16)
            pages[int(table[j // page]), 0, 0, j % page, rank] = 8.0
            pages[int(table[j // page]), 0, 0, j % page, :rank] = 1.0
            got = attend(q, pages.cuda(), table, pos0, rank, window, splits).float()
            i = torch.arange(pos0, pos0 + n, device="cuda")
            sees = (i >= j) & ((i - j < window) if window else True)
            assert ((got.amin((1, 2)) > 0.9) == sees).all() and ((got.amax((1, 2)) < 0.1) == ~sees).all(), (j, pos0)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("splits,heads,rank,rot,n", LATENT)
def test_latent_attention_against_reference(splits, heads, rank, rot, n, dtype):
    page, n_keys = 64, 700
    width = -(-(rank + rot) // 64) * 64
    blocks = -(-n_keys // page)
    table = torch.randperm(blocks, generator=torch.Generator().manual_seed(1)).to(torch.int32)
    pages = torch.nn.functional.pad(rnd(blocks, 1, 1, page, rank + rot, dtype=dtype), (0, width - rank - rot))
    q = torch.nn.functional.pad(rnd(n, heads, rank + rot, seed=2, scale=2 * rank**-0.5, dtype=dtype), (0, width - rank - rot))
    for window in (0, 150):
        want = ref.paged_latent_attention(q.cpu().float(), pages.cpu(), table[None], torch.tensor([[0, 0, n, n_keys - n]]), rank, 1.0, window)
        for item_tokens in (128, 5):
            got = attend(q, pages, table, n_keys - n, rank, window, splits, item_tokens).float().cpu()
            torch.testing.assert_close(got, want, rtol=2e-2, atol=2e-2)


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("heads,dim,rot,rank,hw", [(6, 64, 48, 96, 128), (3, 17, 6, 29, 24), (5, 40, 16, 48, 64), (2, 96, 32, 512, 128)])
def test_latent_append(heads, dim, rot, rank, hw, dtype):
    T, page, width = 37, 64, -(-(rank + rot) // 64) * 64
    n_q = heads * hw
    proj = rnd(T, -(-(n_q + rank + rot) // 8) * 8, dtype=dtype)
    pos = torch.randint(0, 3000, (T, ), generator=torch.Generator().manual_seed(0)).int()
    slot = torch.randperm(5 * page, generator=torch.Generator().manual_seed(1))[:T].int()
    from hcache_deepspeed_b200.models.hybrid import rotation_frequencies
    freq, g = rotation_frequencies(rot, 5e3).cuda(), 1 + rnd(rank, scale=0.2)
    pages, q = torch.full((5, 1, 1, page, width), 3.0, dtype=dtype, device="cuda"), torch.zeros(T, n_q, dtype=dtype, device="cuda")
    k().latent_append(proj, q, pages, pos.cuda(), slot.cuda(), heads, dim, rot, hw, rank, freq, g, 1e-5)
    p = proj.cpu().float()
    want_q = p[:, :n_q].reshape(T, heads, hw).clone()
    want_q[..., dim:dim + rot] = ref.rotate_pairs(want_q[..., dim:dim + rot], pos, freq.cpu())
    rows = ref.latent_rows(p[:, n_q:n_q + rank + rot], pos, rank, freq.cpu(), g.cpu(), 1e-5, width)
    tol = dict(rtol=1e-3, atol=1e-3) if dtype == F32 else dict(rtol=2e-2, atol=2e-2)
    torch.testing.assert_close(q.cpu().float().view(T, heads, hw), want_q, **tol)
    flat = pages.cpu().float().view(-1, width)
    torch.testing.assert_close(flat[slot.long()], rows, **tol)
    untouched = torch.ones(flat.shape[0], dtype=torch.bool)
    untouched[slot.long()] = False
    assert (flat[untouched] == 3.0).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,K,N,copy", [(6, 64, 112, 16), (3, 17, 29, 6), (4, 512, 128, 0), (2, 600, 40, 0), (5, 96, 512, 32)])
def test_head_matmul_skips_long_sequences(heads, K, N, copy, dtype):
    lens = [1, 40, 3, 1, 9]
    T, iw, ow = sum(lens), K + copy + 3, N + copy + 5
    x, w = rnd(T, heads * iw, dtype=dtype), rnd(heads, K, N, dtype=dtype, scale=K**-0.5)
    seq = i32([s for s, n in enumerate(lens) for _ in range(n)])
    spans = i32([[0, n, 0, 0] for n in lens])
    out = torch.full((T, heads * ow), 7.0, dtype=dtype, device="cuda")
    k().head_matmul(x, w, out, seq, spans, 8, iw, ow, copy)
    x3 = x.float().view(T, heads, iw)
    want = torch.cat([torch.einsum("thk,hkn->thn", x3[..., :K], w.float()), x3[..., K:K + copy], torch.zeros(T, heads, 5, device="cuda")], -1)
    live = torch.tensor([n <= 8 for n in lens for _ in range(n)], device="cuda")
    tol = 1e-4 if dtype == F32 else 2e-2
    torch.testing.assert_close(out.float().view(T, heads, ow)[live], want[live], rtol=tol, atol=tol)
    assert (out[~live] == 7.0).all()


# ---- gated delta rule --------------------------------------------------------------------------------------------------
def delta_case(heads, groups, N, P, taps, T, dtype, seed=0, decay=1.0):
    inner, C = heads * P, heads * P + 2 * groups * N
    proj = rnd(T, 8 * ((inner + C + 2 * heads + 7) // 8) + 8, seed=seed, dtype=dtype)
    return proj, (rnd(taps, C, scale=0.6), torch.zeros(C, device="cuda"), rnd(heads, seed=2) - 1, -torch.exp(rnd(heads, seed=3, scale=decay)))


DELTA = [(6, 3, 20, 28, 3), (4, 2, 64, 40, 4), (3, 1, 48, 64, 4), (2, 1, 128, 128, 4), (3, 3, 13, 11, 5), (4, 4, 16, 8, 1), (2, 1, 150, 96, 4), (3, 1, 260, 40, 2),
         (4, 1, 96, 192, 4)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("heads,groups,N,P,taps", DELTA)
@pytest.mark.parametrize("method", [0, 1])
def test_delta_rule_against_reference(heads, groups, N, P, taps, dtype, method):
    """Sequences with their own slots over several launches: long and short portions, single tokens, a slot used again."""
    inner, C, GN = heads * P, heads * P + 2 * groups * N, groups * N
    slots = 4
    state, ring = rnd(slots, heads, P, N, seed=5), rnd(slots, taps, C, seed=6)
    st_ref, ring_ref = state.cpu().clone(), ring.cpu().clone()
    gw, eps = 1 + rnd(P, seed=7, scale=0.2).repeat(heads), 1e-4
    tol = dict(rtol=2e-4, atol=2e-4) if dtype == F32 else dict(rtol=2e-2, atol=1e-2)
    ws = torch.empty(k().delta_workspace_bytes(300, 3, heads, groups), dtype=torch.uint8, device="cuda")
    seen = {}
    for step, plan in enumerate([[(0, 150), (2, 2)], [(0, 1), (2, 1), (3, 1)], [(3, 40), (0, 129), (2, 1)], [(1, 257)], [(1, 1)], [(0, 3), (1, 128)]]):
        if step == 5:
            seen[0] = 0      # slot 0 handed to another sequence
        T = sum(n for _, n in plan)
        proj, (cw, cb, db, a) = delta_case(heads, groups, N, P, taps, T, dtype, seed=10 + step)
        spans, row = [], 0
        for s, n in plan:
            spans.append([row, n, seen.get(s, 0), s])
            row += n
            seen[s] = seen.get(s, 0) + n
        u = torch.zeros(T, 8 * ((C + 7) // 8), dtype=dtype, device="cuda")
        dt, y = torch.zeros(T, heads, device="cuda"), torch.zeros(T, inner, device="cuda")
        out = torch.full((T, inner + 5 if inner % 2 else inner + 8), 4.0, dtype=dtype, device="cuda")
        k().delta_rule(proj, cw, cb, db, a, state, ring, i32(spans), sum(n == 1 for _, n in plan), groups, u, dt, y, out[:, :inner], gw, eps, ws, method)
        assert (out[:, inner:] == 4.0).all()
        for r0, n, at, s in spans:
            p = proj[r0:r0 + n].cpu()
            if at == 0:
                st_ref[s].zero_()
            vkq = ref.short_conv(p[:, inner:inner + C], ring_ref[s], cw.cpu(), cb.cpu(), at).to(dtype).float()
            g = torch.exp(a.cpu() * torch.nn.functional.softplus(p[:, inner + C:inner + C + heads].float() + db.cpu()))
            beta = torch.sigmoid(p[:, inner + C + heads:inner + C + 2 * heads].float())
            v, kk, q = vkq.split([inner, GN, GN], 1)
            want = ref.delta_scan(q.reshape(n, groups, N), kk.reshape(n, groups, N), v.reshape(n, heads, P), g, beta, st_ref[s]).reshape(n, inner)
            want = ref.gated_norm(want, p[:, :inner], gw.cpu(), heads, eps, gate_after=True)
            torch.testing.assert_close(out[r0:r0 + n, :inner].float().cpu(), want, **tol)
            torch.testing.assert_close(state[s].cpu() / st_ref[s].abs().max(), st_ref[s] / st_ref[s].abs().max(), **tol)
            filled = [q % taps for q in range(max(0, at + n - taps), at + n)]
            torch.testing.assert_close(ring[s].cpu()[filled], ring_ref[s][filled])


@pytest.mark.parametrize("heads,groups,N,P", [(4, 2, 128, 128), (3, 1, 48, 32), (2, 2, 64, 64), (2, 1, 16, 8), (6, 3, 96, 40)])
@pytest.mark.parametrize("decay", [0.3, 2.0])
def test_chunked_delta_rule_against_token_scan(heads, groups, N, P, decay):
    """The tensor-core form keeps 16 bits of every fp32 operand: far closer to the fp32 scan than 16-bit rounding would be. Lengths
    around the chunk borders, with and without carried state, slow and fast decays, equal keys (every token rewrites one row)."""
    inner, C, taps = heads * P, heads * P + 2 * groups * N, 4
    for lens in ([2], [128, 127], [129, 3, 300], [64, 1, 256, 2]):
        T = sum(lens)
        proj, (cw, cb, db, a) = delta_case(heads, groups, N, P, taps, T, BF16, seed=T, decay=decay)
        if lens == [129, 3, 300]:
            proj[:, 2 * inner:2 * inner + groups * N] = proj[:1, 2 * inner:2 * inner + groups * N]
        spans, row = [], 0
        for i, n in enumerate(lens):
            spans.append([row, n, 5 if i % 2 else 0, len(lens) - 1 - i])
            row += n
        single = sum(n == 1 for n in lens)
        ws = torch.empty(k().delta_workspace_bytes(T, len(lens) - single, heads, groups), dtype=torch.uint8, device="cuda")
        res = []
        for method in (1, 2):
            state, ring = rnd(len(lens), heads, P, N, seed=5, scale=0.3), rnd(len(lens), taps, C, seed=6)
            u = torch.zeros(T, 8 * ((C + 7) // 8), dtype=BF16, device="cuda")
            dt, y = torch.zeros(T, heads, device="cuda"), torch.zeros(T, inner, device="cuda")
            k().delta_rule(proj, cw, cb, db, a, state, ring, i32(spans), single, groups, u, dt, y, None, torch.ones(inner, device="cuda"), 1e-5, ws,
                           method)
            res.append((y, state, ring))
        for got, want in zip(res[1], res[0]):
            torch.testing.assert_close(got / want.abs().max(), want / want.abs().max(), rtol=0, atol=1e-4)


# ---- norms, router, experts ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cols,groups", [(120, 5), (256, 2), (4096, 32), (51, 3)])
def test_norm_in_front_of_the_gate(cols, groups, dtype):
    y, z, w = rnd(33, cols), rnd(33, cols + 8, dtype=dtype), rnd(cols)
    out = torch.full((33, cols + 8), 3.0, dtype=dtype, device="cuda")
    k().gated_norm(y, z[:, :cols], w, out[:, :cols], groups, 1e-3, gate_after=True)
    want = ref.gated_norm(y, z[:, :cols], w, groups, 1e-3, gate_after=True)
    tol = 1e-5 if dtype == F32 else 1e-2
    torch.testing.assert_close(out[:, :cols].float(), want, rtol=tol, atol=tol)
    assert (out[:, cols:] == 3.0).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,pad", [(75, 80), (4096, 4096)])
@pytest.mark.parametrize("delta", ["f32", "same"])
def test_plain_addition_to_the_stream(H, pad, delta, dtype):
    z = lambda t: torch.nn.functional.pad(t, (0, pad - H))  # noqa: E731
    x, g, d = z(rnd(7, H)), z(rnd(H, seed=1)), z(rnd(7, H, seed=3)).to(F32 if delta == "f32" else dtype)
    wx, wo = ref.norm_residual(x, g, d, 1.7, None, H, 1e-3)
    out = torch.empty(7, pad, dtype=dtype, device="cuda")
    k().norm_residual(x, g, out, delta=d, factor=1.7, cols=H, eps=1e-3)
    tol = 2e-5 if dtype == F32 else 1e-2
    torch.testing.assert_close(out.float(), wo, rtol=tol, atol=tol)
    torch.testing.assert_close(x, wx, rtol=2e-5, atol=2e-5)
    assert d.dtype != F32 or not d.any()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_embedding_norm(dtype):
    w, g = torch.nn.functional.pad(rnd(50, 75, dtype=dtype, scale=0.02), (0, 5)), torch.nn.functional.pad(rnd(75), (0, 5))
    ids = i32([3, 49, -1, 0, 3])
    got = k().embed_f32(ids, w, torch.empty(5, 80, device="cuda"), gamma=g, cols=75, eps=1e-4)
    x = w.float()[[3, 49, 0, 0, 3]] * torch.tensor([1, 1, 0, 1, 1], device="cuda")[:, None]
    torch.testing.assert_close(got, x * torch.rsqrt((x * x).sum(-1, keepdim=True) / 75 + 1e-4) * g, rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("E,top,gated", [(7, 3, False), (12, 1, False), (40, 12, False), (9, 9, True)])
def test_softmax_router_and_experts(E, top, gated, dtype):
    from hcache_deepspeed_b200.models.arch import FeedForwardSpec
    from hcache_deepspeed_b200.models.weights import ExpertWeights, LayerWeights
    from hcache_deepspeed_b200.ops.backend import CpuOps, CudaOps
    W, ff, T = 64, 32, 270
    E8 = -(-E // 8) * 8
    ex = [ExpertWeights(rnd((1 + gated) * ff, W, seed=e, dtype=dtype, scale=0.2), rnd(W, ff, seed=e, dtype=dtype, scale=0.2)) for e in range(E)]
    router = torch.nn.functional.pad(rnd(E, W, seed=99, scale=0.3), (0, 0, 0, E8 - E)).to(dtype)
    lw = LayerWeights(experts=ex, w_router=router, router_bias=rnd(E, scale=0.2))
    lw.stack_experts()
    f = FeedForwardSpec(ff=ff, act="gelu", experts=E, top=top, routing="softmax", gated=gated, router_scale=1.3)
    rows = k().moe_padded_rows(T, E, top)
    z = lambda *s, dt=torch.int32: torch.zeros(s, dtype=dt, device="cuda")  # noqa: E731
    bufs = dict(scores=z(T, top, dt=F32), expert_ids=z(T, top), offsets=z(T, top), mapped_slots=z(T, top), counts=z(E), pad_off=z(E + 1),
                logits=z(T, E8, dt=F32), xs=z(rows, W, dt=dtype), hs=z(rows, ff, dt=dtype), ys=z(rows, W, dt=dtype))
    cl = LayerWeights(experts=[ExpertWeights(e.w_up.cpu(), e.w_down.cpu()) for e in lw.experts], w_router=router.cpu(), router_bias=lw.router_bias.cpu())
    gpu, cpu = CudaOps(), CpuOps()
    for n in (T, 3, 140):
        x = rnd(n, W, seed=n, dtype=dtype)
        acc = rnd(n, W, seed=n + 1)
        want_in_place = acc.clone()
        cpu.softmax_route(x.cpu(), cl, f, None)
        want = cpu.routed_experts(x.cpu(), None, cl, f, 1, acc.cpu(), torch.zeros(n, W), None)
        gpu.softmax_route(x, lw, f, bufs)
        assert not bufs["logits"].any()
        got_ids, order = bufs["expert_ids"][:n].cpu().long().sort(-1)
        same = (got_ids == cpu._picked.sort(-1).values).all(-1)
        assert same.float().mean() > 0.99           # (a close call may fall either way)
        got = gpu.routed_experts(x, None, lw, f, 1, acc, acc, bufs).cpu()
        tol = 1e-4 if dtype == F32 else 3e-2
        torch.testing.assert_close(got[same], want[same], rtol=tol, atol=tol)
        gpu.softmax_route(x, lw, f, bufs)
        base = want_in_place.to(dtype)
        got = gpu.routed_experts(x, None, lw, f, 1, base, torch.full((n, W), 9.0, device="cuda"), bufs).cpu()
        torch.testing.assert_close(got[same], want[same], rtol=tol, atol=tol)


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


def test_prompts_attend_in_the_latent_space_when_scratch_pages_run_out():
    cfg = H.TILED
    w, t = H.weights(cfg, seed=5, run_in=BF16), H.tokens(cfg, 300)
    eng = H.engine(cfg, w, BF16, "cuda")
    eng.model()._latent_bufs.blocks = 1
    assert H.error(H.run(eng, 0, t, [150, 2, 100, 48]), H.expected(cfg, w, t)) < H.TOLERANCE[BF16]


def test_decode_runs_as_a_graph_and_fp16_is_served():
    cfg = H.TILED
    w, t = H.weights(cfg, seed=2, run_in=F16), H.tokens(cfg, 60)
    eng = H.engine(cfg, w, F16, "cuda")
    assert H.error(H.run(eng, 0, t, [20]), H.expected(cfg, w, t)) < H.TOLERANCE[F16]
    assert eng.graph_replays > 20
