"""Lotelix on the CPU back end: every mechanism against its plain restatement, then whole models through the engine."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from hcache_deepspeed_b200.models.arch import AttentionSpec, FeedForwardSpec, GRUSpec, LinearAttentionSpec, RotationSpec, arch_from_hf_config
from hcache_deepspeed_b200.models.weights import ExpertWeights, LayerWeights
from hcache_deepspeed_b200.ops import reference as ref
from hcache_deepspeed_b200.ops.backend import CpuOps

from . import lotelix_helper as H
from . import lotelix_oracle as oracle

pytestmark = pytest.mark.timeout(600)
F32 = torch.float32
MODELS = {"mixed": H.MIXED, "odd": H.ODD, "wide": H.WIDE}


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed + sum(shape)))


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
def test_gru_in_pieces():
    n, C = 30, 11
    z, u = rnd(n, C) * 2, rnd(n, C, seed=1) * 3
    u[3] = 0.0                                        # (zero belongs to the upper branch)
    s, c = oracle.sigmoid(z.double()), torch.where(u >= 0, u.double() + 0.5, oracle.sigmoid(u.double()))
    assert (c[3] == 0.5).all()
    want = oracle.gru_recurrence(s, c)
    state, out = torch.zeros(C), []
    for a, b in ((0, 11), (11, 12), (12, n)):
        out.append(ref.gru_scan(z[a:b], u[a:b], state))
    torch.testing.assert_close(torch.cat(out), want.float(), rtol=1e-5, atol=1e-6)
    torch.testing.assert_close(state, want[-1].float(), rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("heads,N,P,tau", [(4, 6, 7, 1.0), (3, 5, 4, 16.0), (1, 9, 3, 0.5)])
def test_linear_recurrence_in_pieces(heads, N, P, tau):
    n = 30
    q, k, v, z = rnd(n, heads, N), rnd(n, heads, N, seed=1), rnd(n, heads, P, seed=2), rnd(n, heads, N, seed=3) * 4
    alpha = oracle.sigmoid(z.double())**(1 / tau)
    torch.testing.assert_close(ref.linear_decay(z, tau), alpha.float(), rtol=1e-4, atol=1e-6)
    want = oracle.linear_recurrence(q.double() * N**-0.5, k.double(), v.double(), alpha)
    state, out = torch.zeros(heads, P, N), []
    for a, b in ((0, 11), (11, 12), (12, n)):
        out.append(ref.linear_scan(q[a:b], k[a:b], v[a:b], alpha[a:b].float(), state))
    torch.testing.assert_close(torch.cat(out), want.float(), rtol=1e-4, atol=1e-4)


def test_decay_of_extreme_inputs():
    z = torch.tensor([-1e4, -90.0, 0.0, 90.0, 1e4])
    d = ref.linear_decay(z, 16.0)
    assert torch.isfinite(d).all() and d[0] == 0.0 and (d[3:] == 1.0).all()
    torch.testing.assert_close(d[1], torch.tensor(np.exp(-90 / 16), dtype=F32), rtol=1e-5, atol=0)


@pytest.mark.parametrize("adjacent", [False, True])
@pytest.mark.parametrize("dim,dims,scaling", [(20, 12, None), (64, 64, (8.0, 1.0, 4.0, 64)), (70, 2, None), (24, 24, (3.0, 0.5, 6.0, 300)), (130, 34, None)])
def test_rotation_of_reordered_rows(dim, dims, scaling, adjacent):
    """Heads whose rows were reordered at load, rotated by halves of the page size, score like heads rotated as the design pairs them."""
    from hcache_deepspeed_b200.models.hybrid import _query_rows, rotated_places
    n, heads, base = 90, 3, 700.0
    sc = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    rot = {"base": base, "dims": dims, "scaling": sc}
    slow = dict(slow_factor=sc["factor"], slow_low=sc["low"], slow_high=sc["high"], original=sc["original"]) if sc else {}
    spec = AttentionSpec(heads, heads, dim, dim, 1.0, rot=RotationSpec(dims, base, adjacent, **slow))
    D = spec.page_dim
    places = rotated_places(spec)
    assert len(set(places.tolist())) == dim and int(places.max()) < D
    f = torch.tensor(spec.rot.frequencies(), dtype=torch.float64)
    torch.testing.assert_close(f, oracle.frequencies(rot), rtol=1e-12, atol=0)
    freq = torch.cat([f, torch.zeros(D // 2 - dims // 2)]).float()
    q, k = rnd(n, heads, dim), rnd(n, heads, dim, seed=1)
    rows = [ref.rope_rotate_half(_query_rows(x.reshape(n, -1).t(), heads, spec).t().reshape(n, heads, D), torch.arange(n), freq, D) for x in (q, k)]
    want = [oracle.rotate(x.double(), rot, adjacent) for x in (q, k)]
    got = torch.einsum("ihd,jhd->hij", *rows)
    torch.testing.assert_close(got, torch.einsum("ihd,jhd->hij", *want).float(), rtol=1e-4, atol=1e-3)


def test_three_ranges_of_a_slowed_rotation():
    r = RotationSpec(32, 1e4, slow_factor=8.0, slow_low=1.0, slow_high=4.0, original=200)
    plain, f = RotationSpec(32, 1e4).frequencies(), r.frequencies()
    ratio = [a / b for a, b in zip(f, plain)]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 8) and any(1 / 8 < x < 1 for x in ratio)


def attend(q, cache, table, items, n_kv, **kw):
    return ref.paged_attention(q, cache, table[None], torch.tensor(items, dtype=torch.int32), q.shape[1], n_kv, 1.0, **kw)


@pytest.mark.parametrize("window", [1, 2, 7, 16, 64])
@pytest.mark.parametrize("kind", ["sink", "sigmoid"])
def test_attention_window_edges(kind, window):
    """One cached key of huge score at a time: exactly the queries whose window holds it return its value."""
    n, heads, page = 50, 2, 16
    cache0, table = H.attention_case(8, heads, 1, page, F32, "cpu", n)
    q = torch.zeros(n, heads, 8)
    q[..., 0] = 50.0
    i = torch.arange(n)
    opts = {"sink": torch.full((heads, ), 8.0)} if kind == "sink" else {"sigmoid_bias": torch.full((heads, ), -20.0)}
    for j in (0, 1, 15, 16, 31, 40, n - 1):
        cache = cache0.clone()
        cache[int(table[j // page]), 0, :, j % page, 0] = 1.0
        cache[int(table[j // page]), 1, :, j % page] = 1.0
        for items in ([[0, 0, n, 0]], [[0, 0, 20, 0], [0, 20, 1, 20], [0, 21, n - 21, 21]]):
            got = attend(q, cache, table, items, 1, window=window, **opts)
            sees = (i >= j) & (i - j < window)
            assert ((got.amin((1, 2)) > 0.9) == sees).all() and ((got.amax((1, 2)) < 0.1) == ~sees).all(), j


def test_sink_takes_its_share_and_sigmoid_weights_add_up():
    """Equal keys: with a sink, n of n + exp(sink) shares are left for them; sigmoid weights grow with the number of keys."""
    n, heads, page = 40, 3, 16
    cache, table = H.attention_case(8, heads, 1, page, F32, "cpu", n)
    cache[:, 1] = 1.0
    q, sink = torch.zeros(n, heads, 8), torch.tensor([0.0, 2.0, -30.0])
    count = torch.arange(1, n + 1).float()[:, None]
    got = attend(q, cache, table, [[0, 0, n, 0]], 1, sink=sink)[..., 0]
    torch.testing.assert_close(got, count / (count + sink.exp()), rtol=1e-5, atol=1e-6)
    got = attend(q, cache, table, [[0, 0, n, 0]], 1, sigmoid_bias=sink)[..., 0]
    torch.testing.assert_close(got, count * oracle.sigmoid(sink), rtol=1e-5, atol=1e-6)
    gate = rnd(n, heads * 8)
    got = attend(q, cache, table, [[0, 0, n, 0]], 1, sigmoid_bias=sink, gate=gate)
    torch.testing.assert_close(got, (count * oracle.sigmoid(sink))[..., None] * oracle.sigmoid(gate).view(n, heads, 8), rtol=1e-5, atol=1e-6)


def test_attention_mixers_end_to_end():
    """Projections, biases, norms, rotation, mask, weights, gate and output of one mixer of each kind, cut into portions."""
    for layer in (H.attention(size=9), H.parallel(), H.gru()):
        cfg = H.config([(layer, None)])
        w, t = H.weights(cfg), H.tokens(cfg, 33)
        assert H.error(H.run(H.engine(cfg, w), 0, t, [2, 3, 1, 17]), H.expected(cfg, w, t)) < H.TOLERANCE[F32], layer["type"]


@pytest.mark.parametrize("scale", [0.0, -0.3])
def test_scales_that_are_not_positive(scale):
    for layer in (H.attention(scale=scale), H.parallel(scale=scale)):
        cfg = H.config([(layer, None)])
        w, t = H.weights(cfg), H.tokens(cfg, 20)
        assert H.error(H.run(H.engine(cfg, w), 0, t, [7, 2]), H.expected(cfg, w, t)) < H.TOLERANCE[F32]


def test_values_are_mixed_with_the_first_mixing_layers():
    """The share of a later layer is audible, that of the first one is not; layers in between that do not mix change nothing."""
    cfg = H.config([(H.attention(), None), (H.attention(v_mix=True), None), (H.attention(size=5), None), (H.attention(v_mix=True), None)])
    w, t = H.weights(cfg), H.tokens(cfg, 40)
    want = H.expected(cfg, w, t)
    assert H.error(H.run(H.engine(cfg, w), 0, t, [2, 30]), want) < H.TOLERANCE[F32]
    w["l1.mix.vmix"] = torch.tensor(9.0)
    assert H.error(H.run(H.engine(cfg, w), 0, t, [2, 30]), want) < H.TOLERANCE[F32]
    del w["l1.mix.vmix"]
    assert H.error(H.run(H.engine(cfg, w), 0, t, [2, 30]), want) < H.TOLERANCE[F32]
    w["l3.mix.vmix"] = torch.tensor(0.0)
    assert H.error(H.run(H.engine(cfg, w), 0, t, [2, 30]), want) > 0.02


@pytest.mark.parametrize("cols,groups", [(20, 1), (20, 4), (20, 20), (75, 5)])
def test_grouped_norm_and_two_normed_outputs(cols, groups):
    pad = -(-cols // 8) * 8
    z = lambda t: torch.nn.functional.pad(t, (0, pad - cols))  # noqa: E731
    x, d, d2, g, p, p2 = (z(t) for t in (rnd(6, cols), rnd(6, cols, seed=1), rnd(6, cols, seed=2), rnd(cols), rnd(cols, seed=3), rnd(cols, seed=4)))
    s, o = ref.norm_residual(x, g, d, 1.0, p, cols, 1e-3, groups, d2, p2)
    want = x + z(oracle.rms(d[:, :cols], 1e-3)) * p + z(oracle.rms(d2[:, :cols], 1e-3)) * p2
    torch.testing.assert_close(s, want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(o, z(oracle.grouped_rms(want[:, :cols], groups, 1e-3)) * g, rtol=1e-5, atol=1e-5)


def test_router_weighs_what_experts_read():
    T, W, E, top = 40, 12, 6, 2
    x, w = rnd(T, W), {"router": rnd(E, W, seed=1)}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = rnd(8, W, seed=e), rnd(W, 8, seed=e)
    want = oracle.mixture(x.double(), oracle.cast(w), "", {"top": top}).float()
    lw = LayerWeights(experts=[ExpertWeights(w[f"e{e}.up"], w[f"e{e}.down"]) for e in range(E)], w_router=torch.cat([w["router"], torch.zeros(2, W)]))
    f = FeedForwardSpec(ff=8, act="relu2", experts=E, top=top, routing="sigmoid", gated=False)
    ops = CpuOps()
    ops.sigmoid_route(x, lw, f, None)
    torch.testing.assert_close(ops.routed_experts(x, None, lw, f, 6, None, torch.zeros(T, W), None), want, rtol=1e-4, atol=1e-4)
    s = oracle.sigmoid(x @ w["router"].T)            # weighing the outputs instead would be another function
    outputs = sum((s[:, e:e + 1] * oracle.expert(x, w, f"e{e}.")) * (s >= s.topk(top).values[:, -1:])[:, e:e + 1] for e in range(E))
    assert (outputs - want).abs().max() > 0.1


def test_embedding_factor():
    ids, w = torch.tensor([3, 0, 5], dtype=torch.int32), rnd(7, 16)
    torch.testing.assert_close(CpuOps().embed_f32(ids, w, torch.empty(3, 16), scale=2.5), w[ids.long()] * 2.5)


# ---- models through the engine -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_and_portions(name):
    H.check_whole_and_portions(MODELS[name], F32, "cpu", n=150)


def test_mixed_batches_reuse_pages_and_slots():
    H.check_mixed_batches(H.MIXED, F32, "cpu")


def test_stacks_without_recurrent_layers_and_without_attention():
    H.check_whole_and_portions(H.config([(H.attention(v_mix=True), H.moe()), (H.attention(size=30, v_mix=True), None)]), F32, "cpu", n=120)
    H.check_whole_and_portions(H.config([(H.gru(), H.moe()), (H.gru(width=33), None)]), F32, "cpu", n=120)


def test_attention_without_a_window():
    cfg = H.config([(H.attention(), H.moe()), (H.attention(), None)])
    del cfg["layers"][0]["mixer"]["mask"]
    cfg["layers"][1]["mixer"]["mask"] = None
    H.check_whole_and_portions(cfg, F32, "cpu", n=120)


def test_restore_from_hidden_states():
    H.check_restore(H.MIXED, F32, "cpu")


def test_greedy_generation(tmp_path):
    H.check_greedy(H.MIXED, F32, False, tmp_path / "m")


def test_serialize_round_trip(tmp_path):
    from hcache_deepspeed_b200.inference.v2 import build_hf_engine
    cfg = H.MIXED
    w, t = H.weights(cfg), H.tokens(cfg, 20)
    eng = H.engine(cfg, w)
    want = H.run(eng, 0, t)
    eng.serialize(str(tmp_path / "ser"))
    torch.testing.assert_close(H.run(build_hf_engine(str(tmp_path / "ser"), eng.config), 0, t), want)


def test_pages_and_state_of_each_layer():
    eng = H.engine(H.MIXED, H.weights(H.MIXED), tokens=128)
    c, s = eng.state_manager.kv_cache, eng.state_manager.recurrent_states
    assert [None if c.get_cache(i) is None else tuple(c.get_cache(i).shape[1:]) for i in range(8)] == [
        None, (2, 2, 64, 64), (2, 3, 64, 64), (2, 2, 64, 64), None, (2, 2, 64, 64), (2, 2, 64, 128), (2, 1, 64, 64)]
    assert [None if s.ssm(i) is None else tuple(s.ssm(i).shape[1:]) for i in range(8)] == [
        (1, 72, 1), None, (2, 18, 10), None, (1, 96, 1), None, None, (3, 40, 24)]


def test_errors_name_what_is_wrong():
    for name, piece in (("l0.mix.a", None), ("l0.mix.right.a2.b", "linear.a2_b"), ("l1.mix.z.b", "gru.z_b"), ("l2.mix.sink", "attn.sink"),
                        ("l3.mix.vmix", "attn.vmix"), ("l0.mix.left.pb", "attn.pb"), ("l0.mlp.router", "moe.router"), ("l0.norm2", "norm2.g")):
        w = H.weights(H.ODD)
        if piece is None:
            H.engine(H.ODD, dict(w, **{name: w["l0.norm1"]}))        # (a tensor nobody asked for does no harm)
            continue
        del w[name]
        with pytest.raises(ValueError, match=piece):
            H.engine(H.ODD, w)
    arch = lambda *layers, **kw: arch_from_hf_config(dict(H.config(list(layers), **kw), model_type="lotelix"))  # noqa: E731
    for bad in ([(H.gru(), {"kind": "lattice"})], [({"type": "rings", "mixer": {}}, None)], [(H.attention(rot=22), None)], [(H.attention(rot=7), None)],
                [(H.attention(heads=5), None)], [(H.attention(v_mix=True), None), (H.attention(vdim=20, v_mix=True), None)]):
        with pytest.raises(ValueError, match="lotelix"):
            arch(*bad)
    with pytest.raises(ValueError, match="groups"):
        arch((H.gru(), None), groups=3)


def test_parameter_count_matches_the_checkpoint():
    for cfg in (H.MIXED, H.ODD, H.TILED, H.WIDE):
        spec = H.engine(cfg, H.weights(cfg), tokens=64).model().spec          # (ranks are known once weights are there)
        first = sum(n.endswith("vmix") for n in H.weights(cfg)) > 0          # (the first mixing layer's share is not used)
        assert spec.param_count() + first == sum(t.numel() for t in H.weights(cfg).values())


def test_specs_of_one_layer():
    assert GRUSpec(37).inner == 40 and GRUSpec(37).in_dim == 120
    g = LinearAttentionSpec(3, 7, 9)
    assert (g.keys, g.inner, g.state) == (24, 32, 7)


def test_named_stacks_build_and_run():
    from hcache_deepspeed_b200.models.arch import named_arch
    spec = named_arch("lotelix-2048")
    assert len(spec.layers) >= 3 and {type(l.mixer.recurrent) for l in spec.layers} == {GRUSpec, LinearAttentionSpec, type(None)}


def test_trace_runner_process(tmp_path):
    cfg = H.ODD
    w, a, b = H.weights(cfg), H.tokens(cfg, 30), H.tokens(cfg, 12, seed=2)
    path = H.save(tmp_path / "m", cfg, w)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20].tolist(), "want": [0, 19]}, {"id": "b", "tokens": b[:2].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:].tolist(), "want": [9]}, {"id": "a", "tokens": a[20:21].tolist(), "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[21:].tolist(), "want": []}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "128", "--device", "cpu"], input="\n".join(map(json.dumps, steps)), capture_output=True, text=True, timeout=500)
    assert out.returncode == 0 and out.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"], out.stderr[-2000:]
    got = [torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy()) for i in (0, 1)]
    wa, wb = H.expected(cfg, w, a), H.expected(cfg, w, b)
    assert H.error(got[0], wa[[0, 19]]) < 1e-4 and H.error(got[1], torch.stack([wb[11], wa[20]])) < 1e-4
    assert not os.path.exists(tmp_path / "2.f32")
