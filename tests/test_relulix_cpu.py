"""Relulix on the CPU back end: every mechanism against its plain restatement, then whole models through the engine."""
import copy
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from hcache_deepspeed_b200.models.arch import AttentionSpec, FeedForwardSpec, RetentionSpec, RotationSpec, arch_from_hf_config
from hcache_deepspeed_b200.models.weights import ExpertWeights, LayerWeights
from hcache_deepspeed_b200.ops import reference as ref
from hcache_deepspeed_b200.ops.backend import CpuOps

from . import relulix_helper as H
from . import relulix_oracle as oracle

pytestmark = pytest.mark.timeout(600)
F32 = torch.float32
MODELS = {"mixed": H.MIXED, "odd": H.ODD, "wide": H.WIDE}


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed + sum(shape)))


def spec_of(cfg):
    return arch_from_hf_config(dict(cfg, model_type="relulix"))


# ---- rotation --------------------------------------------------------------------------------------------------------
ROTATIONS = [(22, 12, None), (64, 64, (2.0, 64, 8.0, 1.0)), (70, 2, (4.0, 4096, 32.0, 1.0)), (40, 24, (8.0, 300, 32.0, 1.0)), (130, 34, (1.0, 90, 9.0, 0.5)),
             (16, 16, (3.0, 7, 1.0, 1.0))]


@pytest.mark.parametrize("dim,dims,scaling", ROTATIONS)
def test_rotation_of_reordered_rows(dim, dims, scaling):
    """Heads whose rows were reordered at load, rotated by halves of the row, score like heads rotated as the design pairs them: attention's
    rows and retention's, positions far along, amplitudes included."""
    from hcache_deepspeed_b200.models.hybrid import _rotated_rows, rotation_table
    n, heads = 90, 3
    rot = H.rotation(dims, 700.0, scaling)
    cfg = H.config([(H.attention(heads=heads, kv=heads, dim=dim, vdim=dim, rot=dims, base=700.0, scaling=scaling), None),
                    (H.retention(heads=heads, dim=dim, rot=dims, base=700.0, scaling=scaling), None)])
    attn, ret = (l.mixer for l in spec_of(cfg).layers)
    freq, amplitude = oracle.rotation(rot)
    assert attn.attn.rot == ret.retention.rot and attn.attn.rot.amplitude == pytest.approx(amplitude, rel=1e-12)
    torch.testing.assert_close(torch.tensor(attn.attn.rot.frequencies(), dtype=torch.float64), freq, rtol=1e-12, atol=0)
    for width, r in ((attn.attn.page_dim, attn.attn.rot), (ret.retention.width, ret.retention.rot)):
        f, amp = rotation_table(r, width)
        assert len(set(r.places(dim, width))) == dim and max(r.places(dim, width)) < width
        q, k = rnd(n, heads, dim), rnd(n, heads, dim, seed=1)
        rows = [ref.rotate_halves(_rotated_rows(x.reshape(n, -1).t(), heads, dim, width, r).t().reshape(n, heads, width), torch.arange(n), f.float(),
                                  None if amp is None else amp.float()) for x in (q, k)]
        want = [oracle.rotate(x.double(), rot) for x in (q, k)]
        got = torch.einsum("ihd,jhd->hij", *rows)
        torch.testing.assert_close(got, torch.einsum("ihd,jhd->hij", *want).float(), rtol=1e-4, atol=1e-3)


def test_ranges_of_a_ramped_rotation():
    """Fast pairs as they are, slow ones slowed, a line in between; a ramp without room is a step."""
    plain = RotationSpec(32, 2e4).frequencies()
    ratio = [a / b for a, b in zip(RotationSpec(32, 2e4, slow_factor=4.0, slow_low=1.0, slow_high=16.0, original=256, ramp=True).frequencies(), plain)]
    assert ratio[0] == 1.0 and ratio[-1] == pytest.approx(1 / 4)
    steps = [a - b for a, b in zip(ratio, ratio[1:])]
    inside = [s for s in steps if s > 1e-9]
    assert len(inside) > 2 and max(inside) - min(inside) < 1e-9
    step = RotationSpec(32, 2e4, slow_factor=4.0, slow_low=1e4, slow_high=1e4, original=256, ramp=True)     # both indices below zero
    assert [a / b for a, b in zip(step.frequencies(), plain)] == pytest.approx([1.0] + [0.25] * 15)
    assert math.isclose(0.1 * math.log(3.0) + 1, spec_of(H.config([(H.attention(), None)])).layers[0].mixer.attn.rot.amplitude)


# ---- retention -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("heads,N,P", [(4, 6, 8), (3, 16, 5), (1, 2, 1)])
def test_retention_in_pieces(heads, N, P):
    n = 30
    q, k, v = rnd(n, heads, N), rnd(n, heads, N, seed=1), rnd(n, heads, P, seed=2)
    decay = torch.tensor([0.5, 1.0, 0.999, 0.0][:heads])
    want = oracle.retention_recurrence(q.double(), k.double() * 0.3, v.double(), decay.double())
    log2, state, out = decay.log2().clamp(min=-200), torch.zeros(heads, P, N), []
    for a, b in ((0, 11), (11, 12), (12, n)):
        out.append(ref.retention_scan(q[a:b], k[a:b], v[a:b], log2, 0.3, state))
    torch.testing.assert_close(torch.cat(out), want.float(), rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("decay", [[0.0, 1.0, 0.5], [0.99, 0.9, 1e-30]])
def test_extreme_decays_through_the_engine(decay):
    cfg = H.config([(H.retention(heads=3, decay=decay), None)])
    w, t = H.weights(cfg), H.tokens(cfg, 40)
    assert H.error(H.run(H.engine(cfg, w), 0, t, [2, 17, 3]), H.expected(cfg, w, t)) < H.TOLERANCE[F32]


def test_norm_over_a_heads_own_values():
    """Padded heads: the mean is taken over what the head has, and eps counts in full."""
    from hcache_deepspeed_b200.ops.backend import padded_head_norm
    m = RetentionSpec(2, 10, 21, [0.5, 0.5])
    y = torch.zeros(5, 2, m.vwidth)
    y[..., :21] = rnd(5, 2, 21) * 1e-2
    eps, scale = padded_head_norm(m, 1e-3)
    got = ref.gated_norm(y.reshape(5, -1), torch.ones(5, m.inner), torch.ones(m.inner), 2, eps, scale, gate_after=True).reshape(5, 2, -1)[..., :21]
    torch.testing.assert_close(got, oracle.rms(y[..., :21], 1e-3) * oracle.silu(torch.tensor(1.0)), rtol=1e-5, atol=1e-6)


def test_a_far_key_is_remembered_and_its_place_matters():
    """One token writes to the state, all the others nothing: it is read hundreds of tokens later, turned by its distance."""
    cfg = H.config([(H.retention(heads=2, dim=16, vdim=16, rot=16, base=50.0, decay=[0.9999, 0.99]), None)])
    w = H.weights(cfg)
    e = w["embed"].float()
    e = e - (e @ e[5])[:, None] / e[5].pow(2).sum() * e[5]
    w["embed"] = torch.where(torch.arange(cfg["vocab"])[:, None] == 5, w["embed"].float(), e)
    w["l0.mix.k"] = rnd(32)[:, None] * w["embed"][5]
    t = H.tokens(cfg, 300)
    t[t == 5] = 6
    without, other = t.clone(), t.clone()
    t[3], other[4] = 5, 5
    eng = H.engine(cfg, w)
    want = [H.expected(cfg, w, x) for x in (t, other, without)]
    for uid, (x, portions) in enumerate([(t, [100, 37]), (other, [7, 193])]):
        assert H.error(H.run(eng, uid, x, portions)[6:], want[uid][6:]) < 1e-3
    assert H.error(want[0][200:], want[1][200:]) > 0.1 and H.error(want[0][200:], want[2][200:]) > 0.1


# ---- attention -------------------------------------------------------------------------------------------------------
def attend(q, cache, table, items, n_kv, **kw):
    return ref.paged_attention(q, cache, table[None], torch.tensor(items, dtype=torch.int32), q.shape[1], n_kv, 1.0, **kw)


@pytest.mark.parametrize("window", [1, 2, 7, 16, 64])
def test_attention_window_edges(window):
    """One cached key of a bounded but large score at a time: exactly the queries whose window holds it return its value."""
    n, heads, page = 50, 2, 16
    cache0, table = H.attention_case(8, heads, 1, page, F32, "cpu", n)
    q = torch.zeros(n, heads, 8)
    q[..., 0] = 50.0
    i = torch.arange(n)
    for j in (0, 1, 15, 16, 31, 40, n - 1):
        cache = cache0.clone()
        cache[int(table[j // page]), 0, :, j % page, 0] = 1.0
        cache[int(table[j // page]), 1, :, j % page] = 1.0
        for items in ([[0, 0, n, 0]], [[0, 0, 20, 0], [0, 20, 1, 20], [0, 21, n - 21, 21]]):
            got = attend(q, cache, table, items, 1, window=window, softcap=12.0, sink=torch.zeros(heads))
            sees = (i >= j) & (i - j < window)
            assert ((got.amin((1, 2)) > 0.9) == sees).all() and ((got.amax((1, 2)) < 0.1) == ~sees).all(), j


def test_bounded_scores_and_the_one_more():
    """Equal keys of one score: n e^c of 1 + n e^c shares are theirs, c the bounded score."""
    n, heads, page, cap = 40, 3, 16, 5.0
    count = torch.arange(1, n + 1).float()[:, None]
    for s in (-30.0, -2.0, 0.0, 3.0, 30.0):
        cache, table = H.attention_case(8, heads, 1, page, F32, "cpu", n)
        cache[:, 1], cache[:, 0, ..., 0] = 1.0, s
        q = torch.zeros(n, heads, 8)
        q[..., 0] = 1.0
        e = math.exp(cap * math.tanh(s / cap))
        got = attend(q, cache, table, [[0, 0, n, 0]], 1, sink=torch.zeros(heads), softcap=cap)[..., 0]
        torch.testing.assert_close(got, (count * e / (1 + count * e)).expand(n, heads), rtol=1e-5, atol=1e-6)
    see = torch.ones(n, n, dtype=torch.bool).tril()
    torch.testing.assert_close(oracle.softmax_one_more(torch.full((n, n), 2.0), see).sum(-1), (count * math.exp(2) / (1 + count * math.exp(2)))[:, 0])


@pytest.mark.parametrize("scale", [0.0, -0.3, 2.0])
def test_scales_of_any_sign(scale):
    cfg = H.config([(H.attention(scale=scale), None), (H.attention(scale=-scale, size=5, kv_from=0), None)])
    w, t = H.weights(cfg), H.tokens(cfg, 20)
    assert H.error(H.run(H.engine(cfg, w), 0, t, [7, 2]), H.expected(cfg, w, t)) < H.TOLERANCE[F32]


def test_every_part_of_attention_is_audible():
    """Biases, the bound, the one more, the amplitude, the window and the source of keys all change the logits."""
    base = H.config([(H.attention(), None), (H.attention(scale=0.4), None), (H.attention(size=30, kv_from=0), None)])
    w, t = H.weights(base), H.tokens(base, 60)
    want = H.expected(base, w, t)
    assert H.error(H.run(H.engine(base, w), 0, t, [2, 3, 17]), want) < H.TOLERANCE[F32]
    for path, value in ((("softcap", ), 0.5), (("mask", "size"), 12), (("rot", "scaling", "factor"), 6.0), (("rot", "dims"), 10)):
        cfg = copy.deepcopy(base)
        for i in (0, 2):
            at = cfg["layers"][i]["mixer"]
            for key in path[:-1]:
                at = at[key]
            at[path[-1]] = value
        assert H.error(H.expected(cfg, w, t), want) > 1e-2, path
        assert H.error(H.run(H.engine(cfg, w), 0, t, [50]), H.expected(cfg, w, t)) < H.TOLERANCE[F32], path
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l2.mix.q.b"):
        other = dict(w, **{name: torch.zeros_like(w[name])})
        assert H.error(H.expected(base, other, t), want) > 1e-2, name
    src = copy.deepcopy(base)
    src["layers"][2]["mixer"]["kv_from"] = 1
    assert H.error(H.expected(src, w, t), want) > 1e-2
    assert H.error(H.run(H.engine(src, w), 0, t, [50]), H.expected(src, w, t)) < H.TOLERANCE[F32]


# ---- router and experts ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top", [(6, 2), (5, 1), (4, 4)])
def test_router_and_clamped_experts(E, top):
    T, W, limit = 40, 12, 0.7
    x, w = rnd(T, W), {"router": rnd(E, W, seed=1), "router.b": rnd(E, seed=2) * 2}
    for e in range(E):
        for i, n in enumerate(("gate", "up")):
            w[f"e{e}.{n}"] = rnd(8, W, seed=10 * e + i)
        w[f"e{e}.down"] = rnd(W, 8, seed=e)
    f = {"router": {"experts": E, "top": top}, "expert": {"limit": limit}}
    want = oracle.mixture(x.double(), oracle.cast(w), "", f).float()
    up = [torch.stack([w[f"e{e}.gate"], w[f"e{e}.up"]], 1).reshape(16, W) for e in range(E)]
    lw = LayerWeights(experts=[ExpertWeights(up[e], w[f"e{e}.down"]) for e in range(E)], w_router=torch.cat([w["router"], torch.zeros(2, W)]),
                      router_bias=w["router.b"])
    spec = FeedForwardSpec(ff=8, act="swiglu_clamped", limit=limit, experts=E, top=top, routing="chosen")
    ops = CpuOps()
    ops.chosen_route(x, lw, spec, None)
    torch.testing.assert_close(ops.routed_experts(x, None, lw, spec, 5, None, torch.zeros(T, W), None), want, rtol=1e-4, atol=1e-4)
    h = x @ w["e0.gate"].T
    assert (h > limit).any() and (h < -limit).any()            # (the gate is bounded above only)


# ---- models through the engine -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_and_portions(name):
    H.check_whole_and_portions(MODELS[name], F32, "cpu", n=150)


def test_residual_stream_of_a_layer_without_feed_forward_and_of_other_orders():
    for layers in ([(H.retention(), None)], [(H.attention(), H.moe())], [(H.attention(), None), (H.attention(size=3, kv_from=0), H.moe()), (H.retention(), H.moe())]):
        H.check_whole_and_portions(H.config(layers), F32, "cpu", n=120)


def test_mixed_batches_reuse_pages_and_slots():
    H.check_mixed_batches(H.MIXED, F32, "cpu")
    H.check_mixed_batches(H.config([(H.attention(), H.moe()), (H.attention(size=30, kv_from=0), None)]), F32, "cpu")


def test_long_decode():
    H.check_long_decode(H.MIXED, F32, "cpu")


def test_attention_without_a_window_or_a_bound():
    cfg = H.config([(H.attention(), H.moe()), (H.attention(), None)])
    del cfg["layers"][0]["mixer"]["mask"]
    cfg["layers"][1]["mixer"]["mask"] = None
    H.check_whole_and_portions(cfg, F32, "cpu", n=120)


def test_restore_from_hidden_states():
    H.check_restore(H.MIXED, F32, "cpu")
    assert not spec_of(H.MIXED).pages_hold_context
    assert not spec_of(H.config([(H.attention(), None), (H.attention(kv_from=0), None)])).pages_hold_context


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
        None, (2, 2, 64, 64), None, None, (2, 4, 64, 128), None, None, None]
    assert [None if s.ssm(i) is None else tuple(s.ssm(i).shape[1:]) for i in range(8)] == [
        (3, 32, 64), None, None, (2, 32, 64), None, None, (5, 48, 64), None]


def test_errors_name_what_is_wrong():
    for name, piece in (("l0.mix.g", None), ("l1.mix.g", "retention.g"), ("l0.mix.k.b", "attn.k_b"), ("l3.mix.q.b", "attn.q_b"), ("l0.mlp.router.b", "moe.router_b"),
                        ("l0.mlp.e1.gate", "moe.experts.1.gate"), ("l0.norm1", "norm1.g")):
        w = H.weights(H.ODD)
        if piece is None:
            H.engine(H.ODD, dict(w, **{name: w["l1.mix.g"]}))        # (a tensor nobody asked for does no harm)
            continue
        del w[name]
        with pytest.raises(ValueError, match=piece):
            H.engine(H.ODD, w)
    other = H.attention(rot=8, kv_from=0)
    for bad in ([(H.retention(), {"kind": "lattice"})], [({"type": "rings", "mixer": {}}, None)], [(H.attention(rot=22), None)], [(H.retention(rot=7), None)],
                [(H.attention(heads=5), None)], [(H.retention(heads=3, decay=[0.5]), None)], [(H.attention(), None), (other, None)],
                [(H.attention(kv_from=0), None)], [(H.retention(), None), (H.attention(kv_from=0), None)],
                [(H.attention(), None), (H.attention(kv_from=0), None), (H.attention(kv_from=1), None)], [(H.retention(), H.moe(experts=2, top=3))]):
        with pytest.raises(ValueError, match="relulix"):
            spec_of(H.config(bad))


def test_parameter_count_matches_the_checkpoint():
    for cfg in (H.MIXED, H.ODD, H.TILED, H.WIDE):
        assert spec_of(cfg).param_count() == sum(t.numel() for t in H.weights(cfg).values())


def test_specs_of_one_layer():
    m = RetentionSpec(3, 7, 33, [0.5] * 3)
    assert (m.width, m.vwidth, m.keys, m.inner, m.state) == (64, 48, 192, 144, 64)
    assert [RetentionSpec(1, d, 16, [0.5]).width for d in (64, 65, 128, 130)] == [64, 128, 128, 144]
    assert AttentionSpec(4, 2, 64, 64, 1.0, kv_from=0).cached_heads == 0 and AttentionSpec(4, 2, 64, 64, 1.0).cached_heads == 2


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
