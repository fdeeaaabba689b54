"""Dedelorn on the CPU back end: every mechanism against its plain restatement, then whole models through the engine."""
import os
import subprocess
import sys

import pytest
import torch

from hcache_deepspeed_b200.models.arch import DeltaSpec, FeedForwardSpec, LatentAttentionSpec
from hcache_deepspeed_b200.models.weights import ExpertWeights, LayerWeights
from hcache_deepspeed_b200.ops import reference as ref
from hcache_deepspeed_b200.ops.backend import CpuOps

from . import dedelorn_helper as H
from . import dedelorn_oracle as oracle

pytestmark = pytest.mark.timeout(600)
F32 = torch.float32
MODELS = {"mixed": H.MIXED, "odd": H.ODD, "wide": H.WIDE}


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed + sum(shape)))


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("heads,groups,N,P", [(4, 1, 6, 7), (6, 3, 5, 4), (5, 5, 9, 3)])
def test_delta_rule_in_pieces(heads, groups, N, P):
    n = 30
    q, k, v = rnd(n, groups, N), rnd(n, groups, N, seed=1), rnd(n, heads, P, seed=2)
    g, beta = torch.sigmoid(rnd(n, heads, seed=3) + 2), torch.sigmoid(rnd(n, heads, seed=4))
    of = torch.arange(heads) // (heads // groups)
    want, S = oracle.delta_recurrence((oracle.unit(q.double()) * N**-0.5)[:, of], oracle.unit(k.double())[:, of], v.double(), g.double(), beta.double())
    state, out = torch.zeros(heads, P, N), []
    for a, b in ((0, 11), (11, 12), (12, n)):
        out.append(ref.delta_scan(q[a:b], k[a:b], v[a:b], g[a:b], beta[a:b], state))
    torch.testing.assert_close(torch.cat(out), want.float(), rtol=1e-4, atol=1e-5)
    torch.testing.assert_close(state, S.float().transpose(1, 2), rtol=1e-4, atol=1e-5)


def test_delta_rule_small_keys_feel_the_unit_epsilon():
    """Keys and queries of about the size of the epsilon's root are no unit vectors."""
    n, N, P = 9, 4, 3
    q, k, v = rnd(n, 1, N) * 1e-3, rnd(n, 1, N, seed=1) * 1e-3, rnd(n, 1, P, seed=2)
    g, beta = torch.full((n, 1), 0.9), torch.full((n, 1), 0.8)
    want, _ = oracle.delta_recurrence(oracle.unit(q.double()) * N**-0.5, oracle.unit(k.double()), v.double(), g.double(), beta.double())
    torch.testing.assert_close(ref.delta_scan(q, k, v, g, beta, torch.zeros(1, P, N)), want.float(), rtol=1e-4, atol=1e-6)


def test_norm_in_front_of_the_gate():
    y, z, w = rnd(9, 12) * 0.01, rnd(9, 12, seed=1), rnd(4, seed=2)
    want = oracle.norm_then_gate(y.double().reshape(9, 3, 4), z.double(), w.double(), 1e-4).float()
    torch.testing.assert_close(ref.gated_norm(y, z, w.repeat(3), 3, 1e-4, gate_after=True), want, rtol=1e-5, atol=1e-6)


def test_delta_mixer_end_to_end():
    """Projections, convolutions, decay, step, recurrence, norm and gate of one mixer, cut into portions, against the restatement."""
    cfg = H.config([(H.delta(heads=6, kv=2, dim=9, vdim=5, conv=4), None)])
    w, t = H.weights(cfg), H.tokens(cfg, 33)
    assert H.error(H.run(H.engine(cfg, w), 0, t, [2, 3, 1, 17]), H.expected(cfg, w, t)) < H.TOLERANCE[F32]


@pytest.mark.parametrize("dims,base", [(2, 10.0), (10, 300.0), (32, 2e4)])
def test_rotation_of_adjacent_pairs(dims, base):
    from hcache_deepspeed_b200.models.hybrid import rotation_frequencies
    x = rnd(400, 3, dims)
    want = oracle.rotate_pairs(x.double(), base).float()
    torch.testing.assert_close(ref.rotate_pairs(x, torch.arange(400), rotation_frequencies(dims, base)), want, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("window", [0, 1, 2, 7, 16, 64])
def test_latent_attention_window_edges(window):
    """One cached row of huge score at a time: exactly the queries whose window holds it return its latent."""
    n, heads, rank, rot, page = 50, 2, 5, 4, 16
    table = torch.tensor([[2, 0, 3, 1]], dtype=torch.int32)
    q = torch.zeros(n, heads, rank + rot)
    q[..., 0] = 50.0
    i = torch.arange(n)
    for j in (0, 1, 15, 16, 31, 40, n - 1):
        pages = torch.zeros(4, 1, 1, page, 16)
        pages[int(table[0, j // page]), 0, 0, j % page, 0] = 1.0
        for items in ([[0, 0, n, 0]], [[0, 0, 20, 0], [0, 20, 1, 20], [0, 21, n - 21, 21]]):
            got = ref.paged_latent_attention(q, pages, table, torch.tensor(items, dtype=torch.int32), rank, 1.0, window)
            sees = (i >= j) & ((i - j < window) if window else True)
            assert ((got[..., 0].amin(1) > 0.9) == sees).all() and ((got[..., 0].amax(1) < 0.1) == ~sees).all(), j


def test_router_chooses_by_corrected_and_weighs_by_plain_scores():
    T, W, E, top = 40, 12, 6, 2
    x, w = rnd(T, W), {"router": rnd(E, W, seed=1), "correction": torch.tensor([0.0, 2.0, 0.0, -3.0, 0.4, 0.0])}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = rnd(8, W, seed=e), rnd(W, 8, seed=e)
    want = oracle.mixture(x.double(), oracle.cast(w), "", {"top": top, "scale": 1.6}).float()
    lw = LayerWeights(experts=[ExpertWeights(w[f"e{e}.up"], w[f"e{e}.down"]) for e in range(E)], router_bias=w["correction"],
                      w_router=torch.cat([w["router"], torch.zeros(2, W)]))
    f = FeedForwardSpec(ff=8, act="gelu", experts=E, top=top, routing="softmax", gated=False, router_scale=1.6)
    ops = CpuOps()
    ops.softmax_route(x, lw, f, None)
    assert (ops._picked == 1).any(-1).all() and not (ops._picked == 3).any()
    base = rnd(T, W, seed=9)
    torch.testing.assert_close(ops.routed_experts(x, None, lw, f, 1, base, torch.zeros(T, W), None), base + want, rtol=1e-4, atol=1e-4)
    acc = base.clone()
    torch.testing.assert_close(ops.routed_experts(x, None, lw, f, 1, acc, acc, None), base + want, rtol=1e-4, atol=1e-4)


def test_embedding_norm_and_plain_addition():
    ids, w, g = torch.tensor([3, 0, 3, 5], dtype=torch.int32), rnd(7, 20) * 1e-2, rnd(24, seed=2)
    pad = torch.nn.functional.pad(w, (0, 4))
    got = CpuOps().embed_f32(ids, pad, torch.empty(4, 24), gamma=g, cols=20, eps=1e-4)
    torch.testing.assert_close(got[:, :20], oracle.rms(w[ids.long()], 1e-4) * g[:20], rtol=1e-5, atol=1e-6)
    x, d = rnd(6, 20), rnd(6, 20, seed=1)
    s, o = ref.norm_residual(x, g[:20], d, 0.5, None, 20, 1e-4)
    torch.testing.assert_close(s, x + 0.5 * d)
    torch.testing.assert_close(o, oracle.rms(x + 0.5 * d, 1e-4) * g[:20], rtol=1e-5, atol=1e-6)


def test_two_activations():
    z = torch.linspace(-6, 6, 301)
    torch.testing.assert_close(ref.apply_act(z, 4), oracle.gelu_tanh(z), rtol=1e-5, atol=1e-6)
    torch.testing.assert_close(ref.apply_act(z, 1), oracle.gelu_erf(z), rtol=1e-5, atol=1e-6)
    assert (oracle.gelu_tanh(z) - oracle.gelu_erf(z)).abs().max() > 1e-4


# ---- models through the engine -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_and_portions(name):
    H.check_whole_and_portions(MODELS[name], F32, "cpu", n=150)


def test_mixed_batches_reuse_pages_and_slots():
    H.check_mixed_batches(H.MIXED, F32, "cpu")


def test_a_stack_without_recurrent_layers():
    H.check_whole_and_portions(H.config([(H.latent(), H.moe()), (H.latent(size=None, kv_from=0), H.dense())]), F32, "cpu", n=120)


def test_restore_from_hidden_states():
    H.check_restore(H.MIXED, F32, "cpu")


def test_sessions_are_saved_and_restored_without_pages():
    from hcache_deepspeed_b200.hcache import HCacheSessionManager
    cfg = H.MIXED
    w, t = H.weights(cfg), H.tokens(cfg, 90)
    eng = H.engine(cfg, w, enabled=True, capture="sync")
    m = HCacheSessionManager(eng)
    m.prefill(3, t[:50])
    assert "kv" not in m.end_turn(3).kinds
    eng.put([8], [H.tokens(cfg, 70, seed=4)])        # another sequence takes over pages and slot meanwhile
    eng.flush(8)
    assert H.error(m.prefill(3, t[50:]).float(), H.expected(cfg, w, t)[-1:]) < H.TOLERANCE[F32]
    with pytest.raises(ValueError, match="latents"):
        eng.restore_session(4, t[:50], kv=None, kv_layers=list(range(8)))


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


def test_only_owning_layers_hold_pages():
    eng = H.engine(H.MIXED, H.weights(H.MIXED), tokens=128)
    c = eng.state_manager.kv_cache
    assert [None if c.get_cache(i) is None else tuple(c.get_cache(i).shape[1:]) for i in range(8)] == [
        (1, 1, 64, 64), None, (1, 1, 64, 64), None, None, None, None, None]


def test_errors_name_what_is_wrong():
    from hcache_deepspeed_b200.models.arch import arch_from_hf_config
    w = H.weights(H.ODD)
    del w["l1.mlp.correction"]
    with pytest.raises(ValueError, match="moe.correction"):
        H.engine(H.ODD, w)
    arch = lambda *layers: arch_from_hf_config(dict(H.config(list(layers)), model_type="dedelorn"))  # noqa: E731
    for bad in ([(H.latent(), {"kind": "lattice", "ff": 8})], [({"type": "rings", "mixer": {}}, None)], [(H.latent(kv_from=0), None)],
                [(H.delta(), None), (H.latent(kv_from=0), None)], [(H.latent(), None), (H.latent(rank=40, kv_from=0), None)],
                [(H.latent(), None), (H.latent(kv_from=0), None), (H.latent(kv_from=1), None)]):
        with pytest.raises(ValueError, match="dedelorn"):
            arch(*bad)


def test_parameter_count_matches_the_checkpoint():
    from hcache_deepspeed_b200.models.arch import arch_from_hf_config
    for cfg in (H.MIXED, H.ODD, H.TILED):
        spec = arch_from_hf_config(dict(cfg, model_type="dedelorn"))
        assert spec.param_count() + cfg["width"] == sum(t.numel() for t in H.weights(cfg).values())    # (+ the embedding norm)


def test_specs_of_one_layer():
    c, d = LatentAttentionSpec(4, 50, 20, 30, 100, 0.1), DeltaSpec(6, 2, 10, 5)
    assert (c.page_width, c.head_width) == (128, 128) and (d.inner, d.conv_dim, d.in_dim) == (30, 70, 112)


def test_trace_runner_process(tmp_path):
    import json

    import numpy as np
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
