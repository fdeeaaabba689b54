"""Nipolorn on the CPU back end: every mechanism against its plain restatement, then whole models through the engine."""
import os
import subprocess
import sys

import pytest
import torch

from hcache_deepspeed_b200.ops import reference as ref

from . import nipolorn_helper as H
from . import nipolorn_oracle as oracle

pytestmark = pytest.mark.timeout(600)
F32 = torch.float32
MODELS = {"mixed": H.MIXED, "odd": H.ODD, "wide": H.WIDE}


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed + sum(shape)))


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("size,keep", [(1, 0), (1, 3), (7, 2), (16, 0), (5, 40), (64, 1)])
def test_window_with_kept_tokens(size, keep):
    n, d = 50, 8
    q, k, v = rnd(n, 2, d), rnd(n, 1, d, seed=1), rnd(n, 1, d, seed=2)
    cache = torch.zeros(4, 2, 1, 16, d)
    table = torch.tensor([[2, 0, 3, 1]], dtype=torch.int32)
    slots = torch.tensor([int(table[0, i // 16]) * 16 + i % 16 for i in range(n)])
    ref.kv_append(cache, k, v, slots)
    see = oracle.visible(n, size, keep)
    for items in ([[0, 0, n, 0]], [[0, 0, 20, 0], [0, 20, 1, 20], [0, 21, n - 21, 21]]):
        got = ref.paged_attention(q, cache, table, torch.tensor(items, dtype=torch.int32), 2, 1, 0.4, window=size, keep_first=keep)
        s = (torch.einsum("qhd,kd->hqk", q, k[:, 0]) * 0.4).masked_fill(~see, float("-inf"))
        torch.testing.assert_close(got, torch.einsum("hqk,kd->qhd", s.softmax(-1), v[:, 0]), rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("taps", [1, 2, 4, 6])
def test_short_convolution_in_pieces(taps):
    n, c = 23, 5
    u, w, b = rnd(n, c), rnd(c, taps, seed=1), rnd(c, seed=2)
    want = oracle.silu(oracle.causal_conv(u.double(), w.double(), b.double())).float()
    for cuts in ([n], [1] * n, [2, 3, 2, 1, 15], [20, 3]):
        ring, out, at = torch.full((taps, c), 9.0), [], 0     # whatever a slot held before must not matter
        for k in cuts:
            out.append(ref.short_conv(u[at:at + k], ring, w.t().contiguous(), b, at))
            at += k
        torch.testing.assert_close(torch.cat(out), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("heads,groups", [(4, 1), (6, 3), (5, 5)])
def test_recurrence_in_pieces(heads, groups):
    n, P, N = 30, 6, 7
    x, B, C = rnd(n, heads, P), rnd(n, groups, N, seed=1), rnd(n, groups, N, seed=2)
    dt, A, D = torch.nn.functional.softplus(rnd(n, heads, seed=3)), rnd(heads, seed=4), rnd(heads, seed=5)
    want, S = oracle.recurrence(*(t.double() for t in (x, B, C, dt, A, D)))
    state, out = torch.zeros(heads, P, N), []
    for a, b in ((0, 11), (11, 12), (12, n)):
        out.append(ref.selective_scan(x[a:b], B[a:b], C[a:b], dt[a:b], -torch.exp(A), D, state))
    torch.testing.assert_close(torch.cat(out), want.float(), rtol=1e-4, atol=1e-4)
    torch.testing.assert_close(state, S.float().transpose(1, 2), rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("groups", [1, 3, 4])
def test_gated_group_norm(groups):
    y, z, w = rnd(9, 12) * 3, rnd(9, 12, seed=1), rnd(12, seed=2)
    want = oracle.gated_group_norm(y.double(), z.double(), w.double(), groups, 1e-5).float()
    torch.testing.assert_close(ref.gated_norm(y, z, w, groups, 1e-5), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(ref.gated_norm(y, z, w, groups, 1e-5, 0.25), want * 0.25, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("factor", [1.0, 0.3, -2.0])
def test_norms_on_both_sides(factor):
    x, d, wb, wn = rnd(6, 20), rnd(6, 20, seed=1) * 1e-2, rnd(20, seed=2), rnd(20, seed=3)
    eps = 1e-4      # large enough to show where it enters
    pad = lambda t: torch.nn.functional.pad(t, (0, 4))  # noqa: E731
    s, o = ref.norm_residual(pad(x), pad(1 + wn), pad(d), factor, pad(1 + wb), 20, eps)
    want = x + oracle.norm(factor * d, wb, eps)
    torch.testing.assert_close(s[:, :20], want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(o[:, :20], oracle.norm(want, wn, eps), rtol=1e-5, atol=1e-5)
    assert not s[:, 20:].any() and not o[:, 20:].any()


def test_clamped_gate():
    x = rnd(40, 16) * 2
    w = {"gate": rnd(24, 16), "up": rnd(24, 16, seed=1), "down": rnd(16, 24, seed=2)}
    from hcache_deepspeed_b200.models.weights import interleave_gate_up
    h = ref.gemm(x, interleave_gate_up(w["gate"], w["up"]), act=5, gated=True, limit=1.1)
    torch.testing.assert_close(h @ w["down"].t(), oracle.clamped_mlp(x, w, "", 1.1), rtol=1e-4, atol=1e-4)


def test_scale_of_zero_or_less_and_single_sided_mixers():
    for change in ({"scale": -0.3}, {"scale": 0.0}, {"left": 0.0}, {"right": 0.0}, {"left": -0.7}):
        cfg = H.config([(H.mixer(**change), H.dense())])
        w, t = H.weights(cfg), H.tokens(cfg, 40)
        assert H.error(H.run(H.engine(cfg, w), 0, t, [30]), H.expected(cfg, w, t)) < H.TOLERANCE[F32], change


# ---- models through the engine -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(MODELS))
def test_whole_and_portions(name):
    H.check_whole_and_portions(MODELS[name], F32, "cpu", n=150)


def test_mixed_batches_reuse_pages_and_slots():
    H.check_mixed_batches(H.MIXED, F32, "cpu")


def test_restore_from_hidden_states():
    H.check_restore(H.MIXED, F32, "cpu")


def test_sessions_are_saved_and_restored_without_pages():
    """Multi-turn sessions: the planner keeps to hidden states (and recomputation), which bring the recurrent state back."""
    from hcache_deepspeed_b200.hcache import HCacheSessionManager
    cfg = H.MIXED
    w, t = H.weights(cfg), H.tokens(cfg, 90)
    eng = H.engine(cfg, w, enabled=True, capture="sync")
    m = HCacheSessionManager(eng)
    m.prefill(3, t[:50])
    kinds = m.end_turn(3).kinds
    assert "kv" not in kinds
    eng.put([8], [H.tokens(cfg, 70, seed=4)])        # another sequence takes over pages and slot meanwhile
    eng.flush(8)
    assert H.error(m.prefill(3, t[50:]).float(), H.expected(cfg, w, t)[-1:]) < H.TOLERANCE[F32]
    with pytest.raises(ValueError, match="recurrent"):
        eng.restore_session(4, t[:50], kv=None, kv_layers=[0, 1, 2, 3])


def test_greedy_generation(tmp_path):
    H.check_greedy(H.MIXED, F32, False, tmp_path / "m")


def test_admission_counts_state_slots_and_pages():
    from hcache_deepspeed_b200.inference.v2 import SchedulingError, SchedulingResult
    cfg = H.ODD
    eng = H.engine(cfg, H.weights(cfg), tokens=192, live=4, slots=2)
    t = H.tokens(cfg, 60)
    eng.put([1, 2], [t[:3], t[:60]])
    assert eng.can_schedule([3], [1]) == SchedulingResult.EngineSequenceLimitExceeded and eng.query(3, 1, 1) == (0, 0)
    with pytest.raises(SchedulingError):
        eng.put([3], [t[:1]])
    assert eng.can_schedule([2], [70]) == SchedulingResult.KVCacheLimitExceeded
    eng.flush(1)
    assert eng.can_schedule([3], [1]) == SchedulingResult.Success
    with pytest.raises(ValueError):
        eng.put([3], [t[:2]], logits_at=[[2]])


def test_serialize_round_trip(tmp_path):
    from hcache_deepspeed_b200.inference.v2 import build_hf_engine
    cfg = H.MIXED
    w, t = H.weights(cfg), H.tokens(cfg, 20)
    eng = H.engine(cfg, w)
    want = H.run(eng, 0, t)
    eng.serialize(str(tmp_path / "ser"))
    again = build_hf_engine(str(tmp_path / "ser"), eng.config)
    torch.testing.assert_close(H.run(again, 0, t), want)


def test_missing_tensor_and_unknown_kind_are_errors():
    cfg = H.ODD
    w = H.weights(cfg)
    del w["l1.mlp.table"]
    with pytest.raises(ValueError, match="moe.table"):
        H.engine(cfg, w)
    bad = H.config([(H.mixer(), {"kind": "lattice", "ff": 8})])
    with pytest.raises(ValueError, match="lattice"):
        H.engine(bad, H.weights(H.config([(H.mixer(), None)])))


def test_trace_runner_process(tmp_path):
    """bin/trace_run: answers step by step, in order, with pages and slots used again."""
    import json
    import numpy as np
    cfg = H.ODD
    w = H.weights(cfg)
    folder = H.save(tmp_path / "m", cfg, w)
    t = {k: H.tokens(cfg, n, seed=n) for k, n in (("a", 30), ("b", 9), ("c", 12))}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t["a"][:29].tolist(), "want": [28, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": t["b"].tolist(), "want": []}, {"id": "a", "tokens": t["a"][29:].tolist(), "want": [0]}],
              "end": ["a", "b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": t["c"].tolist(), "want": []}], "end": ["c"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "128", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       stdout=subprocess.PIPE, stderr=subprocess.PIPE, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n") == ["done 0", "done 1", "done 2", ""]
    want = H.expected(cfg, w, t["a"])
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4")).reshape(-1, cfg["vocab"])  # noqa: E731
    assert H.error(read(0), want[[28, 3]]) < 1e-4 and H.error(read(1), want[[29]]) < 1e-4
    assert not (tmp_path / "2.f32").exists()
