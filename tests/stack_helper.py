"""Scenarios for models of unlike layers, shared by the designs' tests and by both back ends. A design registers how to make random
checkpoint tensors for a config and its plain oracle (:data:`DESIGNS`)."""
import json
import os

import torch

#: config "architecture" -> (weights(cfg, seed, dtype, settled), oracle module)
DESIGNS = {}


def weights(cfg, seed=0, dtype=torch.bfloat16, run_in=torch.float32):
    """Random checkpoint tensors. For a run in 16 bits (``run_in``) no router's choice may be a close call, which rounding decides."""
    return DESIGNS[cfg["architecture"]][0](cfg, seed, dtype, run_in != torch.float32)


def save(folder, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: t.contiguous() for k, t in w.items()}, os.path.join(folder, "model.safetensors"))
    return str(folder)


def engine(cfg, w, dtype=torch.float32, device="cpu", tokens=1024, live=4, batch=None, slots=None, **hcache):
    """Ragged engine over in-memory weights with a cache pool of exactly ``tokens`` tokens."""
    from hcache_deepspeed_b200.inference.v2 import InferenceEngineV2, RaggedInferenceEngineConfig
    from hcache_deepspeed_b200.inference.v2.checkpoint import NativeConfig
    from hcache_deepspeed_b200.inference.v2.model_implementations import MODEL_TYPE_TO_POLICY

    class Source:
        def parameters(self):
            return iter(w.items())

    pol = MODEL_TYPE_TO_POLICY[cfg["architecture"].lower()](NativeConfig(cfg), checkpoint_engine=Source(), dtype=dtype, device=torch.device(device))
    return InferenceEngineV2(pol, RaggedInferenceEngineConfig(
        state_manager={"max_tracked_sequences": live, "max_ragged_sequence_count": live, "max_ragged_batch_size": batch or tokens,
                       "max_context": tokens, "memory_config": {"mode": "tokens", "size": tokens}, "max_state_slots": slots or live},
        hcache=hcache or {"enabled": False, "capture": "off"}))


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n, ), generator=torch.Generator().manual_seed(seed))


def run(eng, uid, toks, portions=None):
    """All logits of one request fed in the given portions (None: at once); the rest token by token."""
    out, at = [], 0
    for n in (portions if portions is not None else [len(toks)]):
        n = min(n, len(toks) - at)
        if n == 0:
            break
        out.append(eng.put([uid], [toks[at:at + n]], logits_at=[list(range(n))])[0].float().cpu().clone())   # (the engine reuses its logits buffer)
        at += n
    for i in range(at, len(toks)):
        out.append(eng.put([uid], [toks[i:i + 1]])[0].float().cpu().clone())
    return torch.cat(out)


def expected(cfg, w, toks):
    oracle = DESIGNS[cfg["architecture"]][1]
    return oracle.logits(cfg, oracle.cast(w), toks).float()


def error(got, want):
    """Largest row difference (mean removed, root mean square) relative to the spread of the expected logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt().max() / (want.double() - want.double().mean(-1, keepdim=True)).pow(2).mean().sqrt()).item()


#: what rounding alone leaves at the worst position: fp32 arithmetic, or 16-bit operands (whose rounding a norm can magnify where
#: a sublayer's output is small); the fp32 runs are the sharp test of the bookkeeping
TOLERANCE = {torch.float32: 1e-4, torch.bfloat16: 0.15, torch.float16: 3e-2}


# ---- scenarios shared by the CPU and GPU tests ---------------------------------------------------------------------
def check_whole_and_portions(cfg, dtype, device, n=190, tol=None):
    """One request: at once, in portions of several sizes (down to two tokens), and token by token, against the oracle."""
    w, t = weights(cfg, run_in=dtype), tokens(cfg, n)
    want, tol = expected(cfg, w, t), tol or TOLERANCE[dtype]
    eng = engine(cfg, w, dtype, device, tokens=512)
    for uid, portions in enumerate([None, [n - 40], [2, 3, 2, 64, 1, 37, 65], [128, 2, 30], [130, 7]]):
        assert error(run(eng, uid, t, portions), want) < tol, portions
        eng.flush(uid)
    short = tokens(cfg, 9, seed=5)
    assert error(run(eng, 77, short, []), expected(cfg, w, short)) < tol     # decoding from the very first token


def check_mixed_batches(cfg, dtype, device, tol=None):
    """Unequal requests in one batch: portions beside single tokens, a request left out of steps, pages and state slots freed
    and used again by others; every logit as if the request were alone."""
    w, tol = weights(cfg, seed=3, run_in=dtype), tol or TOLERANCE[dtype]
    eng = engine(cfg, w, dtype, device, tokens=512, live=3)
    lengths = {"a": 150, "b": 37, "c": 90, "d": 64, "e": 5, "f": 140, "g": 1}
    toks = {k: tokens(cfg, n, seed=ord(k)) for k, n in lengths.items()}
    want = {k: expected(cfg, w, t) for k, t in toks.items()}
    uid = {k: i for i, k in enumerate(toks)}
    at = {k: 0 for k in toks}
    plan = [[("a", 70), ("b", 2)], [("a", 1), ("b", 1), ("c", 64)], [("b", 34), ("c", 2)], [("a", 3), ("c", 1), ("d", 33)], [("d", 1), ("a", 1)],
            [("a", 75), ("c", 23), ("d", 30)], [("e", 2), ("f", 129)], [("e", 1), ("f", 1), ("g", 1)], [("f", 10), ("e", 2)]]
    for step in plan:
        wants = [list(range(n)) for _, n in step]
        got = eng.put([uid[k] for k, _ in step], [toks[k][at[k]:at[k] + n] for k, n in step], logits_at=wants)[0].float().cpu()
        row = 0
        for k, n in step:
            assert error(got[row:row + n], want[k][at[k]:at[k] + n]) < tol * 1.5, (k, at[k])
            row, at[k] = row + n, at[k] + n
        for k, _ in step:
            if at[k] == len(toks[k]):
                eng.flush(uid[k])
    states = eng.state_manager.recurrent_states
    assert at == lengths and int(eng.free_blocks[0]) == 512 // 64 and (states is None or states.free_slots == 3)


def check_long_decode(cfg, dtype, device, n=330, tol=None):
    w, t = weights(cfg, seed=4, run_in=dtype), tokens(cfg, n, seed=6)
    eng = engine(cfg, w, dtype, device, tokens=384)
    assert error(run(eng, 0, t, [7]), expected(cfg, w, t)) < (tol or TOLERANCE[dtype])


def check_restore(cfg, dtype, device, tol=None):
    """Hidden states saved while a prompt runs rebuild pages AND recurrent state of another sequence."""
    w, t = weights(cfg, seed=7, run_in=dtype), tokens(cfg, 150, seed=8)
    eng = engine(cfg, w, dtype, device, tokens=512, enabled=True, capture="sync")
    first, lat = eng.put([0], [t[:101]])
    _, lat2 = eng.put([0], [t[101:103]])
    saved = torch.cat([lat[0], lat2[0]], dim=1)
    eng.flush(0)
    for defer in (False, True):
        eng.put([5], [tokens(cfg, 80, seed=9)], capture_latents=False)       # leaves its traces in pages and slots
        eng.flush(5)
        eng.restore_kv([1], [t[:103]], [saved], defer=defer)
        got = eng.put([1], [t[103:]], capture_latents=False, logits_at=[list(range(47))])[0].float().cpu()
        assert error(got, expected(cfg, w, t)[103:]) < (tol or TOLERANCE[dtype])
        eng.flush(1)


def check_greedy(cfg, dtype, device_is_gpu, folder, n_new=24):
    """Greedy generation through init_inference: every chosen token is the oracle's best (or as good, within rounding)."""
    import hcache_deepspeed_b200 as hds
    w = weights(cfg, seed=10, run_in=dtype)
    path = save(folder, cfg, w)
    eng = hds.init_inference(path, dtype=dtype, hcache={"max_context": 512, "max_batch_tokens": 512, "max_sessions": 8,
                                                        "kv_memory_bytes": 64 << 20})
    prompts = torch.stack([tokens(cfg, 40, seed=11), tokens(cfg, 40, seed=12)])
    mask = torch.ones_like(prompts)
    mask[1, :13] = 0                                                         # rows of unequal length
    out = eng.generate(prompts, attention_mask=mask, max_new_tokens=n_new, do_sample=False)
    assert out.shape == (2, 40 + n_new)
    for b in range(2):
        seq = torch.cat([out[b, :40][mask[b].bool()], out[b, 40:]])
        lg = expected(cfg, w, seq)
        start = int(mask[b].sum())
        rows = lg[start - 1:len(seq) - 1]
        slack = rows.max(-1).values - rows.gather(-1, seq[start:, None]).squeeze(-1)
        assert float(slack.max()) <= TOLERANCE[dtype] * 2 * float(lg.std()), (b, slack)


def attention_case(d, n_q, n_kv, page, dtype, device, n_keys=700, seed=0):
    """Pages in shuffled order holding zero keys and zero values except where a test plants one."""
    g = torch.Generator().manual_seed(seed)
    blocks = -(-n_keys // page)
    cache = torch.zeros(blocks + 3, 2, n_kv, page, d, dtype=dtype)
    table = torch.randperm(blocks + 3, generator=g)[:blocks].to(torch.int32)
    return cache, table
