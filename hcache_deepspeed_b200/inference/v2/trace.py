"""Replay of recorded requests through the ragged engine: given token ids in, logits out, nothing sampled.

Steps arrive on standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step are one batch (``InferenceEngineV2.put``): portions of prompts beside single decoded tokens. A request is
admitted by its first entry and flushed after the step that lists it in ``end``. The logits at the wanted places are written to
``<out>/<step>.f32`` (little-endian fp32, entries in order), then ``done <step>`` is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional

import torch

#: sequences live at once (batch entries, tracked sequences and recurrent-state slots)
MAX_LIVE = 4
DTYPES = {"bfloat16": torch.bfloat16, "float16": torch.float16, "float32": torch.float32}


class TraceRunner:

    def __init__(self, model_dir: str, dtype: torch.dtype, max_tokens: int, device: Optional[torch.device] = None) -> None:
        from .checkpoint import HuggingFaceCheckpointEngine
        from .config_v2 import RaggedInferenceEngineConfig
        from .engine_v2 import InferenceEngineV2
        from .model_implementations import MODEL_TYPE_TO_POLICY
        ckpt = HuggingFaceCheckpointEngine(model_dir)
        mt = ckpt.model_config.model_type
        if mt not in MODEL_TYPE_TO_POLICY:
            raise ValueError(f"Unsupported model type {mt}")
        policy = MODEL_TYPE_TO_POLICY[mt](ckpt.model_config, checkpoint_engine=ckpt, dtype=dtype, device=device)
        max_tokens = max(int(max_tokens), MAX_LIVE)
        self.engine = InferenceEngineV2(policy, RaggedInferenceEngineConfig(
            state_manager={"max_tracked_sequences": MAX_LIVE, "max_ragged_sequence_count": MAX_LIVE,
                           "max_ragged_batch_size": max_tokens, "max_context": max_tokens,
                           "memory_config": {"mode": "tokens", "size": max_tokens}, "max_state_slots": MAX_LIVE},
            hcache={"enabled": False, "capture": "off"}))
        self._uids: Dict[str, int] = {}
        self._next_uid = 0

    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        """Run one batch; returns the wanted logits (fp32, host) or None."""
        logits = None
        if entries:
            for e in entries:
                if e["id"] not in self._uids:
                    self._uids[e["id"]] = self._next_uid
                    self._next_uid += 1
            logits, _ = self.engine.put([self._uids[e["id"]] for e in entries],
                                        [torch.tensor(e["tokens"], dtype=torch.int32) for e in entries],
                                        logits_at=[e.get("want", []) for e in entries])
            logits = None if logits is None else logits.float().cpu()
        for name in end:
            self.engine.flush(self._uids.pop(name))
        return logits


def main(argv: Optional[List[str]] = None) -> int:
    p = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of requests and write the logits asked for.")
    p.add_argument("--model", required=True, help="folder with config.json and the weights")
    p.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    p.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    p.add_argument("--max-tokens", type=int, required=True,
                   help="tokens the live requests hold at most, each request's count rounded up to whole KV blocks")
    p.add_argument("--device", default="cuda", choices=["cuda", "cpu"], help="cpu: the fp32 restatement of the kernels (for tests)")
    a = p.parse_args(argv)
    if a.device == "cuda" and not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 2
    answers = os.fdopen(os.dup(1), "w")     # only answers go to standard output; build and log messages go to standard error
    os.dup2(2, 1)
    runner = TraceRunner(a.model, DTYPES[a.dtype], a.max_tokens, torch.device(a.device, 0) if a.device == "cuda" else torch.device("cpu"))
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = runner.step(s.get("entries", []), s.get("end", []))
        if logits is not None:
            logits.numpy().astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        answers.write(f"done {s['step']}\n")
        answers.flush()
    return 0
