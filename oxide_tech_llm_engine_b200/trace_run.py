"""Trace replay: feeds given token ids through a model step by step and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Each input line is one step,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

whose entries run as one batch through `LLMEngine.feed` (the engine's own plan, step function, paged
cache, state slots and kernels). Logits of the wanted places go to OUT/<step>.f32 as little-endian
fp32 [wanted, vocab]; after every step the line "done <step>" is printed. Requests in "end" give
their blocks and slots back. The pool holds N tokens, and four requests may be live.

Exit codes: 0 at the end of the input, 2 for bad arguments, 3 when the model cannot run in the dtype.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Optional

import numpy as np

MAX_LIVE = 4


def build_engine(model: str, dtype: str, max_tokens: int, max_live: int = MAX_LIVE, backend: str = "cuda"):
    from .config import EngineConfig
    from .engine.engine import LLMEngine
    from .models.weights import open_weights

    src = open_weights(model)
    blocks = (max_tokens + 15) // 16
    cfg = EngineConfig(model=model, backend=backend, dtype=dtype, max_num_seqs=max_live, num_kv_blocks=blocks,
                       ctx_size=blocks * 16, max_num_batched_tokens=blocks * 16, enable_radix=False, speculative="off",
                       graph_buckets=tuple(b for b in (1, 2, 4, 8, 16) if b <= max_live))
    return LLMEngine(cfg, weights=src)


class Replay:
    """Applies steps to an engine; request names map to engine ids for as long as they live."""

    def __init__(self, engine):
        self.engine = engine
        self.ids: dict = {}
        self._next = 0

    def step(self, line: dict) -> np.ndarray:
        entries, index, base = [], [], 0
        for e in line["entries"]:
            if not e["tokens"]:
                continue
            name = e["id"]
            if name not in self.ids:
                self.ids[name] = self._next
                self._next += 1
            want, inverse = np.unique(np.asarray(e["want"], dtype=np.int64), return_inverse=True)
            entries.append((self.ids[name], e["tokens"], want.tolist()))
            index += (base + inverse.reshape(-1)).tolist()
            base += want.size
        out = self.engine.feed(entries) if entries else np.zeros((0, self.engine.model_cfg.vocab_size), np.float32)
        for name in line.get("end", ()):
            if name in self.ids:
                self.engine.cancel(self.ids.pop(name))
        return out[index] if index else out[:0]


def main(argv: Optional[list] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay given tokens through the engine and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that the live requests hold at most")
    args = ap.parse_args(argv)
    from .errors import ConfigError
    from .models.weights import open_weights

    if args.dtype == "float32" and not open_weights(args.model).cfg.layers:
        print("float32: this model runs with bf16 activations only", file=sys.stderr)
        return 3
    import torch

    if not torch.cuda.is_available():
        raise ConfigError("trace_run needs a CUDA device")
    os.makedirs(args.out, exist_ok=True)
    replay = Replay(build_engine(args.model, args.dtype, args.max_tokens))
    for text in sys.stdin:
        if not text.strip():
            continue
        line = json.loads(text)
        logits = replay.step(line)
        if logits.shape[0]:
            np.ascontiguousarray(logits, dtype="<f4").tofile(os.path.join(args.out, f"{line['step']}.f32"))
        print(f"done {line['step']}", flush=True)
    replay.engine.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
