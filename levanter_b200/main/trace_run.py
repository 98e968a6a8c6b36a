"""Feed given token ids through a model, step by step, and write logits: replays a recorded trace of a server's batches on the
generation engine, without sampling.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

``--model`` is a checkpoint directory (``config.json``, ``model.safetensors``); the model class follows from its config.  Steps are
read from standard input, one JSON object per line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` holds the next tokens of each request and, in ``want``, the places among them whose logits are asked for; the entries of
a step are one batch.  ``end`` lists requests that are finished after the step: their pages and slots are given back.  For a step that
wants logits, ``<out>/<step>.f32`` receives them in the order of the entries and of ``want`` as little-endian fp32
``[wanted, vocab]``.  After every step ``done <step>`` is printed.  The steps run on ``InferenceEngine.forward_packed``, the step
that generation prefills with."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Optional

import numpy as np
import torch

from levanter_b200.compat.hf_checkpoints import HFCheckpointConverter
from levanter_b200.inference.engine import InferenceEngine, InferenceEngineConfig
from levanter_b200.ops import lib

PAGE_SIZE = 16
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def load_for_serving(path: str, dtype: torch.dtype, device):
    conv = HFCheckpointConverter.from_hf(path)
    return conv.load_pretrained(ref=path, dtype=dtype, device=device, resize_vocab_to_match_tokenizer=False).eval()


class TraceRunner:
    """Requests by name on an engine.  The engine is sized by the first batch and rebuilt, while nothing is live, for a batch that
    needs more slots."""

    def __init__(self, model, dtype: torch.dtype, max_tokens: int):
        self.model, self.dtype, self.max_tokens = model, dtype, max(int(max_tokens), 1)
        self.engine: Optional[InferenceEngine] = None
        self.slots: Dict[str, int] = {}

    def _ensure_slots(self, new: int) -> None:
        need = len(self.slots) + new
        if self.engine is not None and need <= self.engine.config.max_seqs:
            return
        if self.slots:
            raise RuntimeError(f"a batch in progress cannot grow from {self.engine.config.max_seqs} slots to {need}")
        seqs = -(-need // 8) * 8
        per_seq = -(-self.max_tokens // PAGE_SIZE)
        cfg = InferenceEngineConfig(max_pages=per_seq + seqs, max_seqs=seqs, page_size=PAGE_SIZE, max_pages_per_seq=per_seq, compute_dtype=self.dtype)
        self.engine = InferenceEngine.from_model_with_config(self.model, None, cfg)

    def step(self, entries, end) -> Optional[np.ndarray]:
        self._ensure_slots(sum(e["id"] not in self.slots for e in entries))
        chunks, rows, at = [], [], 0
        for e in entries:
            if e["id"] not in self.slots:
                self.slots[e["id"]] = self.engine.open_sequence()
            chunks.append((self.slots[e["id"]], e["tokens"]))
            rows += [at + int(w) for w in e["want"]]
            at += len(e["tokens"])
        out = None
        if at:
            logits = self.engine.forward_packed(chunks, rows)
            out = None if logits is None else logits.float().cpu().numpy()
            if logits is not None and logits.is_cuda:
                lib.check_status()
        self.engine.close_sequences([self.slots.pop(i) for i in end])
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="checkpoint directory")
    ap.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16", help="weights, activations and cache; float32 is true 32-bit arithmetic")
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda", help="cpu runs the framework's PyTorch statements of the kernels (for tests)")
    a = ap.parse_args(argv)
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    if a.device == "cuda":
        if not lib.available():
            raise RuntimeError("trace_run needs a B200 (compute capability 10.x)")
        lib.use_serving_library()
    dtype = DTYPES[a.dtype]
    runner = TraceRunner(load_for_serving(a.model, dtype, torch.device(a.device)), dtype, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        got = runner.step(s["entries"], s.get("end", []))
        if got is not None:
            part = os.path.join(a.out, f".{s['step']}.part")
            got.astype("<f4").tofile(part)
            os.replace(part, os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
