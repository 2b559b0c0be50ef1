"""Step-driven serving of given token ids: every step is one batch of portions of live requests (prompt portions beside
single tokens), run by the model runner from the caches and states that earlier steps left; nothing is sampled.

`BatchSession` is the API; `main` replays a trace from standard input (one JSON object a line):

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

and writes the wanted logits of a step as little-endian fp32 rows to <out>/<step>.f32, in the order of the entries and of
their `want` places."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Sequence, Tuple

import torch

from ..cache.kv import KvManager
from ..config import EngineConfig, ModelConfig
from ..models.model import Model
from ..models.plan import make_plan
from .engine import compute_dtype


class BatchSession:
    def __init__(self, cfg: ModelConfig, W: dict, ecfg: EngineConfig = None, device="cuda", max_seqs: int = 4, kv_tokens: int = 4096):
        """`kv_tokens`: the cache pool, shared by the live requests; `max_seqs`: state slots."""
        ecfg = ecfg or EngineConfig()
        self.cfg = cfg
        self.model = Model(cfg, W, device=device, dtype=compute_dtype(ecfg, device), n_slots=max_seqs, kv_tokens=kv_tokens)
        self.kv = KvManager(self.model, granule=64)
        self.free: List[int] = list(range(max_seqs))
        self.slots: Dict[str, int] = {}

    def _room(self, rid: str, n: int) -> int:
        """The request's slot with cache room for `n` more tokens (a request is admitted at its first tokens)."""
        m = self.model
        slot = self.slots.get(rid)
        if slot is None:
            if not self.free:
                raise RuntimeError("no free state slot")
            slot = self.free.pop(0)
            if not self.kv.assign(slot, n):
                self.free.insert(0, slot)
                raise RuntimeError("the KV pool is exhausted")
            self.slots[rid] = slot
            m.reset_slot(slot)
        elif m.seqs[slot].length + n > m.seqs[slot].kv_cap and not self.kv.grow(slot, m.seqs[slot].length + n):
            raise RuntimeError("the KV pool is exhausted")
        return slot

    @torch.no_grad()
    def step(self, entries: Sequence[Tuple[str, Sequence[int], Sequence[int]]]) -> torch.Tensor:
        """entries: (request id, its next tokens, places whose logits are wanted).  One forward over all of them; returns the
        logits [wanted, vocab] (fp32, on the device) in the order of the entries and places."""
        m = self.model
        items, rows, r = [], [], 0
        for rid, toks, want in entries:
            if not toks:
                continue
            for t in toks:
                if not 0 <= t < self.cfg.vocab:
                    raise ValueError(f"token id {t} is outside the vocabulary of {self.cfg.vocab} entries")
            slot = self._room(rid, len(toks))
            items.append((slot, list(toks), m.seqs[slot].length))
            rows += [r + w for w in want]
            r += len(toks)
        if not items:
            return torch.empty(0, self.cfg.vocab, device=m.device)
        plan = make_plan(items, device=m.device)
        plan.logit_rows = torch.tensor(rows, dtype=torch.long, device=m.device)
        plan.gather_logit_rows = True
        return m.forward(plan)

    def end(self, rid: str):
        """The request is finished: its pages and its slot go back."""
        slot = self.slots.pop(rid)
        self.kv.release(slot)
        self.free.append(slot)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids step by step and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time")
    ap.add_argument("--max-seqs", type=int, default=4, help="state slots (live requests)")
    a = ap.parse_args(argv)
    if not torch.cuda.is_available():
        print("trace_run needs a CUDA device", file=sys.stderr)
        return 1
    from ..models.checkpoint import load_checkpoint, load_config
    cfg = load_config(a.model)
    from ..build import kernel_library
    os.environ.setdefault("SPARK_KERNEL_LIB", kernel_library(cfg.family))
    dev = "cuda:0"
    ecfg = EngineConfig(dtype=a.dtype)
    _, W = load_checkpoint(a.model, dev, cfg=cfg, dtype=compute_dtype(ecfg, dev))
    ses = BatchSession(cfg, W, ecfg, dev, max_seqs=a.max_seqs, kv_tokens=a.max_tokens)
    from ..ops import cuda as cu
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        if st["entries"]:
            lg = ses.step([(e["id"], e["tokens"], e.get("want", [])) for e in st["entries"]])
            if lg.shape[0]:
                lg.float().cpu().numpy().astype("<f4").tofile(os.path.join(a.out, f"{st['step']}.f32"))
            status = cu.read_status(torch.device(dev))
            if status[0]:
                raise RuntimeError(f"device status {status}")
        for rid in st.get("end", []):
            ses.end(rid)
        print(f"done {st['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
