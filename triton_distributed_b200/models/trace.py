"""Replay of a recorded trace: JSON steps on standard input, logits as raw fp32 files (command line: ``bin/trace_run``).

A step is ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}``; it runs through
:meth:`Engine.step`, the logits at the wanted places go to ``<out>/<n>.f32``, and ``done <n>`` is printed when the step is
complete.
"""
from __future__ import annotations

import json
import os
import sys

import torch

from .config import ModelConfig
from .engine import Engine


def replay(engine: Engine, lines, out_dir: str, stdout=None):
    stdout = stdout or sys.stdout
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want") or []) for e in st.get("entries", [])]
        if entries:
            logits = engine.step(entries)
            if any(w for _, _, w in entries):
                data = logits.float().contiguous().cpu().numpy().astype("<f4").tobytes()
                with open(os.path.join(out_dir, f"{st['step']}.f32"), "wb") as f:
                    f.write(data)
            elif logits.is_cuda:
                torch.cuda.synchronize()
        engine.end(st.get("end") or [])
        print(f"done {st['step']}", file=stdout, flush=True)


def make_engine(model_dir: str, dtype: torch.dtype, max_tokens: int, backend: str = "triton_dist_gemm_ar") -> Engine:
    cfg = ModelConfig(model_name=model_dir, max_length=max(1, max_tokens), dtype=dtype, checkpoint_dir=model_dir)
    engine = Engine(cfg)
    engine.backend = backend
    return engine
