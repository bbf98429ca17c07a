"""Teacher-forced replay of a token trace through the serving engine (``bin/trace_run``).

Reads steps from standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every step is one engine batch (:meth:`parallax_b200.engine.engine.Engine.feed`): the entries' tokens continue
their requests, slices of several tokens beside single decoded ones. The logits at the wanted places go to
``OUT/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``); requests named in ``end`` give back their cache
pages. ``done <step>`` on standard output follows every step.

``--dtype bfloat16`` is what the server runs; ``float32`` runs the model in 32-bit throughout (families whose
stages support it).
"""

from __future__ import annotations

import argparse
import json
import os
import sys


PAGE = 16
LIVE = 4          # requests that may be live at the same time


def build_engine(model: str, dtype: str, max_tokens: int, device=None):
    import torch

    from parallax_b200.engine.engine import Engine
    from parallax_b200.loader.shard_loader import ShardLoader
    from parallax_b200.models.registry import runs_in_float32

    loader = ShardLoader(model)
    if dtype == "float32" and not runs_in_float32(loader.config.architecture):
        return None
    device = device or ("cuda:0" if torch.cuda.is_available() else "cpu")
    blocks = -(-max_tokens // PAGE)
    return Engine(loader.config, device=device, dtype=getattr(torch, dtype), weights=loader.load_weights("cpu", None),
                  page_size=PAGE, num_blocks=blocks, max_batch_size=LIVE, max_requests=LIVE, chunked_prefill_size=None,
                  max_num_tokens_per_batch=blocks * PAGE, max_total_length=blocks * PAGE, enable_prefix_cache=False)


def replay(engine, lines, out_dir: str, emit) -> None:
    import numpy as np

    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = engine.feed([(e["id"], e["tokens"], e.get("want") or []) for e in step.get("entries") or []])
        if logits is not None:
            data = logits.cpu().numpy().astype(np.dtype("<f4"), copy=False)
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(np.ascontiguousarray(data).tobytes())
        for rid in step.get("end") or []:
            engine.release_fed(rid)
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits of each step")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="most tokens that live requests hold at any time, each rounded up to the page size")
    a = ap.parse_args(argv)
    with open(os.path.join(a.model, "config.json")) as f:
        from parallax_b200.models.config import config_from_hf

        cfg = config_from_hf(json.load(f))
    import torch

    if torch.cuda.is_available():
        from parallax_b200 import _build
        from parallax_b200.models.registry import family_of

        _build.ensure_kernels(family_of(cfg.architecture))
    engine = build_engine(a.model, a.dtype, a.max_tokens)
    if engine is None:
        print(f"{cfg.architecture} does not run in 32-bit", file=sys.stderr)
        return 3
    os.makedirs(a.out, exist_ok=True)
    replay(engine, sys.stdin, a.out, lambda text: print(text, flush=True))
    return 0
