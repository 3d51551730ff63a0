"""Token-trace replay: given token ids go through a model step by step, the logits asked for come out as files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Standard input carries one step per line, ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}``:
every entry is a request's next tokens and the places among them whose logits are wanted; ``end`` names requests that are finished
after the step.  All entries of a step are one engine batch (``RolloutEngine.extend``), so a trace exercises exactly the paths that
generation uses: packed portions of prompts beside decoded tokens, the decode step's CUDA graph, page and state-slot reuse.  A step
that wants something writes ``OUT/<step>.f32`` (little-endian fp32 rows in entry order), and after every step ``done <step>`` is
printed.  ``--max-tokens`` bounds the tokens that live requests hold at any time and sizes the cache pool.

The first call compiles the serving module of the extension when it is missing or out of date.
"""
from __future__ import annotations

import argparse
import fcntl
import json
import sys
from pathlib import Path

MAX_LIVE = 4                      # requests that hold pages and a state slot at one time


def _build() -> None:
    from ..ops import build as B

    B.BUILD.mkdir(parents=True, exist_ok=True)
    with open(B.BUILD / ".lock", "w") as lock:          # concurrent first calls compile once
        fcntl.flock(lock, fcntl.LOCK_EX)
        B.build(modules=("_serve",))


def load_engine(model: str, dtype_name: str, max_tokens: int, device: str):
    import torch

    from ..models import TransformerWeights, get_model_config
    from ..models.hf_io import load_state_dict
    from .engine import PAGE, RolloutEngine

    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    torch.set_float32_matmul_precision("highest")
    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype_name]
    cfg = get_model_config(model)
    w = TransformerWeights(cfg, device=device, dtype=dtype, init=False)
    w.load_state_dict({k: v.to(device, dtype) for k, v in load_state_dict(cfg, model).items()})
    eng = RolloutEngine(cfg, device, max_num_seqs=MAX_LIVE, max_model_len=max_tokens, kv_cache_tokens=max_tokens + PAGE, dtype=dtype)
    eng.set_weights(w.embed, w.layers, w.head)
    return eng


def replay(eng, lines, out: Path, emit=print) -> None:
    live: dict = {}
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        entries = []
        for e in st["entries"]:
            if e["id"] not in live:
                live[e["id"]] = eng.open(str(e["id"]))
            entries.append((live[e["id"]], e["tokens"], e.get("want", [])))
        logits = eng.extend(entries) if entries else None
        if logits is not None:
            (out / f"{st['step']}.f32").write_bytes(logits.cpu().numpy().astype("<f4").tobytes())
        elif eng.is_cuda:
            import torch

            torch.cuda.synchronize(eng.device)
        for rid in st.get("end", []):
            eng.close(live.pop(rid))
        emit(f"done {st['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through the rollout engine.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    import torch

    if a.device.startswith("cuda"):
        if not torch.cuda.is_available():
            print("trace_run: no CUDA device", file=sys.stderr)
            return 1
        _build()
    eng = load_engine(a.model, a.dtype, a.max_tokens, a.device)
    replay(eng, sys.stdin, Path(a.out), emit=lambda s: print(s, flush=True))
    return 0
