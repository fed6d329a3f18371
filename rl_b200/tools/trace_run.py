"""Trace runner: feeds given token ids through the generation engine, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

``DIR`` is a checkpoint folder of any model family the framework serves (``config.json`` + safetensors). Every line of standard
input is one engine step:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries run as one batch through ``GenerationEngine.step``: each request's tokens continue after what earlier steps left in the
cache or state, single tokens beside portions of prompts. ``want`` names the places among the tokens whose logits go to
``OUT/<step>.f32`` (little-endian fp32 [wanted, vocab], in the order of the entries); ``end`` names requests whose pages and state
are given back after the step. ``done <step>`` is printed when a step is complete.

The cache holds ``N`` tokens (requests rounded up to whole pages), the engine has state for ``--max-requests`` live requests.
``bfloat16`` is the serving precision. ``float32`` runs every product in 32-bit; it is available for layer-list models (exit code 3
for the others). The native library is built on first use.
"""

from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="checkpoint folder")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=4, help="most live requests at any time")
    ap.add_argument("--block-size", type=int, default=64, help="tokens per cache page")
    ap.add_argument("--device", default="cuda", help="cuda, or cpu for the PyTorch statement of the same operators (tests)")
    a = ap.parse_args(argv)

    import torch

    from rl_b200.models.config import ModelConfig

    dtype = getattr(torch, a.dtype)
    cfg = ModelConfig.from_pretrained(a.model)
    if a.dtype == "float32" and a.device != "cpu" and not cfg.is_mixer:
        print(f"the {cfg.model_type} family runs in bfloat16 only", file=sys.stderr)
        return 3
    if a.device != "cpu":
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device")
        torch.backends.cuda.matmul.allow_tf32 = False
        from rl_b200.csrc.build import build_all
        from rl_b200.ops import lib as L

        if L.stale():
            build_all()
        L.lib()

    from rl_b200.engine.engine import GenerationEngine
    from rl_b200.models.hf_io import load_pretrained

    model = load_pretrained(a.model, device=a.device, dtype=dtype)
    pages = -(-a.max_tokens // a.block_size)
    engine = GenerationEngine(model, block_size=a.block_size, num_blocks=pages, max_running=a.max_requests, max_model_len=pages * a.block_size,
                              use_cuda_graphs=False, enable_prefix_caching=False)
    engine.wake()
    os.makedirs(a.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want", [])) for e in s.get("entries", [])]
        rows = engine.step(entries, s.get("end", []))
        if any(w for _, _, w in entries):
            z = torch.cat([r for r in rows if r.shape[0]]).float().cpu().contiguous().numpy().astype("<f4")
            part = os.path.join(a.out, f".{s['step']}.part")
            z.tofile(part)
            os.replace(part, os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
