"""Generation from the command line, through the continuous-batching scheduler:

    python -m jgpt_b200.generate --model DIR --prompt 5,17,3 [--prompt ...] --max-new 32 [--dtype float32]

DIR holds config.json and model.safetensors (registry.py picks the design).  Prompts are token ids; one JSON line per prompt.
With --temperature the prompts run one after the other and tokens are drawn on the device.
"""
from __future__ import annotations

import argparse
import json
import sys

import numpy as np

from .decoder import BLOCK_TOKENS
from .registry import load_model
from .runtime import Context
from .scheduler import ContinuousBatcher


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m jgpt_b200.generate", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be given several times")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--seed", type=int, default=None)
    ap.add_argument("--max-running", type=int, default=16)
    ap.add_argument("--max-rows", type=int, default=2048, help="rows of one step")
    a = ap.parse_args(argv)
    prompts = [np.array([int(x) for x in p.split(",")], np.int32) for p in a.prompt]
    with Context(0) as ctx:
        model = load_model(ctx, a.model, a.dtype, max_rows=a.max_rows)
        need = [-(-(p.size + a.max_new) // BLOCK_TOKENS) for p in prompts]
        running = min(a.max_running, len(prompts))
        pool = model.newPool(sum(sorted(need)[-running:]), running)
        if a.temperature > 0:
            rng = np.random.default_rng(a.seed)
            for p in prompts:
                out = model.generateGpuKv(p, a.max_new, a.temperature, a.top_k, pool, rng)
                print(json.dumps({"prompt": p.tolist(), "tokens": out[p.size:].tolist()}), flush=True)
        else:
            batch = ContinuousBatcher(model, pool, running)
            ids = [batch.submit(p, a.max_new) for p in prompts]
            batch.run()
            for p, r in zip(prompts, ids):
                print(json.dumps({"prompt": p.tolist(), "tokens": batch.result(r)[0].tolist()}), flush=True)
            batch.close()
        pool.close(), model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
