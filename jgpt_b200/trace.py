"""Replay of a trace: requests that come and go, step by step, through a model's own step function and pool."""
from __future__ import annotations

import json
import os

import numpy as np

from .decoder import BLOCK_TOKENS


def split_step(sizes, rows):
    """Cuts the entries of a step into batches of at most ``rows`` tokens: [[(entry, first token, count), ...], ...]."""
    batches, cur, room = [], [], rows
    for i, n in enumerate(sizes):
        at = 0
        while at < n:
            take = min(n - at, room)
            cur.append((i, at, take))
            at, room = at + take, room - take
            if room == 0:
                batches.append(cur)
                cur, room = [], rows
    if cur:
        batches.append(cur)
    return batches


def replay(model, lines, out, folder, max_tokens, max_requests=4):
    """``lines``: JSON steps; wanted logits go to ``folder``/<step>.f32 (fp32, little endian), 'done <step>' lines to ``out``.
    The pool holds ``max_tokens`` tokens and ``max_requests`` sequences, so blocks and slots are used again."""
    pool = model.newPool(-(-max_tokens // BLOCK_TOKENS), max_requests)
    seqs = {}
    try:
        for line in lines:
            if not line.strip():
                continue
            step = json.loads(line)
            entries = step["entries"]
            for e in entries:
                if e["id"] not in seqs:
                    seqs[e["id"]] = pool.seq_alloc()
            got = {}
            for batch in split_step([len(e["tokens"]) for e in entries], model.maxRows):
                want, places, row = [], [], 0
                for i, at, n in batch:
                    for w in sorted(set(entries[i]["want"])):
                        if at <= w < at + n:
                            want.append(row + w - at)
                            places.append((i, w))
                    row += n
                logits, _ = model.step(pool, [seqs[entries[i]["id"]] for i, _, _ in batch],
                                       [entries[i]["tokens"][at:at + n] for i, at, n in batch], want, want_logits=bool(want))
                for j, place in enumerate(places):
                    got[place] = logits[j]
            rows = [got[(i, w)] for i, e in enumerate(entries) for w in e["want"]]
            if rows:
                np.ascontiguousarray(rows, "<f4").tofile(os.path.join(folder, f"{step['step']}.f32"))
            for rid in step.get("end", []):
                if rid in seqs:
                    pool.seq_free(seqs.pop(rid))
            print(f"done {step['step']}", file=out, flush=True)
    finally:
        pool.close()
