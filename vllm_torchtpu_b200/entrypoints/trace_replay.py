"""``bin/trace_run``: feed given token ids through a model step by step and write the logits of chosen positions.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every line of standard input is one step (one batch):

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` brings the next tokens of each request and the places among them whose logits are wanted; ``end`` lists
the requests that are finished after the step.  A step in which something is wanted leaves ``OUT/<step>.f32``
(little-endian fp32 [wanted, vocab] in the order of the entries); ``done <step>`` is printed after every step.  The
KV pool holds ``--max-tokens`` tokens.  Exit code 3: the model has no 32-bit kernels (``--dtype float32``).

The kernels a model needs are compiled at the first call if the library is not built.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

BLOCK = 16
MAX_REQS = 4


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda", help="cuda, or cpu for the plain-PyTorch ops")
    return ap.parse_args(argv)


def make_replay(model: str, dtype: str, max_tokens: int, device: str = "cuda"):
    from ..config import ModelConfig
    from ..engine.llm import LLM
    from ..engine.replay import TraceReplay
    from ..models.registry import get_model_class
    mc = ModelConfig.from_pretrained(model)
    if device == "cuda":
        if dtype == "float32" and not getattr(get_model_class(mc), "float32_kernels", False):
            return None
        from ..csrc import build
        from ..ops import cuda
        cuda.load_lib(build.ensure_built(mc.architecture))
    blocks = -(-max_tokens // BLOCK)
    llm = LLM(model, dtype=dtype, device=device, scheduler_cls="replay", max_num_seqs=MAX_REQS, block_size=BLOCK,
              max_model_len=blocks * BLOCK, max_num_batched_tokens=blocks * BLOCK, num_gpu_blocks_override=blocks + 1,
              init_dist=False)
    return TraceReplay(llm.engine)


def main(argv=None) -> int:
    a = parse_args(argv)
    replay = make_replay(a.model, a.dtype, a.max_tokens, a.device)
    if replay is None:
        print(f"{a.model}: this model has no 32-bit kernels", file=sys.stderr)
        return 3
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        rows = replay.step([(e["id"], e["tokens"], e.get("want") or []) for e in s["entries"]], s.get("end") or [])
        if rows is not None:
            rows.numpy().astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0
