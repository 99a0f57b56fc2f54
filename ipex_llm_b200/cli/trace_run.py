"""``trace_run``: replay given token ids through a model step by step and write the logits it is asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N] < steps.jsonl

Nothing is sampled.  Every input line is one step,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

whose entries form one batch: the next tokens of each request and the places among them whose logits are wanted.  The
logits go to ``DIR/<step>.f32`` (little-endian 32-bit floats, [wanted, vocabulary], in the order of the entries), then
``done <step>`` is printed.  Requests under ``end`` are finished and give their cache slot back.  The steps run on the
engine that ``model.generate`` uses: prompts and portions as packed batches, single tokens through the decode step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def build_parser():
    p = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    p.add_argument("--model", required=True, help="checkpoint directory")
    p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    p.add_argument("--out", required=True, help="directory of the logits files")
    p.add_argument("--max-tokens", type=int, default=2048, help="most tokens that live requests hold together")
    return p


def load(path: str, dtype: str):
    import torch
    from ..transformers import AutoModelForCausalLM
    if dtype == "bfloat16":
        model = AutoModelForCausalLM.from_pretrained(path, load_in_low_bit="bf16", torch_dtype=torch.bfloat16,
                                                     device="cuda")
    else:
        model = AutoModelForCausalLM.from_pretrained(path, torch_dtype=torch.float32)
    return model.eval().to("cuda")


class Replay:
    """Requests by name on the slots of one engine."""

    def __init__(self, model, max_tokens: int):
        self.model, self.max_tokens = model, max_tokens
        self.engine = None
        self.slot = {}

    def step(self, entries, end):
        from ..engine import get_engine
        new = [e["id"] for e in entries if e["id"] not in self.slot]
        live = len(self.slot) + len(new)
        if self.engine is None or (not self.slot and live > self.engine.max_batch):
            self.engine = get_engine(self.model, live, self.max_tokens + 1)
            if not hasattr(self.engine, "step_rows"):
                raise NotImplementedError("the engine of this model's family does not replay traces")
        self.engine.open_cache(live)
        for name in new:
            self.slot[name] = self.engine.cache.acquire()
        logits = None
        if entries:
            logits = self.engine.step_rows([(self.slot[e["id"]], e["tokens"], e.get("want", [])) for e in entries])
        for name in end:
            self.engine.cache.release(self.slot.pop(name))
        return logits


def main(argv=None):
    a = build_parser().parse_args(argv)
    os.makedirs(a.out, exist_ok=True)
    import torch
    replay = Replay(load(a.model, a.dtype), a.max_tokens)
    with torch.no_grad():
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = replay.step(step.get("entries", []), step.get("end", []))
            if logits is not None:
                path = os.path.join(a.out, f"{step['step']}.f32")
                logits.float().cpu().numpy().astype("<f4").tofile(path)
            else:
                torch.cuda.synchronize()
            print(f"done {step['step']}", flush=True)
    from ..ops.cuda_ops import check_error_flag
    check_error_flag(torch.device("cuda", torch.cuda.current_device()))
    return 0


if __name__ == "__main__":
    sys.exit(main())
