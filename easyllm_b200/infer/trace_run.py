"""Trace replay: feed given token ids through a model as batched steps and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--device cuda|cpu]

Steps come as JSON lines on standard input,
``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [1]}], "end": []}``: the entries are one batch, ``want``
names the tokens (by place in the entry) whose logits are written to ``DIR/<step>.f32`` (little-endian fp32, in order),
``end`` the requests that are finished.  After every step ``done <step>`` is printed.  The model, the step function and
the cache / state manager are those of ``CausalLM.generate``; nothing is sampled.  Useful to compare two builds, two
dtypes or two batchings on the same requests.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch


class TraceSession:
    """Requests by id over a model's step function and state manager."""

    def __init__(self, model, max_tokens=None, slots=4):
        self.model = model
        self.state = model.new_state(slots, min(max_tokens or 1024, 1024))      # grows when a request is longer
        self.slot = {}

    @torch.no_grad()
    def run(self, entries):
        """One step: ``entries`` are ``(id, tokens, want)``.  Logits fp32 ``[number wanted, vocab]`` or None."""
        for rid, _, _ in entries:
            if rid not in self.slot:
                self.slot[rid] = self.state.open()
        h, _ = self.model.step(self.state, [self.slot[rid] for rid, _, _ in entries], [t for _, t, _ in entries])
        rows, at = [], 0
        for _, tokens, want in entries:
            rows += [at + w for w in want]
            at += len(tokens)
        if not rows:
            return None
        return self.model.logits(h[torch.tensor(rows, device=h.device)])

    def end(self, rid):
        self.state.close(self.slot.pop(rid))


def load_model(path, dtype, device):
    from ..config.registry import MODULE_ZOO_REGISTRY
    from ..models import hf_models  # noqa: F401  (fills the registry)
    if device.type == "cuda":
        from ..ops import build, cuda
        build.ensure_serving()
        cuda.lib()
        torch.backends.cuda.matmul.allow_tf32 = torch.backends.cudnn.allow_tf32 = False
    model = MODULE_ZOO_REGISTRY.build({"type": "AutoCausalLM", "kwargs": {"model_name_or_path": path,
                                                                        "torch_dtype": "torch." + dtype}})
    return model.to(device).eval()


def main(argv=None):
    p = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    p.add_argument("--model", required=True, help="folder with config.json and the weights")
    p.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    p.add_argument("--out", required=True, help="folder the logits are written to")
    p.add_argument("--max-tokens", type=int, default=None, help="most tokens the live requests hold at any time")
    p.add_argument("--device", default="cuda", choices=["cuda", "cpu"])
    a = p.parse_args(argv)
    device = torch.device(a.device, 0) if a.device == "cuda" else torch.device("cpu")
    session = TraceSession(load_model(a.model, a.dtype, device), a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = session.run([(e["id"], e["tokens"], e["want"]) for e in step["entries"]]) if step["entries"] else None
        if device.type == "cuda":
            from ..ops import cuda
            cuda.check_step_errors()
        if logits is not None:
            logits.float().cpu().numpy().astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for rid in step["end"]:
            session.end(rid)
        print(f"done {step['step']}", flush=True)
    return 0
