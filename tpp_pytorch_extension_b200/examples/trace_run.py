"""Replays a trace of token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N] < steps.jsonl

Every input line is one step:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}
The entries of a step form one batch through the runner's forward: either all of them start (prompts of different lengths
are padded on the left) or all go on from the cache. `want` lists the tokens of the entry whose logits are written, to
OUT/<step>.f32 as 32-bit floats [wanted, vocab]; `end` the requests whose cache rows are given back after the step. After
every step a line `done <step>` is printed."""
import argparse
import json
import os
import sys

import torch


class TraceBatch:
    """The live batch: request ids in cache-row order and the cache they share."""

    def __init__(self, runner):
        self.runner, self.rows, self.cache, self.mask = runner, [], None, None  # mask: keep-mask of all tokens so far

    def step(self, entries):
        """Runs one step; returns the wanted logits [n, vocab] in the order asked for (None if nothing is wanted)."""
        from tpp_pytorch_extension_b200.llm.llm_common import TppCache
        if not entries:
            return None
        ids = [e["id"] for e in entries]
        if len(set(ids)) != len(ids) or any(not e["tokens"] for e in entries):
            raise ValueError("a step needs distinct requests with at least one token each")
        if not self.rows:
            self.rows, self.cache = list(ids), TppCache()
            width = max(len(e["tokens"]) for e in entries)
            self.mask = torch.tensor([[0] * (width - len(e["tokens"])) + [1] * len(e["tokens"]) for e in entries])
        else:
            if not set(ids) <= set(self.rows):
                raise ValueError("a request joins a batch that has already started")
            self._keep([r for r in self.rows if r in set(ids)])  # a request that is not fed any more has ended
            width = len(entries[0]["tokens"])
            if any(len(e["tokens"]) != width for e in entries):
                raise ValueError("requests that go on must bring the same number of tokens")
            self.mask = torch.cat([self.mask, torch.ones((len(self.rows), width), dtype=self.mask.dtype)], dim=1)
        by_id = {e["id"]: e for e in entries}
        order = [by_id[r] for r in self.rows]
        tokens = torch.tensor([[0] * (width - len(e["tokens"])) + e["tokens"] for e in order])
        dev = self.runner.embed.device
        row_of = {r: i for i, r in enumerate(self.rows)}
        want = [row_of[e["id"]] * width + width - len(e["tokens"]) + k for e in entries for k in e["want"]]
        self.runner.logit_rows = torch.tensor(want, dtype=torch.int64, device=dev)
        try:
            pos = (self.mask.cumsum(-1) - 1).clamp_(min=0)[:, -width:].contiguous()
            logits, self.cache = self.runner.forward(tokens.to(dev), self.mask.to(dev), pos.to(dev), self.cache)
        finally:
            self.runner.logit_rows = None
        return logits if want else None

    def _keep(self, rows):
        if rows != self.rows:
            kept = [self.rows.index(r) for r in rows]
            self.cache.get_cpp().keep_sequences(kept)
            self.mask, self.rows = self.mask[kept], rows

    def end(self, ids):
        left = [r for r in self.rows if r not in set(ids)]
        if not left:
            self.rows, self.cache, self.mask = [], None, None
        else:
            self._keep(left)


def main(argv=None):
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits files")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens live at any time (the cache grows on demand)")
    a = ap.parse_args(argv)
    from tpp_pytorch_extension_b200.llm import model_registry
    dtype = getattr(torch, a.dtype)
    name = model_registry.architecture_of(a.model)
    if dtype not in model_registry.dtypes_of(name):
        print(f"{name} does not run in {a.dtype}", file=sys.stderr)
        return 3
    from tpp_pytorch_extension_b200 import _build, _lib
    _lib.use_library(_build.ensure(name))
    runner = model_registry.load_model(a.model, dtype)
    batch = TraceBatch(runner)
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = batch.step(st["entries"])
        if logits is not None:
            data = logits.float().cpu().numpy().astype("<f4").tobytes()
            with open(os.path.join(a.out, f"{st['step']}.f32"), "wb") as f:
                f.write(data)
        batch.end(st["end"])
        _lib.assert_no_kernel_error()
        print(f"done {st['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
