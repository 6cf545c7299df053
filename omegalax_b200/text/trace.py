"""Replay of a token trace: given ids go through a model step by step and logits come out.

Nothing is sampled.  Steps arrive as JSON lines,

    {"step": 7, "entries": [{"id": "chat", "tokens": [41], "want": [0]}, ...], "end": ["mail"]}

and run as one batch each through ``text.api.decode`` with a paged cache: either every entry starts a
request, or every entry continues a request of the running batch.  Logits of the wanted places
go to <out>/<step>.f32 (little-endian fp32 [wanted, vocab]), and ``done <step>`` to standard output.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


class TraceRunner:
    def __init__(self, model, cfg, max_tokens: int, *, page_size: int = 64):
        self.model, self.cfg, self.max_tokens, self.page_size = model, cfg, max_tokens, page_size
        self.cache = None
        self.row: dict[str, int] = {}      # request -> row of the running batch

    def _start(self, entries):
        from . import api

        if self.row:
            raise ValueError("a request cannot join a running batch")
        B = len(entries)
        if self.cache is None or self.cache.B != B:
            w = next(self.model.parameters())
            longest = max(self.max_tokens, max(len(e["tokens"]) for e in entries))
            pages = -(-longest // self.page_size) + B        # every sequence may leave one page partly empty
            self.cache = None
            self.cache = api.make_cache(self.cfg, B, longest, 0, dtype=w.dtype, device=w.device, paged=True,
                                        page_size=self.page_size, num_pages=pages)
        self.row = {e["id"]: b for b, e in enumerate(entries)}

    def step(self, entries, end):
        """Logits fp32 [wanted, vocab] on the CPU in the order of the entries, or None."""
        import torch

        from . import api

        out = None
        if entries:
            if not all(e["id"] in self.row for e in entries):
                self._start(entries)
            B = self.cache.B
            rows, wants = [[] for _ in range(B)], [[] for _ in range(B)]
            for e in entries:
                rows[self.row[e["id"]]] = e["tokens"]
                wants[self.row[e["id"]]] = e["want"]
            ids = api.batch_rows(rows, B)
            select = torch.zeros(ids.shape, dtype=torch.bool)
            for b, w in enumerate(wants):
                select[b, w] = True
            w0 = next(self.model.parameters())
            dev_ids = ids if isinstance(self.model, api.StreamDecoder) else ids.to(w0.device)
            logits, self.cache, _ = api.decode(self.model, self.cache, dev_ids, api.NO_TOKEN, self.cfg, select=select)
            place = {bt: i for i, bt in enumerate(map(tuple, select.nonzero().tolist()))}
            order = [place[(self.row[e["id"]], t)] for e in entries for t in e["want"]]
            if order:
                out = logits.float()[torch.tensor(order, device=logits.device)].cpu()
        for name in end:
            self.cache.free_sequence(self.row.pop(name))
        return out


def main(argv=None) -> int:
    p = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through a model and write logits.")
    p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    p.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    p.add_argument("--out", required=True, help="folder for <step>.f32")
    p.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = p.parse_args(argv)

    import torch

    from ..ops import lib
    from . import api

    torch.backends.cuda.matmul.allow_tf32 = False
    cfg = api.resolve_config(a.model)
    serving = isinstance(cfg, api.StreamDecoderConfig)
    if a.dtype == "float32" and not serving:
        print("this model's paged decode path runs in bfloat16 only", file=sys.stderr)
        return 3
    lib.load(api.stream_registry.family_of(cfg).kernels if serving else None)
    torch.cuda.set_device(0)
    model, cfg = api.load_model(a.model, device=torch.device("cuda", 0), dtype=getattr(torch, a.dtype))
    runner = TraceRunner(model, cfg, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        req = json.loads(line)
        logits = runner.step(req["entries"], req["end"])
        lib.check_status()
        if logits is not None:
            logits.numpy().astype("<f4", copy=False).tofile(os.path.join(a.out, f"{req['step']}.f32"))
        print(f"done {req['step']}", flush=True)
    return 0
