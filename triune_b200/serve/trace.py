"""Trace runner: feeds given token ids through a model folder's model, step by step, and writes logits.

Standard input holds one JSON object a line: ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}],
"end": [ids]}``. An entry's tokens follow those its request brought before; ``want`` are places among them whose logits
go to ``<out>/<step>.f32`` (little-endian fp32, in the order of the entries and of ``want``). ``end`` gives finished
requests' caches back. After every step a line ``done <step>`` is printed. Nothing is sampled: the steps run through
:func:`triune_b200.inference.advance`, which is what the generation paths run."""

from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Any, Dict, Iterable, List, Optional

DTYPES = ("bfloat16", "float32")


class TraceRunner:
    """The requests in flight and their caches."""

    def __init__(self, model, max_tokens: int = 0):
        self.model, self.max_tokens = model, int(max_tokens)
        self.device = next(model.parameters()).device
        self.caches: Dict[str, List[Any]] = {}

    def _cache(self, rid: str) -> List[Any]:
        if rid not in self.caches:
            self.caches[rid] = self.model.init_cache(1)
        return self.caches[rid]

    def step(self, entries: Iterable[Dict[str, Any]], end: Iterable[str] = ()):
        """-> the wanted logits [rows, vocab] as one CPU fp32 tensor, or None when nothing is wanted."""
        import torch

        from ..inference import advance
        from ..ops import hybrid as hops

        rows = []
        for e in entries:
            rid, want = str(e["id"]), list(e.get("want", ()))
            cache = self._cache(rid)
            if e["tokens"]:
                ids = torch.tensor([e["tokens"]], dtype=torch.long, device=self.device)
                logits, self.caches[rid] = advance(self.model, ids, cache, positions=want)
                if want:
                    rows.append(logits[0].float())
        for rid in end:
            self.caches.pop(str(rid), None)
        if not rows:
            return None
        out = torch.cat(rows).cpu()
        if self.device.type == "cuda":
            hops.check_status(self.device)
        return out


def load(folder: str, dtype: str, device: Optional[str] = None):
    import torch

    from ..inference import load_model_for_inference

    dev = torch.device(device or "cuda:0")
    if dev.type == "cuda":
        from .._build import ensure_serving

        ensure_serving()
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.set_float32_matmul_precision("highest")
    return load_model_for_inference(folder, dev, {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype])


def run(model, out: Path, lines, stdout, max_tokens: int = 0) -> None:
    runner = TraceRunner(model, max_tokens)
    for line in lines:
        if not line.strip():
            continue
        rec = json.loads(line)
        logits = runner.step(rec["entries"], rec.get("end", ()))
        if logits is not None:
            (out / f"{rec['step']}.f32").write_bytes(logits.contiguous().numpy().astype("<f4").tobytes())
        stdout.write(f"done {rec['step']}\n")
        stdout.flush()


def add_arguments(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=DTYPES)
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default=None, help="default: the first GPU")


def main(argv: Optional[List[str]] = None, args: Optional[argparse.Namespace] = None) -> int:
    if args is None:
        ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
        add_arguments(ap)
        args = ap.parse_args(argv)
    out = Path(args.out)
    out.mkdir(parents=True, exist_ok=True)
    run(load(args.model, args.dtype, args.device), out, sys.stdin, sys.stdout, args.max_tokens)
    return 0
