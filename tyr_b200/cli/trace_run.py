"""Replay a trace of token ids through a model's decoding session and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

The model class follows config.json (``models/registry.py``).  Steps come as JSON objects, one a line, on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An id that is new starts a request with its whole prompt; one that is known goes on by the tokens given.  ``want`` lists places
among an entry's tokens; their logits go to ``<out>/<step>.f32`` (little-endian fp32 [wanted, vocab], in the order of the entries)
when any are wanted.  Requests in ``end`` give back what they hold.  ``done <step>`` is printed after every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from .. import _native
from ..models import registry


@dataclass
class Group:
    """Requests that run as one batch: ``ids[r]`` is row r of the session."""
    session: object
    ids: List[str]


class Replayer:
    def __init__(self, family: registry.Family, model, max_tokens: int):
        self.family, self.model, self.max_tokens = family, model, max_tokens
        self.group_of: Dict[str, Group] = {}

    @torch.no_grad()
    def step(self, entries: List[dict], end: List[str] = ()) -> Optional[torch.Tensor]:
        """Logits [wanted, vocab] of the step (None when nothing is wanted)."""
        seen = [e["id"] for e in entries]
        if len(set(seen)) != len(seen):
            raise ValueError("a request appears twice in one step")
        if any(not e["tokens"] for e in entries):
            raise ValueError("an entry without tokens")
        fresh = [e for e in entries if e["id"] not in self.group_of]
        going = [e for e in entries if e["id"] in self.group_of]
        got: Dict[str, torch.Tensor] = {}
        for batch in self._batches(fresh):
            got.update(self._start(batch))
        groups = {id(self.group_of[e["id"]]): self.group_of[e["id"]] for e in going}
        for g in groups.values():
            got.update(self._continue(g, {e["id"]: e for e in going if self.group_of[e["id"]] is g}))
        wanted = [got[e["id"]] for e in entries if e.get("want")]
        out = torch.cat(wanted) if wanted else None
        self._end(end)
        return out

    def _batches(self, entries):
        if not entries:
            return []
        ragged = self.family.ragged
        if ragged:
            return [entries]
        by_len: Dict[int, list] = {}
        for e in entries:
            by_len.setdefault(len(e["tokens"]), []).append(e)
        return list(by_len.values())

    def _start(self, entries):
        lengths = [len(e["tokens"]) for e in entries]
        S, dev = max(lengths), self.model.device
        ids = torch.tensor([e["tokens"] + [0] * (S - n) for e, n in zip(entries, lengths)], device=dev)
        s = self.family.session(self.model, len(entries), self.max_tokens)
        h = s.hidden(ids, lengths)
        g = Group(s, [e["id"] for e in entries])
        self.group_of.update({i: g for i in g.ids})
        places = [(r, p) for r, e in enumerate(entries) for p in e.get("want") or []]
        if not places:
            return {}
        rows, pos = (torch.tensor(x, device=dev) for x in zip(*places))
        logits = s.head(h[rows, pos])
        counts = [len(e.get("want") or []) for e in entries]
        return dict(zip(g.ids, torch.split(logits, counts)))

    def _continue(self, g: Group, entries: Dict[str, dict]):
        if set(entries) != set(g.ids):
            raise ValueError("the requests of a batch advance together")
        n = {len(e["tokens"]) for e in entries.values()}
        if len(n) != 1:
            raise ValueError("the requests of a batch advance by the same number of tokens")
        per_place = []
        for t in range(n.pop()):
            tok = torch.tensor([entries[i]["tokens"][t] for i in g.ids], device=self.model.device)
            logits = g.session.step(tok)
            asked = [i for i in g.ids if t in (entries[i].get("want") or [])]
            per_place.append({i: logits[g.ids.index(i)].clone() for i in asked})
        return {i: torch.stack([per_place[t][i] for t in entries[i]["want"]]) for i in g.ids if entries[i].get("want")}

    def _end(self, ids):
        gone = set(ids)
        for g in {id(g): g for i, g in self.group_of.items() if i in gone}.values():
            rows = [r for r, i in enumerate(g.ids) if i not in gone]
            if rows:
                g.session.retain(rows)
            else:
                g.session = None
            g.ids = [g.ids[r] for r in rows]
        for i in gone:
            self.group_of.pop(i, None)


def parse(argv):
    p = argparse.ArgumentParser(prog="trace_run")
    p.add_argument("--model", required=True, help="directory with config.json and safetensors weights")
    p.add_argument("--dtype", required=True, choices=("bfloat16", "float32"))
    p.add_argument("--out", required=True, help="directory for the logits")
    p.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    p.add_argument("--device", default="cuda")
    return p.parse_args(argv)


def main(argv=None, lines=None) -> int:
    a = parse(sys.argv[1:] if argv is None else argv)
    dev = torch.device(a.device)
    if dev.type == "cuda" and not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 1
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    family = registry.detect_dir(a.model)
    if family.session_class is None:
        print(f"trace_run: {family.name} has no decoding session", file=sys.stderr)
        return 2
    if dev.type == "cuda" and family.kernel_units is not None:
        _native.use_units(family.kernel_units)
    model = family.load(a.model, dev, getattr(torch, a.dtype))
    replay = Replayer(family, model, a.max_tokens)
    os.makedirs(a.out, exist_ok=True)
    for line in sys.stdin if lines is None else lines:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"], s.get("end") or ())
        if logits is not None:
            data = logits.float().cpu().contiguous().numpy().astype("<f4")
        if dev.type == "cuda":
            from ..ops._common import raise_on_device_error
            raise_on_device_error(dev)
        if logits is not None:
            data.tofile(os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
