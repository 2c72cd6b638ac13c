"""Trace replay: feed given token ids through a model step by step and write logits.

Steps are JSON lines {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: every entry
brings the next tokens of a request, `want` lists the places among them whose logits are written
to <out>/<n>.f32 ([wanted, vocab] little-endian float32, in the order of entries and places), and
`end` names the requests that are finished.  Each step is answered by a line "done <n>".  A step
is one BatchSession.step over the paged cache: what serves requests elsewhere runs here.
"""
import json
import os

from .registry import load_model
from .session import BatchSession

PAGE = 64
MAX_REQUESTS = 256


class Replay:
    def __init__(self, model_dir, dtype, max_tokens):
        context = max(1, max_tokens)
        self.model = load_model(model_dir, dtype=dtype, max_len=1)
        self.batch = BatchSession(self.model, max_seqs=MAX_REQUESTS, page_size=PAGE,
                                  n_pages=(context + PAGE - 1) // PAGE + MAX_REQUESTS, max_context=context)
        self.live = {}

    def run(self, step):
        """Logits [wanted, vocab] of a step, or None when nothing is wanted."""
        entries, want = [], []
        for e in step["entries"]:
            if e["id"] not in self.live:
                self.live[e["id"]] = self.batch.add()
            if e["tokens"]:
                entries.append((self.live[e["id"]], e["tokens"]))
                want.append(e.get("want") or [])
        logits = None
        if entries:
            logits, _ = self.batch.step(entries, want, want_logits=any(want))
        for name in step.get("end", ()):
            if name in self.live:
                self.batch.remove(self.live.pop(name))
        return logits

    def close(self):
        self.batch.close()
        self.model.close()


def replay(model_dir, dtype, max_tokens, out_dir, lines, answer):
    r = Replay(model_dir, dtype, max_tokens)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = r.run(step)
        if logits is not None and len(logits):
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(logits.astype("<f4").tobytes())
            os.replace(path + ".part", path)
        answer(f"done {step['step']}")
    r.close()
