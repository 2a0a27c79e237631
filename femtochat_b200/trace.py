"""Replays a trace of token ids through a model, step by step, and writes the logits that were asked for.

Steps come as JSON lines: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  Each request holds one
cache; a finished request gives its cache back and the next one takes it over.  Nothing is sampled."""
from __future__ import annotations

import argparse
import json
import os
import sys


class TraceRunner:
    def __init__(self, model, max_tokens: int):
        self.model, self.max_tokens = model, max(1, max_tokens)
        self.live, self.free = {}, []

    def cache(self, rid):
        from .generation import KVCache
        if rid not in self.live:
            self.live[rid] = self.free.pop() if self.free else KVCache(self.model.state(1), 1, self.max_tokens)
        return self.live[rid]

    def end(self, rid):
        c = self.live.pop(rid, None)
        if c is not None:
            c.reset()
            self.free.append(c)

    def step(self, entries):
        """fp32 logits [wanted, vocab] on the CPU, in the order of the entries, or None."""
        import torch
        from .generation import extend
        out = []
        for e in entries:
            if not e["tokens"]:
                continue
            want = e.get("want", [])
            order = sorted(set(want))
            z = extend(self.model, self.cache(e["id"]), torch.tensor([e["tokens"]], dtype=torch.int32), want=order)
            if want:
                z = z.cpu()
                out.append(z if order == want else z[[order.index(w) for w in want]])
        return torch.cat(out) if out else None


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed given tokens through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    import torch
    from .models import load_model
    model = load_model(a.model, compute_type=a.dtype)
    runner = TraceRunner(model, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        z = runner.step(s["entries"])
        torch.cuda.synchronize()
        word = model.state(1).status_word()
        if word:
            raise RuntimeError(f"device status word {word}")
        if z is not None:
            with open(os.path.join(a.out, "%d.f32" % s["step"]), "wb") as f:
                f.write(z.contiguous().numpy().astype("<f4").tobytes())
        for rid in s.get("end", []):
            runner.end(rid)
        print("done %d" % s["step"], flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
