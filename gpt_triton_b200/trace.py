"""Replaying a trace: given token ids go through a model step by step, as its generation path would run them, and the
logits at wanted places are written out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every step feeds the entries' next tokens; for a step with wanted places OUT/<step>.f32 receives their logits, little-
endian float32, [wanted, vocab], in order.  ``done <step>`` is printed after every step.  `end` lists the requests whose
memory is given back.  Exit code 3: the model does not run in the dtype that was asked for.
"""

import argparse
import json
import os
import sys


class TraceRunner:
    """Requests by id on top of GenerationSession; sessions of finished requests serve later ones."""

    def __init__(self, model, max_tokens):
        self.model, self.max_tokens = model, max(int(max_tokens), 1)
        self.live, self.free = {}, []

    def _session(self, request):
        from .generation import GenerationSession

        if request not in self.live:
            self.live[request] = self.free.pop() if self.free else GenerationSession(self.model, 1, self.max_tokens)
        return self.live[request]

    def feed(self, request, tokens, want):
        """The next tokens of a request -> logits (len(want), vocab) float32 on the CPU, or None if nothing is wanted."""
        import torch

        session = self._session(request)
        dev = session.pos.device
        ids = torch.tensor([tokens], dtype=torch.int64, device=dev)
        places = torch.tensor(want if want else [len(tokens) - 1], dtype=torch.int64, device=dev)
        rows = session.extend(ids, places)
        if not want:
            return None
        return self.model.head_logits(rows).float().cpu()

    def end(self, request):
        session = self.live.pop(request, None)
        if session is not None:
            session.reset()
            self.free.append(session)


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)

    import torch

    from .build import build

    build()
    from . import kernels
    from .registry import load_model

    model = load_model(args.model, dtype=getattr(torch, args.dtype))
    if args.dtype == "float32" and not model.exact_float32:
        print("this architecture has no true 32-bit path", file=sys.stderr)
        return 3
    runner = TraceRunner(model, args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for entry in step["entries"]:
            if not entry["tokens"]:
                continue
            logits = runner.feed(entry["id"], entry["tokens"], entry.get("want") or [])
            if logits is not None:
                parts.append(logits)
        code = kernels.device_status()
        if code:
            raise RuntimeError(f"a kernel reported code {code}")
        if parts:
            data = torch.cat(parts).contiguous().numpy().astype("<f4")
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data.tobytes())
        for request in step.get("end") or []:
            runner.end(request)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
