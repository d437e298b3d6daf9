"""Replay a trace: feed given token ids through a model step by step and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come one per line on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``tokens`` are a request's next tokens, ``want`` the places among them whose logits are written (little-endian fp32
``[wanted, vocab]``, to ``<out>/<step>.f32``), ``end`` the requests that are finished after the step.  ``done <step>`` is
printed after every step.  Nothing is sampled; the tokens run through the engine's own calls: a request's first tokens and
longer portions through :meth:`PagedDecodeEngine.extend`, single tokens through the decode step
(:meth:`PagedDecodeEngine.feed`, a replay of the captured graph).
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

DTYPES = {"bfloat16": "bfloat16", "float32": "float32"}
EXIT_NO_DTYPE = 3


class TraceRunner:
    def __init__(self, engine, out: Path) -> None:
        self.engine, self.out = engine, out
        self.rows: dict[str, int] = {}

    def step(self, step: dict) -> None:
        import torch

        eng = self.engine
        single = [e for e in step["entries"] if len(e["tokens"]) == 1 and e["id"] in self.rows]
        longer = [e for e in step["entries"] if e["tokens"] and not (len(e["tokens"]) == 1 and e["id"] in self.rows)]
        logits: dict[str, torch.Tensor] = {}
        if longer:
            for e in longer:
                if e["id"] not in self.rows:
                    self.rows[e["id"]] = eng.open_request()
            hidden = eng.extend([(self.rows[e["id"]], e["tokens"]) for e in longer])
            picks, at = [], 0
            for e in longer:
                picks += [at + w for w in e["want"]]
                at += len(e["tokens"])
            if picks:
                rows = eng.model.compute_logits(hidden, torch.tensor(picks, dtype=torch.int64, device=eng.device))
                for e in longer:
                    logits[e["id"]], rows = rows[: len(e["want"])], rows[len(e["want"]):]
        if single:
            rows = eng.feed({self.rows[e["id"]]: e["tokens"][0] for e in single})
            for e, row in zip(single, rows):
                logits[e["id"]] = row.unsqueeze(0).expand(len(e["want"]), -1)
        wanted = [logits[e["id"]] for e in step["entries"] if e["want"]]
        if wanted:
            data = torch.cat([w.to(torch.float32) for w in wanted]).cpu().numpy().astype("<f4")
            (self.out / f"{step['step']}.f32").write_bytes(data.tobytes())
        else:
            torch.cuda.synchronize(eng.device)
        eng.state.check_status()
        for name in step.get("end", []):
            if name in self.rows:
                eng.release(self.rows.pop(name))


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=8, help="most requests alive at any time")
    ap.add_argument("--block-size", type=int, default=16, help="tokens per cache page")
    args = ap.parse_args(argv)

    import torch

    from .checkpoint import load_config
    from .registry import find_model, load_model, new_engine

    dtype = getattr(torch, DTYPES[args.dtype])
    if dtype not in find_model(load_config(args.model)).dtypes:
        print(f"this model does not run in {args.dtype}", file=sys.stderr)
        return EXIT_NO_DTYPE
    model = load_model(args.model, dtype)
    bs = args.block_size
    # every live request can leave one page partly filled; the last block is the pad block
    blocks = -(-args.max_tokens // bs) + args.max_requests + 1
    engine = new_engine(model, num_blocks=blocks, block_size=bs, max_num_seqs=args.max_requests,
                        max_model_len=(-(-args.max_tokens // bs) + 1) * bs)
    runner = TraceRunner(engine, Path(args.out))
    for line in sys.stdin:
        if line.strip():
            step = json.loads(line)
            runner.step(step)
            print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
