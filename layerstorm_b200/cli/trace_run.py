"""``bin/trace_run`` - replay a trace of token ids through the engine's step function and write logits.

Reads one JSON object per line from standard input,

    {"step": 7, "entries": [{"id": "x", "tokens": [11, 4], "want": [1]}, {"id": "y", "tokens": [9]}], "end": ["y"]}

and runs all entries of a line as one batch (``Engine.step``): each request's next tokens, appended to what earlier steps left in the
cache and state.  ``want`` lists the places among an entry's tokens whose logits are asked for; a step that wants any writes
``OUT/<step>.f32`` (little-endian fp32, [wanted, vocab], in the order of the entries).  ``end`` names requests that are finished after the
step; their pages and slot are given back.  ``done <step>`` follows every step.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

SLOTS = 4                     # requests live at a time
PAGE = 64                     # tokens per cache page
CHUNK = 512                   # rows of a pass; larger steps run in several passes


def build_parser() -> argparse.ArgumentParser:
    p = argparse.ArgumentParser(prog="trace_run", description="Replay a token trace through the engine and write logits")
    p.add_argument("--model", required=True, help="checkpoint directory (config.json, *.safetensors)")
    p.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16",
                   help="bfloat16: the precisions this model is served with; float32: everything in fp32")
    p.add_argument("--out", required=True, help="directory for <step>.f32")
    p.add_argument("--max-tokens", type=int, required=True, help="size of the cache pool: tokens of all unfinished requests together")
    return p


def open_engine(args):
    """The engine the server would run this checkpoint on, with a cache pool of ``--max-tokens`` tokens; None when ``--dtype`` float32 is not
    available for this kind of model."""
    from ..models.config import from_hf_config
    cfg = from_hf_config(os.path.join(args.model, "config.json"))
    if args.dtype == "float32" and not cfg.blocks:
        return None
    from .. import build
    build.ensure_for(cfg)
    import torch
    from ..models.block_model import model_class
    from ..models.checkpoint import open_checkpoint
    from ..runtime.engine import Engine
    _, w = open_checkpoint(args.model, cfg)
    kw = {"dtype": args.dtype} if cfg.blocks else {"kv_fmt": "bf16"}
    model = model_class(cfg).from_state_dict(cfg, w, torch.device("cuda", 0), page=PAGE, **kw)
    pages = max(1, (args.max_tokens + PAGE - 1) // PAGE)
    return Engine(model, max_seqs=SLOTS, max_ctx=pages * PAGE, prefill_chunk=CHUNK, max_batch=SLOTS, num_pages=pages)


def replay(eng, lines, out_dir: str, emit) -> None:
    """Runs the steps of ``lines`` on ``eng``; ``emit(text)`` gets the line that follows each step."""
    from ..runtime.engine import Portion
    sids: dict = {}
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        portions = []
        for e in st.get("entries", []):
            if e["id"] not in sids:
                sids[e["id"]] = eng.create_sequence()
            portions.append(Portion(sids[e["id"]], [int(t) for t in e["tokens"]], [int(k) for k in e.get("want", [])]))
        if portions:
            want_any = any(p.want for p in portions)
            res = eng.step(portions, return_logits=want_any)
            if want_any:
                import torch
                rows = torch.cat([lg for _, lg in res]).contiguous()
                path = os.path.join(out_dir, f"{st['step']}.f32")
                with open(path + ".tmp", "wb") as f:
                    f.write(rows.numpy().astype("<f4").tobytes())
                os.replace(path + ".tmp", path)
        for rid in st.get("end", []):
            if rid in sids:
                eng.free_sequence(sids.pop(rid))
        emit(f"done {st['step']}")


def main(argv=None) -> int:
    args = build_parser().parse_args(argv)
    eng = open_engine(args)
    if eng is None:
        print("float32 is not available for this kind of model", file=sys.stderr)
        return 3

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(eng, sys.stdin, args.out, emit)
    return 0


if __name__ == "__main__":
    sys.exit(main())
