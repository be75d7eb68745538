"""Replay of a recorded schedule: given token ids go through the engine step by step, logits come out.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N        (also: nanoengine replay ...)

Standard input carries one JSON object a line, one engine step each:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`entries`: the next tokens of each request and the places among them whose logits are wanted; all entries of a step are one batch
(portions of prompts beside single tokens).  `end`: requests whose pages and state slots are given back after the step.  A step
with wanted places writes OUT/<step>.f32, little-endian fp32 [wanted, vocab] in the order of the entries and of `want`; after every
step the line `done <step>` is printed.  Nothing is sampled.  --max-tokens is the most tokens live requests hold at any time, each
rounded up to whole 64-token pages: the cache pool gets that many pages, and there are state slots for --max-requests requests.

The steps run through `LLM.feed`: the engine's scheduler, pages, state slots, step inputs, graph replay and kernels.  From a tree
that has not been built only the C++ core and the kernels the model's architecture needs are compiled."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a schedule of token ids and write logits")
    ap.add_argument("--model", required=True, help="checkpoint directory (config.json, *.safetensors)")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live requests hold at any time, each rounded up to 64")
    ap.add_argument("--max-requests", type=int, default=4, help="most live requests")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"])
    ap.add_argument("--eager", action="store_true", help="no CUDA graphs for single-token steps")
    a = ap.parse_args(argv)

    import torch
    from ..models.config import ModelConfig
    if a.device == "cuda" and not torch.cuda.is_available():
        raise SystemExit("trace_run: no CUDA device (--device cpu runs the plain PyTorch statements)")
    mc = ModelConfig.from_pretrained(a.model)
    from .. import build_native
    if a.device == "cuda":
        library = build_native.build_for(mc.architecture)
        from ..ops import sm100
        sm100.use_library(library)
    else:
        build_native.OUT.mkdir(parents=True, exist_ok=True)
        build_native.build_core()
    torch.backends.cuda.matmul.allow_tf32 = torch.backends.cudnn.allow_tf32 = False
    from .. import LLM, Config
    pages = max(1, -(-a.max_tokens // PAGE))
    longest = min(pages * PAGE, mc.max_position_embeddings) if mc.learned_positions else pages * PAGE
    llm = LLM(Config(model=a.model, model_config=mc, dtype=a.dtype, device=a.device, max_num_seqs=a.max_requests, kvcache_block_size=PAGE,
                     num_kvcache_blocks=pages, max_model_len=longest, max_num_batched_tokens=pages * PAGE, enable_prefix_caching=False,
                     executor_backend="inproc", enforce_eager=a.eager, status_log_interval_s=0))
    number = {}                     # request name -> sequence id of the engine
    next_id = 1
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        for e in step["entries"]:
            if e["id"] not in number:
                number[e["id"]] = next_id
                next_id += 1
        if step["entries"]:
            logits = llm.feed([(number[e["id"]], e["tokens"]) for e in step["entries"]], [e.get("want", []) for e in step["entries"]])
            if logits is not None:
                logits.astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        llm.end_feed([number.pop(i) for i in step.get("end", []) if i in number])
        print(f"done {step['step']}", flush=True)
    llm.shutdown()
    return 0


if __name__ == "__main__":
    sys.exit(main())
