"""Feed given token ids through a checkpoint, step by step, and write logits.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

Every line of standard input is a step: {"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [0]}], "end": []}. All
entries of a step run as one batch; "want" are the places among an entry's tokens whose logits are written, "end" the requests
that are finished after the step. A step in which something is wanted writes DIR/<step>.f32 (little-endian fp32, [wanted, vocab],
entry by entry); after every step a line "done <step>" is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)

    # a fresh checkout compiles only the kernels that these models need
    from ..build import layered_library
    os.environ.setdefault("OVB_CUDA_LIB", str(layered_library()))

    import torch

    from ..genai.replay import Replay
    from ..models.registry import load_checkpoint
    from ..ops import cuda as K
    from ..runtime.layered_llm import create_executor

    block = 16
    seqs = max(1, min(args.max_tokens, 128))
    longest = (args.max_tokens + block - 1) // block + 1
    with torch.no_grad():
        ex, _ = create_executor(load_checkpoint(args.model), torch.cuda.current_device(), max_num_seqs=seqs,
                                max_num_batched_tokens=max(seqs, min(args.max_tokens, 8192)), max_model_len=args.max_tokens, block_size=block,
                                kv_cache_blocks=longest + seqs, properties={"INFERENCE_PRECISION_HINT": args.dtype})
        replay = Replay(ex)
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            logits = replay.step([(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]])
            K.check_status("step %s" % step["step"])
            if len(logits):
                with open(os.path.join(args.out, "%s.f32" % step["step"]), "wb") as f:
                    f.write(logits.contiguous().numpy().astype("<f4").tobytes())
            for rid in step.get("end", []):
                replay.end(rid)
            print("done %s" % step["step"], flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
