"""``python -m openrlhf.cli.generate``: batch generation with the rollout engine, for any model the registry knows.

Prompts come as JSON lines, from ``--input`` or standard input: a list of token ids, ``{"tokens": [...]}``, or, when the
model folder has a tokenizer, ``{"prompt": "text"}``. One JSON line per sample is printed in the order of the prompts:
``{"prompt": 0, "sample": 0, "tokens": [...], "logprobs": [...], "finish_reason": "length"}`` (plus "text")."""
from __future__ import annotations

import argparse
import json
import os
import sys


def build_parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="generate", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="checkpoint folder or preset name")
    ap.add_argument("--input", default="-", help="JSON lines file; - for standard input")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max_new_tokens", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top_p", type=float, default=1.0)
    ap.add_argument("--top_k", type=int, default=-1)
    ap.add_argument("--n_samples", type=int, default=1)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--ignore_eos", action="store_true")
    ap.add_argument("--max_num_seqs", type=int, default=64, help="rows of the engine (sequences decoded together)")
    ap.add_argument("--max_prefill_tokens", type=int, default=16384, help="prompt tokens per prefill pass")
    ap.add_argument("--device", default="cuda")
    return ap


def read_prompts(lines, tokenizer=None) -> list[list[int]]:
    out = []
    for line in lines:
        if not line.strip():
            continue
        d = json.loads(line)
        if isinstance(d, list):
            out.append([int(t) for t in d])
        elif "tokens" in d:
            out.append([int(t) for t in d["tokens"]])
        elif tokenizer is None:
            raise ValueError("this model folder has no tokenizer: give token ids")
        else:
            out.append(list(tokenizer(d["prompt"])["input_ids"]))
    return out


def main(argv=None) -> int:
    a = build_parser().parse_args(argv)
    import torch

    from ..models.hf_io import load_pretrained
    from ..models.registry import architecture_of, read_config
    from ..ops import _lib
    from ..ops.attention import PAGE
    from ..rollout.engine import RolloutEngine, SamplingParams

    arch = architecture_of(read_config(a.model))
    if a.device.startswith("cuda"):
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device")
        if a.dtype == "float32" and not arch.fp32_on_gpu:
            raise ValueError("this model's kernels are bf16 only")
        if arch.component is not None:
            _lib.prefer_component(arch.component)
    tok = None
    if any(os.path.exists(os.path.join(a.model, f)) for f in ("tokenizer_config.json", "synthetic_tokenizer.json")):
        from ..utils.utils import get_tokenizer

        tok = get_tokenizer(a.model)
    lines = sys.stdin if a.input == "-" else open(a.input)
    prompts = read_prompts(lines, tok)
    if not prompts:
        return 0
    model = load_pretrained(a.model, device=a.device, dtype=getattr(torch, a.dtype))
    model.requires_grad_(False)
    longest = max(len(p) for p in prompts) + a.max_new_tokens + 1
    rows = max(a.n_samples, min(a.max_num_seqs, len(prompts) * a.n_samples))
    eng = RolloutEngine(model, max_num_seqs=rows, max_model_len=(longest + PAGE - 1) // PAGE * PAGE, seed=a.seed,
                        max_prefill_tokens=a.max_prefill_tokens)
    sp = SamplingParams(temperature=a.temperature, top_p=a.top_p, top_k=a.top_k, max_tokens=a.max_new_tokens,
                        n=a.n_samples, ignore_eos=a.ignore_eos, seed=a.seed)
    for i, ro in enumerate(eng.generate(prompts, sp)):
        for c in ro.outputs:
            d = {"prompt": i, "sample": c.index, "tokens": c.token_ids, "logprobs": c.logprob_values,
                 "finish_reason": c.finish_reason}
            if tok is not None:
                d["text"] = tok.decode(c.token_ids)
            print(json.dumps(d), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
