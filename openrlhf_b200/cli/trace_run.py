"""``bin/trace_run`` / ``python -m openrlhf.cli.trace_run``: replay a trace of given tokens through the rollout engine.

Steps come as JSON lines on standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

every step is one batch of the engine (``RolloutEngine.extend``), and the logits at the wanted places are written to
``OUT/<step>.f32`` as little-endian float32 rows. After a step the line ``done <step>`` is printed. "end" lists the
sequences whose pages and state are given back after the step."""
from __future__ import annotations

import argparse
import json
import os
import sys

ROWS = 4                 # sequences that may be live at once
EXIT_NO_FLOAT32 = 3


def build_parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights, or a preset name")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live sequences hold at any time")
    return ap


def make_engine(model_path: str, dtype: str, max_tokens: int, device: str = "cuda"):
    """Model and engine whose pool holds `max_tokens` tokens of at most ROWS sequences."""
    import torch

    from ..models.hf_io import load_pretrained
    from ..ops.attention import PAGE
    from ..rollout.engine import RolloutEngine

    model = load_pretrained(model_path, device=device, dtype=getattr(torch, dtype))
    model.requires_grad_(False)
    # one page backs idle rows; a sequence's last page may be half used
    pages = (max_tokens + PAGE - 1) // PAGE + ROWS // 2 + 1
    return RolloutEngine(model, max_num_seqs=ROWS, max_model_len=(max_tokens + PAGE - 1) // PAGE * PAGE, num_pages=pages)


def replay(engine, steps, out: str, done=print) -> None:
    """Run the steps (an iterable of JSON lines) and write the wanted logits."""
    for line in steps:
        if not line.strip():
            continue
        st = json.loads(line)
        logits = engine.extend([(e["id"], e["tokens"], e.get("want", [])) for e in st.get("entries", [])])
        if logits is not None:
            path = os.path.join(out, f"{st['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(logits.contiguous().cpu().numpy().astype("<f4").tobytes())
            os.replace(path + ".part", path)
        for key in st.get("end", []):
            engine.finish(key)
        done(f"done {st['step']}", flush=True)


def main(argv=None) -> int:
    a = build_parser().parse_args(argv)
    from ..models.registry import architecture_of, read_config

    arch = architecture_of(read_config(a.model))
    if a.dtype == "float32" and not arch.fp32_on_gpu:
        print("trace_run: this model's kernels are bf16 only", file=sys.stderr)
        return EXIT_NO_FLOAT32
    import torch

    if not torch.cuda.is_available():
        raise RuntimeError("trace_run needs a CUDA device")
    from ..ops import _lib

    if arch.component is not None:
        _lib.prefer_component(arch.component)
    replay(make_engine(a.model, a.dtype, a.max_tokens), sys.stdin, a.out)
    return 0


if __name__ == "__main__":
    sys.exit(main())
