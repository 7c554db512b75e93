"""Serving throughput of the hybrid design beside the dense transformer of equal size (``python bench.py --serving``).

For every size: prefill tokens/s of whole prompts and decode tokens/s of a full batch, both through the rollout engine's
own step functions (prefill: one ragged batch, last-position logits; decode: captured CUDA graphs, sampling included),
random weights, device time by CUDA events. The dense model has the same width, depth, attention heads and vocabulary
and as many parameters (its feed-forward makes up the difference). Weights and caches exceed L2."""
from __future__ import annotations

import statistics

import torch

SIZES = {"1b": "sigisun-1b", "3b": "sigisun-3b", "8b": "sigisun-8b"}


def dense_twin(cfg):
    """TransformerLM configuration of the same width, depth, heads, vocabulary and (nearly) parameter count."""
    from openrlhf_b200.models.config import ModelConfig
    from openrlhf_b200.models.hybrid_config import AttentionSpec

    a = next(layer.mixer for layer in cfg.layers if isinstance(layer.mixer, AttentionSpec))
    L, W = cfg.num_hidden_layers, cfg.hidden_size
    twin = ModelConfig("llama", cfg.vocab_size, W, 128, L, a.heads, a.kv_heads, head_dim=128)
    per_ff = 3 * W * L
    twin.intermediate_size = max(128, round((cfg.num_params() - twin.num_params() + per_ff * 128) / per_ff / 128) * 128)
    return twin


def _events(fn, warmup: int, steps: int) -> float:
    """Median milliseconds of one call."""
    ms = []
    for k in range(warmup + steps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        if k >= warmup:
            ms.append(e0.elapsed_time(e1))
    return statistics.median(ms)


def measure(cfg, prompts, decode, warmup: int, steps: int) -> dict:
    """prompts: list of (sequences, tokens each); decode: list of (batch, context)."""
    from openrlhf_b200.models.registry import build_model
    from openrlhf_b200.ops import _lib
    from openrlhf_b200.rollout.engine import RolloutEngine, SamplingParams, _Row

    model = build_model(cfg, device="cuda", seed=0)
    model.requires_grad_(False)
    out = {"params": cfg.num_params(), "prefill": [], "decode": []}
    g = torch.Generator().manual_seed(0)
    ids = lambda n: torch.randint(3, cfg.vocab_size, (n,), generator=g).tolist()
    for n, L in prompts:
        eng = RolloutEngine(model, max_num_seqs=n, max_model_len=L + 128, num_pages=n * (L // 128 + 1) + 1)
        for i in range(n):
            eng.rows[i] = _Row(i, 0, L, 0, [], prefilled=0)
            eng._ensure_pages(i, L - 1)
        items = [(ids(L), 0, i) for i in range(n)]
        ms = _events(lambda: eng._prefill(items), warmup, steps)
        out["prefill"].append({"sequences": n, "tokens_each": L, "ms": round(ms, 3), "tokens_per_s": round(n * L / ms * 1e3)})
        del eng
    for B, ctx in decode:
        interval, bursts = 4, max(2, steps // 8)
        chunks = (B * ctx + 16383) // 16384
        new = interval * (8 * (bursts + 5) + chunks + 4)
        eng = RolloutEngine(model, max_num_seqs=B, max_model_len=ctx + new + 128, num_pages=B * ((ctx + new) // 128 + 2) + 8,
                            check_interval=interval)
        sp = SamplingParams(temperature=1.0, max_tokens=new, ignore_eos=True)
        for i in range(B):
            eng.add_request(i, ids(ctx), sp)
        ready = 0
        for _ in range(chunks + 8):                    # prefill of every row, graph capture, warm-up bursts
            eng.step()
            ready += sum(r is not None and r.prefilled < 0 for r in eng.rows) == B
            if ready == 3:
                break
        assert ready == 3
        torch.cuda.synchronize()
        d0, l0 = eng.decode_steps, _lib.LAUNCHES
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(bursts):
            eng.step()
        e1.record()
        torch.cuda.synchronize()
        n = eng.decode_steps - d0
        ms = e0.elapsed_time(e1) / n
        out["decode"].append({"batch": B, "context": ctx, "ms_per_step": round(ms, 4), "tokens_per_s": round(B / ms * 1e3),
                              "launches_per_step": (_lib.LAUNCHES - l0) // n})
        eng.sleep()
        del eng
        torch.cuda.empty_cache()
    _lib.check_status()
    del model
    torch.cuda.empty_cache()
    return out


def run(sizes, warmup: int, steps: int) -> dict:
    from openrlhf_b200.models.config import PRESETS

    res = {}
    for s in sizes:
        cfg = PRESETS[SIZES[s]]
        prompts, decode = [(4, 2048), (1, 8192)], [(128, 2048), (16, 2048)]
        res[s] = {"sigisun": measure(cfg, prompts, decode, warmup, steps),
                  "dense": measure(dense_twin(cfg), prompts, decode, warmup, steps)}
    return res
