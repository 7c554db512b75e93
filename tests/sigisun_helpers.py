"""Small configurations of the Sigisun architecture, checkpoints with random weights, and drivers that feed sequences
through the rollout engine in chosen portions."""
import json
import os

import torch
from safetensors.torch import save_file

import sigisun_oracle as O


def mamba(heads, vdim, state, groups=1, conv=4, norm_groups=1, ff=None):
    m = dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)
    return {"type": "mamba2", "mixer": m, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def attn(heads, kv_heads, dim, vdim, scale, size, keep, rot=None, base=10000.0, factor=4.0, kv_from=None, ff=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask={"size": size, "keep_first": keep},
             rot={"dims": dim if rot is None else rot, "base": base, "scaling": {"factor": factor}})
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def config(layers, width=72, vocab=203, eps=1e-5, cap=20.0):
    return {"architecture": "Sigisun", "layers": layers, "logit_softcap": cap, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


CONFIGS = {
    # both kinds of layer, groups and norm groups above 1, a shared cache with another mask, a layer without feed-forward
    "mix": config([mamba(6, 16, 32, 2, 4, 3, 100), attn(6, 2, 40, 24, 0.2, 37, 3, 16, ff=88), mamba(4, 24, 16, 1, 3, 1),
                   attn(6, 2, 40, 24, 0.15, 130, 1, 16, 500.0, 2.0, kv_from=1, ff=64), mamba(2, 64, 128, 1, 2, 2, 60)]),
    # sizes that are no multiples of anything, one tap, one head, one kept token
    "odd": config([mamba(5, 7, 11, 5, 1, 5, 31), attn(3, 1, 22, 13, 0.3, 5, 1, 6, 100.0, 1.0, ff=17),
                   attn(3, 3, 10, 6, 0.5, 9, 0, 2, ff=9), mamba(1, 9, 8, 1, 5, 1, 12)], width=37, vocab=101, eps=1e-3, cap=7.0),
    # attention first, window of one page and of one token, value heads wider than key heads, whole head rotates
    "attn": config([attn(8, 2, 32, 64, 0.18, 128, 2, ff=96), attn(4, 4, 64, 32, 0.125, 1, 4, 32),
                    attn(8, 2, 32, 64, 0.18, 65, 130, kv_from=0, ff=32), mamba(3, 32, 48, 3, 6, 1, 40)], width=64, vocab=160,
                   cap=50.0),
    # recurrent only
    "ssm": config([mamba(4, 32, 64, 2, 4, 2, 48), mamba(8, 8, 16, 4, 4, 4)], width=48, vocab=97),
}


def write_checkpoint(path, cfg, seed=0, weights=None):
    os.makedirs(path, exist_ok=True)
    w = O.random_weights(cfg, seed) if weights is None else weights
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    return w


def make_engine(path, device, dtype, rows=4, max_len=1024, pages=None, **kw):
    from openrlhf_b200.models.hf_io import load_pretrained
    from openrlhf_b200.rollout.engine import RolloutEngine

    model = load_pretrained(str(path), device=device, dtype=dtype)
    return RolloutEngine(model, max_num_seqs=rows, max_model_len=max_len,
                         num_pages=pages if pages is not None else rows * (max_len // 128) + 2, **kw)


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def feed(eng, toks, cuts, key="s"):
    """Logits at every position of one sequence fed in portions of the given sizes (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = cuts[min(k, len(cuts) - 1)]
        part = toks[at:at + n]
        out.append(eng.extend([(key, part, list(range(len(part))))]).cpu())
        at += len(part)
        k += 1
    eng.finish(key)
    return torch.cat(out)


def rel_rms(got, want, quantile=1.0):
    """Root mean square over the vocabulary of the difference (mean taken off), over the logits' own spread: worst row, or
    a quantile of the rows. (In bf16 a few positions of a random model amplify rounding, wherever its kernels run.)"""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).quantile(quantile))
