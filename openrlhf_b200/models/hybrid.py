"""Hybrid decoder (``HybridConfig``): every layer has a sequence mixer of its own kind and size, and mixer and
feed-forward are parallel: both read one RMS norm and both add to an fp32 residual stream.

That shape makes a layer two matrix products. ``w1`` stacks the mixer's input projections on the feed-forward's up
projection, ``w2`` puts the output projection beside the down projection, and what lies between (convolution,
recurrence and gate, or rotation and attention, plus the activation) fills one activation buffer that ``w2`` reads.

The model owns no cache and no loop: ``step`` runs one ragged batch (``StepBatch``: prompts, portions of prompts and
single tokens) against the per-layer caches that the rollout engine allocates from ``cache_specs``."""
from __future__ import annotations

import math

import torch

from ..ops import hybrid as H
from .flat import FlatModel, ParamSpec, SpecList
from .hybrid_config import AttentionSpec, HybridConfig, Mamba2Spec


def build_hybrid_specs(cfg: HybridConfig) -> list[ParamSpec]:
    layout = SpecList()
    W = cfg.width_pad
    layout.add("embed.weight", (cfg.vocab_size, W))
    for i, layer in enumerate(cfg.layers):
        p, m = f"layers.{i}.", layer.mixer
        layout.add(p + "norm1.weight", (W,), False, "ones")
        layout.add(p + "w1.weight", (layer.in_pad + layer.ff_pad, W))
        if isinstance(m, Mamba2Spec):
            layout.add(p + "conv.weight", (m.conv_channels, m.conv), False, "conv")
            layout.add(p + "conv.bias", (m.conv_channels,), False, "zeros")
            layout.add(p + "dt_bias", (m.heads,), False, "dt_bias")
            layout.add(p + "A_log", (m.heads,), False, "a_log")
            layout.add(p + "D", (m.heads,), False, "ones")
            layout.add(p + "gate_norm.weight", (m.inner,), False, "ones")
        layout.add(p + "w2.weight", (W, layer.out_pad + layer.ff_pad))
    layout.add("norm.weight", (W,), False, "ones")
    layout.add("lm_head.weight", (cfg.vocab_pad, W))
    return layout.specs


class HybridLM(FlatModel):
    def __init__(self, cfg: HybridConfig, device="cpu", dtype=torch.bfloat16, with_lm_head: bool = True,
                 with_value_head: bool = False, init_std: float = 0.02, seed: int | None = 0,
                 flat: torch.Tensor | None = None, shard_world: int = 1):
        super().__init__()
        if with_value_head or not with_lm_head:
            raise NotImplementedError("hybrid models are language models only (no value head)")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("hybrid models run in bfloat16 or float32")
        self.cfg, self.with_lm_head, self.with_value_head = cfg, True, False
        self.init_flat(build_hybrid_specs(cfg), device, dtype, flat, shard_world)
        self.lora = self.ep = self.tp_train = None
        self.requires_grad_(False)                # served only: there are no backward kernels
        self._max_pos = 0
        if seed is not None:
            self.reset_parameters(init_std, seed)
        self._bind()

    # ------------------------------------------------------------------ parameters
    def init_special(self, s: ParamSpec, p, g: torch.Generator) -> bool:
        if s.init not in ("conv", "dt_bias", "a_log"):
            return False
        u = torch.rand(s.shape, generator=g, device=p.device, dtype=torch.float32)
        if s.init == "conv":
            v = (2 * u - 1) / math.sqrt(s.shape[1])
        elif s.init == "a_log":
            v = (1 + 15 * u).log()                # decay rates between 1 and 16
        else:                                     # step sizes between 1e-3 and 1e-1 before the projection's share
            dt = (math.log(1e-3) + u * (math.log(1e-1) - math.log(1e-3))).exp()
            v = dt + torch.log(-torch.expm1(-dt))
        p.copy_(v)
        return True

    @torch.no_grad()
    def reset_parameters(self, std: float = 0.02, seed: int = 0):
        super().reset_parameters(std, seed)
        from .hf_io import _select

        for s, p in self.named_specs():           # the padding of fused matrices is zero
            keep = [(sel, _select(p, sel).clone()) for _, sel in self.cfg.checkpoint_names(s.name)]
            p.zero_()
            for sel, t in keep:
                _select(p, sel).copy_(t)

    def lm_head_weight(self) -> torch.Tensor:
        return self.p("lm_head.weight")

    def _bind(self):
        """Per-layer weight handles (views of the flat buffer: they follow in-place weight updates)."""
        self._mamba = {}
        for i, layer in enumerate(self.cfg.layers):
            if isinstance(layer.mixer, Mamba2Spec):
                q = lambda n: self.p(f"layers.{i}." + n)
                self._mamba[i] = H.Mamba2Weights(q("conv.weight"), q("conv.bias"), q("dt_bias"), q("A_log"), q("D"),
                                                 q("gate_norm.weight"))

    # ------------------------------------------------------------------ state
    def cache_specs(self):
        """What the engine keeps per layer: (layer, name, "page" or "row", shape per token or per row, dtype)."""
        dt = self.flat.dtype
        out = []
        for i, layer in enumerate(self.cfg.layers):
            m = layer.mixer
            if isinstance(m, Mamba2Spec):
                out.append((i, "ring", "row", (m.conv, m.conv_channels), dt))
                out.append((i, "state", "row", (m.heads, m.state, m.vdim), torch.float32))
            elif m.kv_from is None:
                out.append((i, "k", "page", (m.kv_heads, m.k_ld), dt))
                out.append((i, "v", "page", (m.kv_heads, m.v_ld), dt))
        return out

    def ensure_positions(self, max_pos: int):
        """Rotary tables reach at least this position (before any CUDA-graph capture)."""
        self._max_pos = max(self._max_pos, max_pos)
        for layer in self.cfg.layers:
            if isinstance(layer.mixer, AttentionSpec) and layer.mixer.rot_dims:
                self._table(layer.mixer)

    def _table(self, m: AttentionSpec):
        return H.rotary_table(m.rot_dims, m.rot_base, m.rot_factor, self._max_pos, self.flat.device) if m.rot_dims else None

    # ------------------------------------------------------------------ one step
    @torch.no_grad()
    def step(self, batch: H.StepBatch, cache, want: torch.Tensor | None = None, tap=None) -> torch.Tensor | None:
        """Run the batch's tokens. `want` int32: rows of the packed stream whose logits are returned (None: all rows; an
        empty tensor: no logits are computed and None is returned). `tap(layer, x)` sees the residual stream after every
        layer (debugging and tests)."""
        cfg, n, eps = self.cfg, self.cfg.hidden_size, self.cfg.norm_eps
        x = H.embed(batch.ids, self.p("embed.weight"))
        h = H.rmsnorm(x, self.p("layers.0.norm1.weight"), n, eps) if cfg.layers else None
        last = len(cfg.layers) - 1
        for i, layer in enumerate(cfg.layers):
            m = layer.mixer
            pre = f"layers.{i}."
            new = torch.empty if m.out_cols == layer.out_pad else torch.zeros
            a = new(batch.T, layer.out_pad + layer.ff_pad, dtype=h.dtype, device=h.device)
            p = H.project(h, self.p(pre + "w1.weight"), layer.in_pad, a[:, layer.out_pad:])
            ff = p.cols - layer.in_pad            # 0: the projection has already turned the feed-forward columns
            if isinstance(m, Mamba2Spec):
                H.mamba2(p, m, self._mamba[i], cache.get(i, "ring"), cache.get(i, "state"), batch, eps, a, layer.out_pad,
                         layer.in_pad, ff)
            else:
                src = i if m.kv_from is None else m.kv_from
                H.window_attention(p, m, self._table(m), cache.get(src, "k"), cache.get(src, "v"), batch, a, layer.out_pad,
                                   layer.in_pad, ff)
            # the norm that follows rides on the residual add (the last layer's too, when every row's logits are wanted)
            nxt = self.p(f"layers.{i + 1}.norm1.weight") if i < last else (self.p("norm.weight") if want is None else None)
            h = H.add_norm(x, a, self.p(pre + "w2.weight"), nxt, n, eps)
            if tap is not None:
                tap(i, x)
        if want is not None:
            if want.numel() == 0:
                return None
            h = H.rmsnorm(x, self.p("norm.weight"), n, eps, rows=want)
        elif not cfg.layers:
            h = H.rmsnorm(x, self.p("norm.weight"), n, eps)
        return H.head_logits(h, self.p("lm_head.weight"), cfg.vocab_size, cfg.logit_softcap)

    def forward(self, *_a, **_k):
        raise NotImplementedError("hybrid models run through the rollout engine (RolloutEngine), which owns their caches")
