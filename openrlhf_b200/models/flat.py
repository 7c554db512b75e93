"""Base of every model definition here: all parameters are views into one flat buffer (the unit of ZeRO sharding, weight
sync and checkpointing), laid out by a list of ``ParamSpec``."""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch
import torch.nn as nn

ALIGN = 128  # every parameter starts on a 256-byte boundary of the flat buffer (TMA needs 16 B; shards like 256 B)


@dataclass
class ParamSpec:
    name: str
    shape: tuple
    offset: int
    numel: int
    decay: bool       # subject to weight decay (matrices) or exempt (norms, biases)
    init: str         # normal | ones | zeros | a model's own kinds (``FlatModel.init_special``)


class SpecList:
    """Collects parameter specs with aligned offsets."""

    def __init__(self):
        self.specs: list[ParamSpec] = []
        self._off = 0

    def add(self, name, shape, decay=True, init="normal"):
        n = math.prod(shape)
        self.specs.append(ParamSpec(name, tuple(shape), self._off, n, decay, init))
        self._off += (n + ALIGN - 1) // ALIGN * ALIGN


class FlatModel(nn.Module):
    def init_flat(self, specs: list[ParamSpec], device, dtype, flat: torch.Tensor | None, shard_world: int):
        self.specs = specs
        total = specs[-1].offset + (specs[-1].numel + ALIGN - 1) // ALIGN * ALIGN
        if flat is None:
            # room for the padding that makes the flat index space divisible into `shard_world` aligned shards
            per = ((total + shard_world - 1) // shard_world + 255) // 256 * 256
            flat = torch.zeros(per * shard_world, dtype=dtype, device=device)
        assert flat.numel() >= total
        self.flat = flat                      # not a Parameter: parameters are views into it
        self.total_numel = total
        self._params: dict[str, nn.Parameter] = {}
        for s in specs:
            view = flat[s.offset:s.offset + s.numel].view(s.shape)
            p = nn.Parameter(view, requires_grad=True)
            self._params[s.name] = p
            self.register_parameter(s.name.replace(".", "__"), p)

    def p(self, name: str) -> nn.Parameter:
        return self._params[name]

    def named_specs(self):
        return [(s, self._params[s.name]) for s in self.specs]

    def init_special(self, spec: ParamSpec, p: nn.Parameter, g: torch.Generator) -> bool:
        """Initialise a parameter that is neither constant nor N(0, std); True when handled."""
        return False

    @torch.no_grad()
    def reset_parameters(self, std: float = 0.02, seed: int = 0):
        g = torch.Generator(device=self.flat.device).manual_seed(seed)
        for s, p in self.named_specs():
            if s.init == "ones":
                p.fill_(1.0)
            elif s.init == "zeros":
                p.zero_()
            elif self.init_special(s, p, g):
                continue
            else:
                # chunked to bound the fp32 temporary for large embeddings
                flat = p.view(-1)
                step = 1 << 26
                for a in range(0, flat.numel(), step):
                    b = min(flat.numel(), a + step)
                    flat[a:b].copy_(torch.randn(b - a, generator=g, device=p.device, dtype=torch.float32) * std)
