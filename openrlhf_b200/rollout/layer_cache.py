"""Per-layer caches of models whose layers differ (``cache_specs``): paged tensors with one entry per token of a page
(keys and values), and row tensors with one entry per engine row (recurrent state, convolution history). All of them
are slices of one buffer, so that the engine can place them in its VMM arena and drop them together when it sleeps."""
from __future__ import annotations

import math

import torch

_ALIGN = 256


class LayerCache:
    def __init__(self, specs, num_pages: int, page: int, rows: int, device):
        self.specs, self.page, self.device = list(specs), page, device
        self._place, off = {}, 0
        for layer, name, unit, shape, dtype in self.specs:
            assert unit in ("page", "row")
            full = ((num_pages * page if unit == "page" else rows),) + tuple(shape)
            nbytes = math.prod(full) * torch.empty(0, dtype=dtype).element_size()
            self._place[(layer, name)] = (off, nbytes, full, dtype, unit)
            off += (nbytes + _ALIGN - 1) // _ALIGN * _ALIGN
        self.nbytes = max(off, _ALIGN)
        self._t: dict = {}

    @staticmethod
    def bytes_per(specs, unit: str, page: int) -> int:
        """Bytes of one page (or one row) over all layers."""
        size = lambda shape, dt: math.prod(shape) * torch.empty(0, dtype=dt).element_size()
        return sum(size(shape, dt) * (page if unit == "page" else 1) for _, _, u, shape, dt in specs if u == unit)

    def bind(self, buf: torch.Tensor):
        """`buf`: uint8 buffer of at least ``nbytes``. Everything starts as zeros: a stale value row meets zero weights
        and must be finite."""
        assert buf.dtype == torch.uint8 and buf.numel() >= self.nbytes
        buf[:self.nbytes].zero_()
        self._t = {k: buf[o:o + nb].view(dt).view(full) for k, (o, nb, full, dt, _) in self._place.items()}

    def release(self):
        self._t = {}

    def get(self, layer: int, name: str) -> torch.Tensor:
        return self._t[(layer, name)]

    def copy_page(self, src: int, dst: int):
        P = self.page
        for k, t in self._t.items():
            if self._place[k][4] == "page":
                t[dst * P:(dst + 1) * P].copy_(t[src * P:(src + 1) * P])

    def copy_row(self, src: int, dst: list):
        for k, t in self._t.items():
            if self._place[k][4] == "row":
                for d in dst:
                    t[d].copy_(t[src])
