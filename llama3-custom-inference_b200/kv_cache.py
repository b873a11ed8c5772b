"""Static per-layer caches of a decoder and the requests that occupy their rows.

A layer's cache is a set of named planes, each a dense tensor [max_batch, max_len, *shape]: keys and values of an
attention layer ({"k": (heads, size), "v": (heads, size)}), the one row per token of a latent-attention layer
({"latent": (width,)}).  A plane given as `State(shape, dtype)` holds one value per sequence instead of one per token, dense
[max_batch, *shape]: the matrix state of a recurrent layer, the inputs a short convolution still needs.  Batch row b of every plane belongs to sequence b of a batch (`DecodeLoop.generate`) or, when
requests come and go (`DecodeLoop.extend`), to the request that holds slot b.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


@dataclass(frozen=True)
class State:
    """A plane per sequence; dtype None: the cache's type.  A kernel that carries it starts from zero at position 0, whatever
    the row holds."""
    shape: tuple
    dtype: Optional[torch.dtype] = None


class StaticCache:
    def __init__(self, planes: list, max_batch: int, max_len: int, dtype, device):
        self.max_batch, self.max_len = max_batch, max_len

        def plane(p):
            if isinstance(p, State):
                return torch.zeros(max_batch, *p.shape, dtype=p.dtype or dtype, device=device)
            return torch.zeros(max_batch, max_len, *p, dtype=dtype, device=device)

        self.layers = [{name: plane(p) for name, p in layer.items()} for layer in planes]
        self._free = list(range(max_batch - 1, -1, -1))
        self._slot: dict = {}
        self._length: dict = {}

    # ---- requests -----------------------------------------------------------------------------------------
    def slot(self, request) -> int:
        """The request's slot; its first use takes a free one.  What an earlier holder left in the rows is never
        read: a query sees the positions up to its own, which the request has written by then, and a recurrent layer starts
        from zero at position 0."""
        if request not in self._slot:
            if not self._free:
                raise RuntimeError(f"no free slot: {self.max_batch} requests are live")
            self._slot[request] = self._free.pop()
            self._length[request] = 0
        return self._slot[request]

    def length(self, request) -> int:
        """Tokens of the request that are cached."""
        return self._length.get(request, 0)

    def advance(self, request, tokens: int) -> None:
        self._length[request] += tokens

    def release(self, request) -> None:
        """Gives the request's slot back."""
        if request in self._slot:
            self._free.append(self._slot.pop(request))
            del self._length[request]
