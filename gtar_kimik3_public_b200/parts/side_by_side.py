"""Two mixers side by side: both read the same input, and the result is ``left_scale * left(x) + right_scale * right(x)``
(the sum formed in 32-bit).  The two keep what they need between steps independently: the pair's cache request is the
list of both mixers' requests, the left one's first.  Their tensors sit under the prefixes ``left.`` and ``right.``.

Where both are mixers of one packed input product and one output product (``ProjectedMixer``), the pair makes two products
and not four: the input matrices stand one above the other, the read-outs, each already times its mixer's scale, side by side in
one row, and the output matrices side by side, so that the second product is the sum."""

from __future__ import annotations

import torch

from ..ops import functional as F
from ..ops.linear import linear
from .base import Mixer, ProjectedMixer, StepContext, register_part


def _as_list(request) -> list:
    if request is None:
        return []
    return list(request) if isinstance(request, (list, tuple)) else [request]


def _up8(n: int) -> int:
    return -(-n // 8) * 8


class SideBySide(Mixer):
    def __init__(self, left: Mixer, right: Mixer, left_scale: float = 1.0, right_scale: float = 1.0,
                 names: dict[str, str] | None = None):
        self.left, self.right, self.left_scale, self.right_scale = left, right, float(left_scale), float(right_scale)
        self.names = {"left": "left.", "right": "right.", **(names or {})}
        self.w_in = self.w_o = None  # of both, where they are packed
        self.right_at = 0

    @property
    def graph_safe(self) -> bool:
        return self.left.graph_safe and self.right.graph_safe

    def children(self):
        return [(self.names["left"], self.left), (self.names["right"], self.right)]

    def tensor_specs(self):
        return {prefix + name: spec for prefix, part in self.children() for name, spec in part.tensor_specs().items()}

    def load(self, tensors):
        for prefix, part in self.children():
            part.load({name: tensors[prefix + name] for name in part.tensor_specs() if prefix + name in tensors})
        pair = (self.left, self.right)
        if (all(isinstance(part, ProjectedMixer) and part.packable for part in pair) and self.left.w_in.dtype == self.right.w_in.dtype
                and self.left.w_o.dtype == self.right.w_o.dtype):
            self.right_at = self.left.w_in.shape[0]
            self.w_in = torch.cat([part.w_in for part in pair], dim=0).contiguous()
            # each mixer's read-outs begin at a multiple of 8 columns; no read-out stands in the columns between
            self.read_at = [0, _up8(self.left.out_columns)]
            self.read_columns = self.read_at[1] + _up8(self.right.out_columns)
            w_o = self.left.w_o.new_zeros((self.left.w_o.shape[0], self.read_columns))
            for part, at in zip(pair, self.read_at):
                w_o[:, at:at + part.out_columns] = part.w_o
            self.w_o = w_o
            for part in pair:  # held here from now on
                part.w_in = part.w_o = None

    def weight_bytes(self):
        own = sum(t.numel() * t.element_size() for t in (self.w_in, self.w_o) if t is not None)
        return own + self.left.weight_bytes() + self.right.weight_bytes()

    def cache_request(self):
        return _as_list(self.left.cache_request()) + _as_list(self.right.cache_request())

    @staticmethod
    def _views(request, views: list):
        """The storage of one of the two, in the form its own request has: one view, None, or a tuple."""
        if request is None:
            return None
        if isinstance(request, (list, tuple)):
            return tuple(views.pop(0) for _ in request)
        return views.pop(0)

    def forward(self, x, ctx: StepContext, cache):
        views = list(cache) if isinstance(cache, (list, tuple)) else ([] if cache is None else [cache])
        left_views = self._views(self.left.cache_request(), views)
        right_views = self._views(self.right.cache_request(), views)
        if self.w_in is not None:
            proj = linear(x, self.w_in)
            gaps = self.read_columns > self.left.out_columns + self.right.out_columns
            rows = (torch.zeros if gaps else torch.empty)((ctx.n_tokens, self.read_columns), dtype=ctx.dtype, device=x.device)
            self.left.core(proj, 0, ctx, left_views, rows, self.read_at[0], self.left_scale)
            self.right.core(proj, self.right_at, ctx, right_views, rows, self.read_at[1], self.right_scale)
            return linear(rows, self.w_o)
        left = self.left.forward(x, ctx, left_views)
        right = self.right.forward(x, ctx, right_views)
        return F.scaled_sum(left, self.left_scale, right, self.right_scale)


register_part("mixer", "side_by_side", SideBySide)
