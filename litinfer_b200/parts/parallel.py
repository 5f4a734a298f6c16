"""Two mixers side by side: both read the same input, the result is ``left_scale * left + right_scale * right``.

The two are parts of any registered kind (``left``, ``right`` in the spec, with their tensor-name prefixes below this
mixer's).  Each keeps what it needs between steps: the requirement of this mixer is the tuple of theirs, and the
cache it is handed has one part for each (``cache.parts``, in that order).  The weighted sum is taken in float32.

``out_norms`` (a mapping with the tensor names ``left`` and ``right`` below the prefix, and ``eps``): each output is first divided
by its root mean square and multiplied by a weight of the model's width.

Where both mixers offer their first product (``shared_projection`` / ``forward_projected``), it is one product over both
matrices; the left one's columns come first.
"""

from __future__ import annotations

import torch

from .. import kernels as K
from ..weights.loader import ParamSpec
from .base import MIXERS, Mixer


@MIXERS.register("parallel")
class ParallelMixer(Mixer):
    def __init__(self, spec, prefix, dtype, device):
        super().__init__(spec, prefix, dtype, device)
        prefixes = spec.get("prefixes", {})
        self.left = MIXERS.build(spec["left"], prefix + prefixes.get("left", "left."), dtype, device)
        self.right = MIXERS.build(spec["right"], prefix + prefixes.get("right", "right."), dtype, device)
        self.left_scale = float(spec.get("left_scale", 1.0))
        self.right_scale = float(spec.get("right_scale", 1.0))
        norms = spec.get("out_norms")
        self.norm_names = [prefix + str(norms[k]) for k in ("left", "right")] if norms else []
        self.norm_eps = float(norms["eps"]) if norms else 0.0
        self.hidden = int(spec["hidden_size"]) if norms else 0
        self.norms = None
        self.joined = None                  # the one first product of both, where they offer theirs
        self.ctas_per_work_unit = max(self.left.ctas_per_work_unit, self.right.ctas_per_work_unit)

    def parts(self):
        return [self.left, self.right]

    def params(self):
        return [ParamSpec(n, (self.hidden,), role="vector", init="ones_normal") for n in self.norm_names]

    def bind_all(self, tensors):
        super().bind_all(tensors)
        left, right = (getattr(m, "shared_projection", lambda: None)() for m in (self.left, self.right))
        if left is not None and right is not None:
            # (a bias of zeros where only the other has one)
            bias = None
            if left.bias is not None or right.bias is not None:
                bias = torch.cat([p.bias if p.bias is not None else torch.zeros(p.weight.shape[0], dtype=torch.float32, device=p.weight.device)
                                  for p in (left, right)]).contiguous()
            self.joined = (torch.cat([left.weight, right.weight], dim=0).contiguous(), bias, left.weight.shape[0])
            left.weight = right.weight = None

    def bind(self, tensors):
        if self.norm_names:
            self.norms = tuple(tensors.pop(n) for n in self.norm_names) + (self.norm_eps,)

    def cache_requirement(self):
        return (self.left.cache_requirement(), self.right.cache_requirement())

    def _caches(self, cache):
        """The parts of ``cache`` in the order of (left, right); a mixer that keeps nothing gets None."""
        it = iter(cache.parts)
        return [next(it) if m.cache_requirement() is not None else None for m in (self.left, self.right)]

    # forward_pair: the two outputs and their factors as they are, for a block whose write-back takes the sum in
    # (parts.block.HyperPreNormBlock); forward: the sum itself
    produces_pairs = True

    def forward_pair(self, h, ctx, cache) -> "K.WeightedPair":
        cl, cr = self._caches(cache)
        if self.joined is not None:
            weight, bias, col = self.joined
            proj = torch.empty((h.shape[0], weight.shape[0]), dtype=self.dtype, device=h.device)
            K.linear(h, weight, bias, proj)
            left, right = self.left.forward_projected(proj, 0, ctx, cl), self.right.forward_projected(proj, col, ctx, cr)
        else:
            left, right = self.left.forward(h, ctx, cl), self.right.forward(h, ctx, cr)
        return K.WeightedPair(left, right, self.left_scale, self.right_scale, self.norms)

    def forward(self, h, ctx, cache):
        return self.forward_pair(h, ctx, cache).materialize()
