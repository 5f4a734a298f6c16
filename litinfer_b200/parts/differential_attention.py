"""Differential attention: two attention maps per head over the same values, the second taken off the first.

With the mixer's input h, H query heads and G key/value heads (query head a reads key/value head ``a // (H / G)``), two
queries and two keys of ``head_dim`` elements per head, laid out head by head as (map 1 | map 2), and ``value_dim`` values:

    q = W_q h, k = W_k h, v = W_v h              (biases if ``qkv_bias``; no positions enter)
    s^m_ij = scale * q^m_i . k^m_j               for j in the window of i (i itself and the ``window - 1`` tokens before it)
    s <- softcap * tanh(s / softcap)             (``softcap``; optional)
    a^m_i = sum_j softmax(s^m_i)_j v_j           m = 1, 2
    mix = exp(lq1 . lk1) - exp(lq2 . lk2) + diff  one number for the layer; lq1 ... are stored vectors of head_dim elements
    o_i = a^1_i - mix a^2_i;  o_i <- o_i / sqrt(mean(o_i^2) + eps) (1 - diff)   per head, no weight
    output W_o (o * sigmoid(W_g h))              heads side by side; the gate (``gate``) is optional, element by element

How a step runs it: the two keys of a head lie side by side in one cached key row of ``2 head_dim`` elements, so the cache
holds every value once and the attention kernels see G key/value heads.  A query row holds the two queries the same way and
stands for two heads of the attention (``kernels.paged_attention(..., maps=2)``): each takes its half of the query against its
half of the key.  The cache's head size is the larger of ``2 head_dim`` and ``value_dim``, rounded up to a multiple of 16;
queries, keys and values are padded with zero rows of their matrices, which changes no sum.  One kernel behind attention takes
the difference, the norm and the gate (``kernels.map_difference``).  Scores, softmax, difference, norm and gate are float32.
"""

from __future__ import annotations

from typing import Dict, List

import torch

from .. import kernels as K
from ..weights.loader import ParamSpec
from .base import MIXERS, Mixer, PagedKV
from .linear import FusedLinear, undefer

MAPS = 2


@MIXERS.register("differential_attention")
class DifferentialAttention(Mixer):
    takes_deferred = True            # both products of the input apply the factor

    def __init__(self, spec, prefix, dtype, device):
        super().__init__(spec, prefix, dtype, device)
        self.hidden = int(spec["hidden_size"])
        self.num_heads = int(spec["num_heads"])
        self.num_kv_heads = int(spec["num_kv_heads"])
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} heads are not a multiple of {self.num_kv_heads} key/value heads")
        self.qk_dim = int(spec["head_dim"])
        self.value_dim = int(spec["value_dim"])
        self.head_dim = -(-max(MAPS * self.qk_dim, self.value_dim) // 16) * 16          # the cache's head size
        self.ctas_per_work_unit = MAPS * self.num_heads
        self.scale = float(spec["scale"])
        self.softcap = float(spec.get("softcap") or 0.0)
        self.window = spec.get("window")
        self.eps = float(spec["eps"])
        self.diff = float(spec["diff"])
        n = dict(spec.get("names", {}))
        suffixes = tuple(spec.get("suffixes", (".weight", ".bias")))
        H, G = self.num_heads, self.num_kv_heads
        self.qkv = FusedLinear(prefix, [n.get("q", "q_proj"), n.get("k", "k_proj"), n.get("v", "v_proj")], self.hidden,
                               [H * MAPS * self.qk_dim, G * MAPS * self.qk_dim, G * self.value_dim], bool(spec.get("qkv_bias", False)), dtype,
                               suffixes=suffixes)
        gate = spec.get("gate")
        self.gate = FusedLinear(prefix, [gate], self.hidden, [H * self.value_dim], False, dtype, suffixes=suffixes) if gate else None
        self.out = FusedLinear(prefix, [n.get("o", "o_proj")], H * self.value_dim, [self.hidden], False, dtype, suffixes=suffixes)
        self.mix_names = [prefix + n.get(k, k) for k in ("lq1", "lk1", "lq2", "lk2")]
        self.mix = 0.0
        self.weight = self.bias = None                   # what the first product reads, made when the weights are bound
        self.joined = False

    def params(self) -> List[ParamSpec]:
        return (self.qkv.params() + (self.gate.params() if self.gate is not None else []) + self.out.params()
                + [ParamSpec(name, (self.qk_dim,), role="vector", std=0.1) for name in self.mix_names])

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.qkv.bind(tensors)
        if self.gate is not None:
            self.gate.bind(tensors)
        self.out.bind(tensors)
        lq1, lk1, lq2, lk2 = (tensors.pop(name).float() for name in self.mix_names)
        self.mix = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + self.diff
        if self.head_dim != MAPS * self.qk_dim or self.head_dim != self.value_dim:
            self._pad_heads()
        # a gate whose heads are as wide as the cache's joins the q|k|v product (its rows behind them, with a bias of zeros)
        self.joined = self.gate is not None and self.value_dim == self.head_dim
        self.weight, self.bias = self.qkv.weight, self.qkv.bias
        if self.joined:
            self.weight = torch.cat([self.qkv.weight, self.gate.weight], dim=0).contiguous()
            if self.bias is not None:
                self.bias = torch.cat([self.bias, torch.zeros(self.gate.out_features, dtype=self.bias.dtype, device=self.bias.device)]).contiguous()
            self.qkv.weight = self.gate.weight = None

    def _pad_heads(self) -> None:
        """Zero rows of q, k and v (with their biases) up to the cache's head size, behind each map's queries and keys."""
        H, G, D = self.num_heads, self.num_kv_heads, self.head_dim
        shapes = ((H * MAPS, self.qk_dim, D // MAPS), (G * MAPS, self.qk_dim, D // MAPS), (G, self.value_dim, D))
        cuts = tuple(n * d for n, d, _ in shapes)

        def pad(t):
            pieces = []
            for piece, (n, d, to) in zip(torch.split(t, cuts, dim=0), shapes):
                full = torch.zeros((n, to) + tuple(t.shape[1:]), dtype=t.dtype, device=t.device)
                full[:, :d] = piece.view(n, d, *t.shape[1:])
                pieces.append(full.view(n * to, *t.shape[1:]))
            return torch.cat(pieces, dim=0).contiguous()

        self.qkv.weight = pad(self.qkv.weight)
        if self.qkv.bias is not None:
            self.qkv.bias = pad(self.qkv.bias)
        self.qkv.out_features = self.qkv.weight.shape[0]

    def cache_requirement(self):
        return PagedKV(self.num_kv_heads, self.head_dim, self.window)

    def forward(self, h, ctx, cache):
        return self.out(self._attend(h, ctx, cache))

    def forward_into(self, h, ctx, cache, tail):
        return tail.apply_linear(self.out, self._attend(h, ctx, cache))

    def _attend(self, h, ctx, cache):
        """Everything before the output projection: [tokens, heads * value_dim]."""
        H, G, D = self.num_heads, self.num_kv_heads, self.head_dim
        view = ctx.group(cache.group)
        gate = self.gate(h) if self.gate is not None and not self.joined else None
        h, row_scale = undefer(h, self.weight)
        T = h.shape[0]
        if self.joined:
            gate = torch.empty((T, H * D), dtype=self.dtype, device=h.device)
        qkv = torch.empty((T, (H + 2 * G) * D), dtype=self.dtype, device=h.device)
        # projection (with the gate's) and keys and values into the cache: one call (and for few tokens one kernel)
        K.linear_rope_kv(h, self.weight, self.bias, qkv, ctx.positions, None, 0, view.slot_mapping, cache.k, cache.v, H, G, D, cache.writes,
                         row_scale=row_scale, extra=gate if self.joined else None)
        both = torch.empty((T, MAPS * H * D), dtype=self.dtype, device=h.device)
        K.paged_attention(
            qkv, both, cache.k, cache.v, view.block_table, ctx.q_start, ctx.ctx_lens, ctx.seq_of_token, ctx.positions,
            MAPS * H, G, D, self.scale, self.window, ctx.max_q_len, ctx.max_ctx_len, old_lens=ctx.old_lens, singles=ctx.num_single,
            units=ctx.attn_units, unit_slots=ctx.attn_unit_slots, softcap=self.softcap, maps=MAPS)
        o = torch.empty((T, H * self.value_dim), dtype=self.dtype, device=h.device)
        K.map_difference(both, D, gate, 0, self.mix, self.eps, 1.0 - self.diff, o, H, self.value_dim)
        return o
