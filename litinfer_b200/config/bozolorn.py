"""Configuration of the Bozolorn decoder, read from config.json.

config.json names the design under ``architecture`` and lists the layers one by one: each entry gives its ``type``
(which mixer it has), the mixer's sizes (``mixer``) and its feed-forward (``mlp``, or null for none).  Model-wide keys:
``vocab``, ``width``, ``norm.eps``, ``embedding.scale`` (a factor on the token embedding) and ``token_side.dim``.

A sublayer stands between two RMS norms: ``x += norm1b(mixer(norm1(x)))``, then ``x += norm2b(ff(norm2(x)))``.  Behind them every
layer adds something of the token itself (``token_side``): its ``dim`` columns of the token's row of one table, opened by a gate
that reads the stream, mapped to the width and normed.

Layer types:

* ``attention``: grouped-query softmax attention without positions but for a penalty per head that grows with the distance
  (``2^(-8 (h + 1) / heads)`` a position), in chunks of ``mask.size`` positions, with a gate per output element.  With
  ``kv_from``: j the layer has no keys and values of its own and reads the cache of layer j.
* ``parallel``: two mixers over the same input, half the sum of their outputs, each normed over the width.  ``left``: grouped-query
  causal attention with biased projections, an RMS norm per query and key head, rotation of the first ``rot.dims`` elements
  (pairs of neighbours, base ``rot.base``, frequencies blended by the pair's index with ``rot.scaling``: factor, original, fast,
  slow) and a denominator that is one larger.  ``right``: the gated delta rule with one decay per head (``heads``, ``kv_heads``,
  ``dim``, ``vdim``, ``conv`` taps) and a full gate with silu.

The feed-forward (``kind`` moe) is a mixture of ``router.experts`` gated units with bounded operands (``expert.ff``,
``expert.limit``; the unit's 1.702 is the design's): sigmoid scores, a stored correction on the choice scores, ``router.groups``
(``count``, ``keep``; a group counts as its two best), ``router.top`` choices, whose weights are their scores as they are.

Tensor names follow the file: ``l<i>.`` per layer, ``mix.`` / ``mlp.`` / ``side.`` / ``norm1`` / ``norm1b`` / ``norm2`` /
``norm2b`` below it, weights under the bare stem and biases under ``<stem>.b``.  Sizes and constants all come from config.json.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .filasun import _float, _int
from .gorulorn import MAX_POSITIONS, SUFFIXES, _opt_int
from .pifazen import GLU_ALPHA
from .qwen2 import ConfigError
from .spec import BlockSpec, ModelSpec, PartSpec, ScheduleEntry

TOKEN_TABLE = "side.embed"


def distance_slopes(heads: int) -> Tuple[float, ...]:
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


@dataclass(frozen=True)
class BozolornConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[Mapping[str, Any], ...]
    side_dim: int = 0                                     # 0: layers add nothing of the token
    max_positions: int = MAX_POSITIONS

    ARCHITECTURE = "Bozolorn"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BozolornConfig":
        norm = d.get("norm")
        if not isinstance(norm, Mapping):
            raise ConfigError("config.json: missing key 'norm' (with 'eps')")
        eps = _float(norm, "eps", "norm.")
        if eps <= 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps}")
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        emb, side = d.get("embedding") or {}, d.get("token_side")
        if not isinstance(emb, Mapping):
            raise ConfigError("config.json: 'embedding' must be an object ('scale')")
        if side is not None and not isinstance(side, Mapping):
            raise ConfigError("config.json: 'token_side' must be an object with 'dim'")
        cfg = cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), eps=eps, embedding_scale=_float(emb, "scale", "embedding.", 1.0),
                  layers=tuple(layers), side_dim=_int(side, "dim", "token_side.") if side is not None else 0,
                  max_positions=_int(d, "max_positions", "") if d.get("max_positions") is not None else MAX_POSITIONS)
        cfg.to_model_spec()                       # every layer's keys are read (and refused) here, not at the first step
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                               "embedding": {"scale": self.embedding_scale}, "layers": [dict(x) for x in self.layers]}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        if self.max_positions != MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    # ------------------------------------------------------------------
    def _heads(self, m: Mapping[str, Any], where: str) -> Tuple[int, int]:
        heads = _int(m, "heads", where)
        kv = _opt_int(m, "kv_heads", where) or heads
        if heads % kv:
            raise ConfigError(f"config.json: {where}{heads} heads are not a multiple of {kv} key/value heads")
        return heads, kv

    def _rotation(self, m: Mapping[str, Any], dim: int, where: str) -> Optional[PartSpec]:
        rot = m.get("rot")
        if rot is None:
            return None
        if not isinstance(rot, Mapping):
            raise ConfigError(f"config.json: {where}'rot' must be an object with 'dims' and 'base'")
        dims = _int(rot, "dims", where + "rot.")
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}rot.dims {dims} must be even and at most dim {dim}")
        params: Dict[str, Any] = {"theta": _float(rot, "base", where + "rot."), "rotary_dim": dims, "pairing": "interleaved"}
        sc = rot.get("scaling")
        if sc is not None:
            keys = ("factor", "original", "fast", "slow")
            if not isinstance(sc, Mapping):
                raise ConfigError(f"config.json: {where}rot.'scaling' must be an object with {', '.join(keys)}")
            params["scaling"] = dict({k: _float(sc, k, where + "rot.scaling.") for k in keys}, kind="yarn")
            if min(params["scaling"][k] for k in keys) <= 0:
                raise ConfigError(f"config.json: {where}rot.scaling needs factor, original, fast and slow > 0")
        return PartSpec("rope", params)

    def _attention(self, m: Mapping[str, Any], where: str) -> PartSpec:
        heads, kv = self._heads(m, where)
        dim = _int(m, "dim", where)
        mask = m.get("mask")
        if mask is not None and not isinstance(mask, Mapping):
            raise ConfigError(f"config.json: {where}'mask' must be an object with 'size'")
        return PartSpec("attention", {
            "hidden_size": self.width, "num_heads": heads, "num_kv_heads": kv, "head_dim": dim, "value_dim": _opt_int(m, "vdim", where) or dim,
            "scale": _float(m, "scale", where), "window": None, "chunk": _int(mask, "size", where + "mask.") if mask is not None else None,
            "qkv_bias": False, "out_bias": False, "position": None, "distance_slopes": distance_slopes(heads), "element_gate": "g",
            "shared_kv": m.get("kv_from") is not None, "names": {"q": "q", "k": "k", "v": "v", "o": "o"}, "suffixes": SUFFIXES})

    def _rotary_attention(self, m: Mapping[str, Any], where: str) -> PartSpec:
        heads, kv = self._heads(m, where)
        dim = _int(m, "dim", where)
        return PartSpec("attention", {
            "hidden_size": self.width, "num_heads": heads, "num_kv_heads": kv, "head_dim": dim, "value_dim": _opt_int(m, "vdim", where) or dim,
            "scale": _float(m, "scale", where), "window": None, "qkv_bias": True, "out_bias": False, "position": self._rotation(m, dim, where),
            "qk_norm": {"q": "q.norm", "k": "k.norm", "eps": self.eps}, "sink_score": 0.0, "names": {"q": "q", "k": "k", "v": "v", "o": "o"},
            "suffixes": SUFFIXES})

    def _delta(self, m: Mapping[str, Any], where: str) -> PartSpec:
        heads, kv = self._heads(m, where)
        dim = _int(m, "dim", where)
        return PartSpec("gated_delta_rule", {
            "hidden_size": self.width, "num_heads": heads, "num_kv_heads": kv, "head_dim": dim, "value_dim": _opt_int(m, "vdim", where) or dim,
            "conv": _int(m, "conv", where), "decay": "head", "gate": "silu", "eps": self.eps, "conv_suffix": ".conv",
            "names": {"q": "q", "k": "k", "v": "v", "b": "b", "a": "a", "g": "g", "o": "o", "dt_bias": "dt_bias", "A_log": "A_log", "norm": "norm"},
            "suffixes": SUFFIXES})

    def _mixer(self, layer: Mapping[str, Any], where: str) -> PartSpec:
        kind, m = layer.get("type"), layer.get("mixer")
        if not isinstance(m, Mapping):
            raise ConfigError(f"config.json: {where}'mixer' is missing")
        where += "mixer."
        if kind == "attention":
            return self._attention(m, where)
        if kind == "parallel":
            left, right = m.get("left"), m.get("right")
            if not isinstance(left, Mapping) or not isinstance(right, Mapping):
                raise ConfigError(f"config.json: {where}'left' and 'right' are both needed")
            return PartSpec("parallel", {
                "hidden_size": self.width, "left": self._rotary_attention(left, where + "left."), "right": self._delta(right, where + "right."),
                "prefixes": {"left": "left.", "right": "right."}, "left_scale": 0.5, "right_scale": 0.5,
                "out_norms": {"left": "left.out", "right": "right.out", "eps": self.eps}})
        raise ConfigError(f"config.json: {where[:-6]}layer type {kind!r} is not supported (attention, parallel)")

    def _feed_forward(self, layer: Mapping[str, Any], where: str) -> Optional[PartSpec]:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        if not isinstance(mlp, Mapping) or mlp.get("kind") != "moe":
            raise ConfigError(f"config.json: {where}mlp.kind {mlp.get('kind') if isinstance(mlp, Mapping) else mlp!r} is not supported (moe)")
        router, expert = mlp.get("router"), mlp.get("expert")
        if not isinstance(router, Mapping) or not isinstance(expert, Mapping):
            raise ConfigError(f"config.json: {where}mlp needs 'router' (experts, top, groups) and 'expert' (ff, limit)")
        rw = where + "mlp.router."
        experts, top = _int(router, "experts", rw), _int(router, "top", rw)
        groups = router.get("groups")
        count = keep = 1
        if groups is not None:
            if not isinstance(groups, Mapping):
                raise ConfigError(f"config.json: {rw}'groups' must be an object with 'count' and 'keep'")
            count, keep = _int(groups, "count", rw + "groups."), _int(groups, "keep", rw + "groups.")
        if experts % count or keep > count:
            raise ConfigError(f"config.json: {rw}groups: {experts} experts do not form {count} equal groups of which {keep} are kept")
        if top > keep * (experts // count):
            raise ConfigError(f"config.json: {rw}top {top} is more than the {keep * (experts // count)} experts of the kept groups")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": _int(expert, "ff", where + "mlp.expert."), "experts": experts, "top": top,
            "scoring": "sigmoid_grouped", "groups": count, "keep_groups": keep, "weight_on": "output", "activation": "glu_clamped",
            "limit": _float(expert, "limit", where + "mlp.expert."), "alpha": GLU_ALPHA,
            "names": {"router": "router", "correction": "correction", "expert": "e{}.", "gate": "gate", "up": "up", "down": "down"},
            "suffixes": SUFFIXES})

    def schedule(self) -> Tuple[ScheduleEntry, ...]:
        """The layers in order; a layer with ``kv_from`` reads the cache of that layer's entry, which must be an attention
        layer before it with keys and values of its own and the same head counts and sizes (its mask may be another)."""
        out = []
        for i, layer in enumerate(self.layers):
            m = layer.get("mixer") if isinstance(layer, Mapping) else None
            src = m.get("kv_from") if isinstance(m, Mapping) and layer.get("type") == "attention" else None
            if src is None:
                out.append(ScheduleEntry(i))
                continue
            where = f"layers[{i}].mixer."
            if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
                raise ConfigError(f"config.json: {where}kv_from {src!r} must name a layer before this one")
            other = self.layers[src]
            om = other.get("mixer") if isinstance(other, Mapping) else None
            if other.get("type") != "attention" or not isinstance(om, Mapping) or om.get("kv_from") is not None:
                raise ConfigError(f"config.json: {where}kv_from names layer {src}, which is no attention layer with keys and values of its own")
            for key in ("kv_heads", "dim", "vdim"):
                mine, theirs = (x.get(key) or x.get({"kv_heads": "heads", "vdim": "dim"}.get(key, key)) for x in (m, om))
                if mine != theirs:
                    raise ConfigError(f"config.json: {where}'{key}' differs from layer {src}'s, whose keys and values this layer reads")
            out.append(ScheduleEntry(i, cache_from=src))
        return tuple(out)

    def to_model_spec(self) -> ModelSpec:
        def norm(tensor):
            return PartSpec("rmsnorm", {"size": self.width, "eps": self.eps, "tensor": tensor})

        blocks = []
        for i, layer in enumerate(self.layers):
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            where = f"layers[{i}]."
            ff = self._feed_forward(layer, where)
            side = PartSpec("gated_token_row", {
                "hidden_size": self.width, "dim": self.side_dim, "table": TOKEN_TABLE, "column": i * self.side_dim, "eps": self.eps,
                "names": {"gate": "gate", "proj": "proj", "norm": "norm"}, "suffixes": SUFFIXES}) if self.side_dim else None
            blocks.append(BlockSpec.of(
                "sandwich", f"l{i}.",
                prefixes={"mixer": "mix.", "feed_forward": "mlp.", "token_input": "side.", "mixer_norm": "", "mixer_post_norm": "", "feed_forward_norm": "",
                          "feed_forward_post_norm": ""},
                mixer=self._mixer(layer, where), feed_forward=ff, mixer_norm=norm("norm1"), mixer_post_norm=norm("norm1b"),
                feed_forward_norm=norm("norm2") if ff else None, feed_forward_post_norm=norm("norm2b") if ff else None, token_input=side))
        return ModelSpec(
            architecture=self.ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, blocks=tuple(blocks), schedule=self.schedule(),
            final_norm=norm("norm"), tie_word_embeddings=False, max_position_embeddings=self.max_positions, embedding_name="embed",
            final_norm_prefix="final.", lm_head_name="head", embedding_scale=self.embedding_scale if self.embedding_scale != 1.0 else None,
            token_tables={TOKEN_TABLE: len(self.layers) * self.side_dim} if self.side_dim else {})
