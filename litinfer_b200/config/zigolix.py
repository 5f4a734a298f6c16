"""Configuration of the Zigolix decoder, read from config.json.

config.json names the design under ``architecture`` and lists the layers one by one: each entry gives its ``type``
(which mixer it has), the mixer's sizes (``mixer``) and its feed-forward (``mlp``, or null for none).  Model-wide keys:
``vocab``, ``width``, ``norm.eps``, ``logit_scale`` (a factor on the logits) and ``loop`` (``start``, ``stop``, ``times``): the
layers start .. stop - 1 run ``times`` times in a row with the same weights, each pass with a cache of its own.  Right before
pass t the residual stream x becomes ``loop.in [x; x0] + loop.step[t]`` with x0 the embedding output.

A layer is pre-norm, ``x += mixer(norm1(x))``, then ``x += ff(norm2(x))``, with RMS norms.

Layer types:

* ``attention``: grouped-query softmax attention without a value map (a key as projected is its value), rotation of the first
  ``rot.dims`` elements of each query and key head (pairs of neighbours, base ``rot.base``, frequencies blended by the pair's
  index with ``rot.scaling``: factor, original, fast, slow), then each head divided by its root mean square, scores scaled by
  ``scale``, a sliding window of ``mask.size`` positions, a learned sink per head in the softmax's denominator.
* ``attention_2``: differential attention: two maps per head over the same values, the second taken off the first with a
  learned factor around ``diff``, biased projections, no positions, scores scaled by ``scale`` and capped by ``softcap``, a
  sliding window of ``mask.size`` positions, a norm per head and a gate per output element.

The feed-forward is dense (``kind`` dense: a gated unit of width ``ff`` with gelu) or a mixture (``kind`` moe): ``router.experts``
gated units with bounded operands (``expert.ff``, ``expert.limit``; the unit's 1.702 is the design's), ``router.top`` of them per
token by the softmax over all experts, renormalised, and a shared one that every token takes (``shared.ff``, ``shared.limit``).

Tensor names follow the file: ``l<i>.`` per layer, ``mix.`` / ``mlp.`` / ``norm1`` / ``norm2`` below it, weights under the bare
stem and biases under ``<stem>.b``.  Sizes and constants all come from config.json.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .filasun import _float, _int
from .gorulorn import LOOP_TABLE, MAX_POSITIONS, SUFFIXES, _opt_int
from .pifazen import GLU_ALPHA
from .qwen2 import ConfigError
from .spec import BlockSpec, ModelSpec, PartSpec, ScheduleEntry

LOOP_MAP = "loop.in"


@dataclass(frozen=True)
class ZigolixConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[Mapping[str, Any], ...]
    loop: Optional[Tuple[int, int, int]] = None            # (start, stop, times)
    logit_scale: float = 1.0
    max_positions: int = MAX_POSITIONS

    ARCHITECTURE = "Zigolix"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ZigolixConfig":
        norm = d.get("norm")
        if not isinstance(norm, Mapping):
            raise ConfigError("config.json: missing key 'norm' (with 'eps')")
        eps = _float(norm, "eps", "norm.")
        if eps <= 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps}")
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        loop = d.get("loop")
        if loop is not None:
            if not isinstance(loop, Mapping):
                raise ConfigError("config.json: 'loop' must be an object with 'start', 'stop' and 'times'")
            start, stop, times = loop.get("start"), loop.get("stop"), _int(loop, "times", "loop.")
            if any(isinstance(v, bool) or not isinstance(v, int) for v in (start, stop)) or not 0 <= start < stop <= len(layers):
                raise ConfigError(f"config.json: loop {start!r} .. {stop!r} does not lie within the {len(layers)} layers")
            loop = (start, stop, times)
        cfg = cls(vocab=_int(d, "vocab", ""), width=_int(d, "width", ""), eps=eps, layers=tuple(layers), loop=loop,
                  logit_scale=_float(d, "logit_scale", "") if d.get("logit_scale") is not None else 1.0,
                  max_positions=_int(d, "max_positions", "") if d.get("max_positions") is not None else MAX_POSITIONS)
        cfg.to_model_spec()                       # every layer's keys are read (and refused) here, not at the first step
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                               "layers": [dict(x) for x in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.logit_scale != 1.0:
            out["logit_scale"] = self.logit_scale
        if self.max_positions != MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        return out

    # ------------------------------------------------------------------
    def _window(self, m: Mapping[str, Any], where: str) -> Optional[int]:
        mask = m.get("mask")
        if mask is None:
            return None
        if not isinstance(mask, Mapping):
            raise ConfigError(f"config.json: {where}'mask' must be an object with 'size'")
        return _opt_int(mask, "size", where + "mask.")

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
        vdim = _opt_int(m, "vdim", where) or dim
        if vdim != dim:
            raise ConfigError(f"config.json: {where}vdim {vdim} must be dim {dim}: the values are the keys")
        return PartSpec("attention", {
            "hidden_size": self.width, "num_heads": heads, "num_kv_heads": kv, "head_dim": dim, "value_dim": dim,
            "scale": _float(m, "scale", where), "window": self._window(m, where), "qkv_bias": False, "out_bias": False,
            "position": self._rotation(m, dim, where), "norm_after": {"eps": self.eps}, "keys_are_values": True, "sink": "sink",
            "names": {"q": "q", "k": "k", "o": "o"}, "suffixes": SUFFIXES})

    def _differential_attention(self, m: Mapping[str, Any], where: str) -> PartSpec:
        heads, kv = self._heads(m, where)
        dim = _int(m, "dim", where)
        return PartSpec("differential_attention", {
            "hidden_size": self.width, "num_heads": heads, "num_kv_heads": kv, "head_dim": dim, "value_dim": _opt_int(m, "vdim", where) or dim,
            "scale": _float(m, "scale", where), "softcap": _float(m, "softcap", where) if m.get("softcap") is not None else None,
            "window": self._window(m, where), "diff": _float(m, "diff", where), "eps": self.eps, "qkv_bias": True, "gate": "g",
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "lq1": "lq1", "lk1": "lk1", "lq2": "lq2", "lk2": "lk2"}, "suffixes": SUFFIXES})

    def _mixer(self, layer: Mapping[str, Any], where: str) -> PartSpec:
        kind, m = layer.get("type"), layer.get("mixer")
        if not isinstance(m, Mapping):
            raise ConfigError(f"config.json: {where}'mixer' is missing")
        if kind == "attention":
            return self._attention(m, where + "mixer.")
        if kind == "attention_2":
            return self._differential_attention(m, where + "mixer.")
        raise ConfigError(f"config.json: {where}layer type {kind!r} is not supported (attention, attention_2)")

    def _unit(self, d: Mapping[str, Any], where: str) -> Dict[str, Any]:
        """The sizes and constants of a gated unit with bounded operands."""
        return {"hidden_size": self.width, "intermediate_size": _int(d, "ff", where), "limit": _float(d, "limit", where), "alpha": GLU_ALPHA,
                "suffixes": SUFFIXES}

    def _feed_forward(self, layer: Mapping[str, Any], where: str) -> Optional[PartSpec]:
        mlp = layer.get("mlp")
        if mlp is None:
            return None
        names = {"gate": "gate", "up": "up", "down": "down"}
        kind = mlp.get("kind") if isinstance(mlp, Mapping) else mlp
        if kind == "dense":
            return PartSpec("geglu", {"hidden_size": self.width, "intermediate_size": _int(mlp, "ff", where + "mlp."), "names": names,
                                      "suffixes": SUFFIXES})
        if kind != "moe":
            raise ConfigError(f"config.json: {where}mlp.kind {kind!r} is not supported (dense, moe)")
        router, expert, shared = mlp.get("router"), mlp.get("expert"), mlp.get("shared")
        if not isinstance(router, Mapping) or not isinstance(expert, Mapping):
            raise ConfigError(f"config.json: {where}mlp needs 'router' (experts, top) and 'expert' (ff, limit)")
        if shared is not None and not isinstance(shared, Mapping):
            raise ConfigError(f"config.json: {where}mlp.'shared' must be an object with 'ff' and 'limit'")
        rw = where + "mlp.router."
        experts, top = _int(router, "experts", rw), _int(router, "top", rw)
        if top > experts:
            raise ConfigError(f"config.json: {rw}top {top} is more than the {experts} experts")
        return PartSpec("routed_experts", dict(
            self._unit(expert, where + "mlp.expert."), experts=experts, top=top, scoring="softmax", renormalize=True, weight_on="output",
            activation="glu_clamped", names=dict(names, router="router", expert="e{}.", shared="shared."),
            shared=PartSpec("clamped_glu", dict(self._unit(shared, where + "mlp.shared."), names=names)) if shared is not None else None))

    def schedule(self) -> Tuple[ScheduleEntry, ...]:
        """The layers in the order they run; a looped span's passes one after the other, each entry with a cache of its own; the
        first layer of pass t behind the map of the stream and row t of the loop's table."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(ScheduleEntry(i) for i in range(n))
        start, stop, times = self.loop
        out = [ScheduleEntry(i) for i in range(start)]
        for t in range(times):
            out.append(ScheduleEntry(start, add=(LOOP_TABLE, t), join=LOOP_MAP))
            out += [ScheduleEntry(i) for i in range(start + 1, stop)]
        return tuple(out + [ScheduleEntry(i) for i in range(stop, n)])

    def to_model_spec(self) -> ModelSpec:
        def norm(tensor, gain=1.0):
            return PartSpec("rmsnorm", {"size": self.width, "eps": self.eps, "tensor": tensor, "gain": gain})

        blocks = []
        for i, layer in enumerate(self.layers):
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            where = f"layers[{i}]."
            ff = self._feed_forward(layer, where)
            blocks.append(BlockSpec.of(
                "prenorm", f"l{i}.", prefixes={"mixer": "mix.", "feed_forward": "mlp.", "mixer_norm": "", "feed_forward_norm": ""},
                mixer=self._mixer(layer, where), feed_forward=ff, mixer_norm=norm("norm1"), feed_forward_norm=norm("norm2") if ff else None))
        # (the factor on the logits goes into the weight of the norm before them)
        return ModelSpec(
            architecture=self.ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, blocks=tuple(blocks), schedule=self.schedule(),
            final_norm=norm("norm", self.logit_scale), tie_word_embeddings=False, max_position_embeddings=self.max_positions, embedding_name="embed",
            final_norm_prefix="final.", lm_head_name="head",
            stream_tables={LOOP_TABLE: self.loop[2]} if self.loop is not None else {}, stream_maps=(LOOP_MAP,) if self.loop is not None else ())
