"""Configuration of the Kidarax design, read from its own config.json keys.

Keys: ``architecture`` ("Kidarax"), ``width``, ``vocab``, ``norm.eps``, ``logit_scale`` (1 when absent), ``loop`` (``start``,
``stop``, ``times``: layers start .. stop-1 run that many times in a row on the same weights, every pass with a cache or state
of its own, and the embedding's output is added to the stream ahead of every pass but the first; absent: every layer once) and
``layers``, a list whose entries give ``type``, the mixer's sizes under ``mixer`` and the feed-forward under ``mlp`` (null for
none):

* "retention": ``heads``, ``dim``, ``vdim``, ``decay`` (one factor per head);
* "attention": ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot`` (``base``, ``dims`` and optionally ``scaling.factor``);
* "latent_attention": ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``rot`` (``base``, ``dims`` and optionally
  ``scaling`` with ``factor``, ``original``, ``fast``, ``slow``);
* ``mlp``: ``kind`` "dense" with ``ff``, or "moe" with ``expert.ff``, ``router`` (``experts``, ``top``) and optionally ``shared.ff``.

Every size and constant that the file gives is kept as it stands, layer by layer; nothing is assumed equal to anything else.
The design has no context length of its own: ``max_position`` (optional) only sets the engine's default.

Translation into parts (``model_spec``): every layer is a ``sandwich`` block with ``dynamic_tanh`` norms. "retention" becomes the
``linear_attention`` mixer without activations and with a norm per head, "attention" the ``attention`` mixer with biases and a
gate per output value, "latent_attention" the mixer of that name without a query latent and with a gate per head; the dense
feed-forward is a squared-ReLU ``mlp``, the mixture ``routed_experts`` whose weights scale the experts' inputs, with a gated shared
expert. A layer that the loop runs again gets one further (weightless) layer per extra pass, which runs the owner's parts on
a cache of its own; the schedule entries that start a further pass name the ``embedding_add`` stream input. The head is the
embedding table, its logits times ``logit_scale``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .nipadra import DEFAULT_CONTEXT, _int, _num, _obj

MIXER_TYPES = ("retention", "attention", "latent_attention")


def _plain(v: float):
    return int(v) if v == int(v) else v


@dataclass(frozen=True)
class RetentionSizes:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    def to_json(self):
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int
    factor: Optional[float] = None                              # None: the pairs' frequencies as they are
    ramp: Optional[Tuple[float, float, float]] = None           # original, fast, slow: only slow pairs are stretched

    def to_json(self):
        out: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.factor is not None:
            out["scaling"] = {"factor": self.factor}
            if self.ramp is not None:
                out["scaling"].update(zip(("original", "fast", "slow"), map(_plain, self.ramp)))
        return out

    def spec(self, head_dim: int) -> PartSpec:
        params: Dict[str, Any] = {"head_dim": head_dim, "rotary_dim": self.dims, "theta": self.base, "pairing": "half_split"}
        if self.ramp is not None:
            params["ramp_scaling"] = dict(zip(("original", "fast", "slow"), self.ramp), factor=self.factor)
        elif self.factor is not None:
            params["linear_scaling"] = {"factor": self.factor}
        return PartSpec("rope_on_device", params)


@dataclass(frozen=True)
class GatedAttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation

    def to_json(self):
        return {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "rot": self.rot.to_json(), "scale": self.scale,
                "vdim": self.vdim}


@dataclass(frozen=True)
class LatentSizes:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Rotation

    def to_json(self):
        return {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "rot": self.rot.to_json(), "rot_dim": self.rot_dim,
                "scale": self.scale, "vdim": self.vdim}


@dataclass(frozen=True)
class DenseSizes:
    ff: int

    def to_json(self):
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class ExpertSizes:
    ff: int
    experts: int
    top: int
    shared_ff: Optional[int] = None         # None: no shared expert

    def to_json(self):
        out: Dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class KidaraxLayer:
    type: str                               # one of MIXER_TYPES
    mixer: Any
    mlp: Any                                # DenseSizes, ExpertSizes or None: the layer has no feed-forward

    def to_json(self):
        return {"type": self.type, "mixer": self.mixer.to_json(), "mlp": None if self.mlp is None else self.mlp.to_json()}


def _retention(m: Dict[str, Any], what: str) -> RetentionSizes:
    heads, dim, vdim = (_int(m, k, what) for k in ("heads", "dim", "vdim"))
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != heads:
        raise ConfigError(f"config.json: {what}.decay must be a list with one factor per head")
    return RetentionSizes(heads, dim, vdim, tuple(_num({"decay": d}, "decay", what) for d in decay))


def _rotation(m: Dict[str, Any], what: str, size: int, ramp: bool) -> Rotation:
    r = _obj(m.get("rot"), what + ".rot")
    base, dims = _num(r, "base", what + ".rot"), _int(r, "dims", what + ".rot")
    if dims % 2 or dims > size or not base > 0:
        raise ConfigError(f"config.json: {what}.rot: 'dims' must be even and at most {size}, 'base' positive")
    if r.get("scaling") is None:
        return Rotation(base, dims)
    s = _obj(r["scaling"], what + ".rot.scaling")
    names = ("factor", "original", "fast", "slow") if ramp else ("factor",)
    values = tuple(_num(s, k, what + ".rot.scaling") for k in names)
    if min(values) <= 0:
        raise ConfigError(f"config.json: {what}.rot.scaling: the numbers must be positive")
    return Rotation(base, dims, values[0], values[1:] if ramp else None)


def _attention(m: Dict[str, Any], what: str) -> GatedAttentionSizes:
    heads, kv_heads, dim, vdim = (_int(m, k, what) for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv_heads:
        raise ConfigError(f"config.json: {what}: heads must be a multiple of kv_heads")
    return GatedAttentionSizes(heads, kv_heads, dim, vdim, _num(m, "scale", what), _rotation(m, what, dim, ramp=False))


def _latent(m: Dict[str, Any], what: str) -> LatentSizes:
    heads, dim, rot_dim, vdim, kv_rank = (_int(m, k, what) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    rot = _rotation(m, what, rot_dim, ramp=True)
    if rot.dims != rot_dim:
        raise ConfigError(f"config.json: {what}.rot.dims must equal rot_dim: the rotated part is rotated as a whole")
    return LatentSizes(heads, dim, rot_dim, vdim, kv_rank, _num(m, "scale", what), rot)


def _feed_forward(f: Dict[str, Any], what: str):
    if f.get("kind") == "dense":
        return DenseSizes(_int(f, "ff", what))
    if f.get("kind") != "moe":
        raise ConfigError(f"config.json: {what} has the unknown kind {f.get('kind')!r} (known: dense, moe)")
    ff = _int(_obj(f.get("expert"), what + ".expert"), "ff", what + ".expert")
    r = _obj(f.get("router"), what + ".router")
    experts, top = _int(r, "experts", what + ".router"), _int(r, "top", what + ".router")
    if top > experts:
        raise ConfigError(f"config.json: {what}.router.top exceeds the {experts} experts")
    shared = None if f.get("shared") is None else _int(_obj(f["shared"], what + ".shared"), "ff", what + ".shared")
    return ExpertSizes(ff, experts, top, shared)


_MIXERS = {"retention": _retention, "attention": _attention, "latent_attention": _latent}


@dataclass(frozen=True)
class KidaraxConfig:
    width: int
    vocab: int
    eps: float
    layers: Tuple[KidaraxLayer, ...]
    logit_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None         # start, stop, times
    max_position: int = DEFAULT_CONTEXT

    architecture = "Kidarax"
    model_type = "kidarax"

    @classmethod
    def from_json(cls, j: Any) -> "KidaraxConfig":
        j = _obj(j, "the configuration")
        width, vocab = _int(j, "width", "the model"), _int(j, "vocab", "the model")
        eps = _num(_obj(j.get("norm"), "norm"), "eps", "norm")
        if not eps >= 0:
            raise ConfigError("config.json: norm.eps must be >= 0")
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[KidaraxLayer] = []
        for i, entry in enumerate(raw):
            what = f"layer {i}"
            entry = _obj(entry, what)
            kind = entry.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {what} has the unknown type {kind!r} (known: {', '.join(MIXER_TYPES)})")
            mixer = _MIXERS[kind](_obj(entry.get("mixer"), what + ".mixer"), what + ".mixer")
            mlp = None if entry.get("mlp") is None else _feed_forward(_obj(entry["mlp"], what + ".mlp"), what + ".mlp")
            layers.append(KidaraxLayer(kind, mixer, mlp))
        scale = 1.0 if j.get("logit_scale") is None else _num(j, "logit_scale", "the model")
        loop = None
        if j.get("loop") is not None:
            lp = _obj(j["loop"], "loop")
            start = lp.get("start")
            if isinstance(start, bool) or not isinstance(start, int) or start < 0:
                raise ConfigError("config.json: loop.start must be a layer index")
            stop, times = _int(lp, "stop", "loop"), _int(lp, "times", "loop")
            if not (start < stop <= len(layers)):
                raise ConfigError(f"config.json: loop {start} .. {stop} does not lie inside the {len(layers)} layers")
            loop = (start, stop, times)
        max_position = DEFAULT_CONTEXT if j.get("max_position") is None else _int(j, "max_position", "the model")
        return cls(width, vocab, eps, tuple(layers), scale, loop, max_position)

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
                               "layers": [l.to_json() for l in self.layers]}
        if self.logit_scale != 1.0:
            out["logit_scale"] = self.logit_scale
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.max_position != DEFAULT_CONTEXT:
            out["max_position"] = self.max_position
        return out

    # ------------------------------------------------------------------ the order of runs
    def runs(self) -> List[Tuple[int, int, bool]]:
        """(layer, pass, whether a further pass of the loop starts with it) in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, 0, False) for i in range(n)]
        start, stop, times = self.loop
        return [(i, 0, False) for i in range(start)] + [(i, p, p > 0 and i == start) for p in range(times) for i in range(start, stop)] + \
               [(i, 0, False) for i in range(stop, n)]

    # ------------------------------------------------------------------ translation into parts
    def _mixer_spec(self, layer: KidaraxLayer) -> PartSpec:
        D, m = self.width, layer.mixer
        if layer.type == "retention":
            return PartSpec("linear_attention", {
                "hidden_size": D, "num_heads": m.heads, "key_dim": m.dim, "value_dim": m.vdim, "decay": list(m.decay), "norm_eps": self.eps,
                "activation": "none", "query_scale": m.dim ** -0.5, "norm_per_head": True, "norm_weights": False, "gate": "silu"})
        if layer.type == "attention":
            return PartSpec("attention", {
                "hidden_size": D, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
                "scale": m.scale, "window": None, "position": m.rot.spec(m.dim), "bias": True, "output_gate": True})
        return PartSpec("latent_attention", {
            "hidden_size": D, "num_heads": m.heads, "head_dim": m.dim, "rotary_dim": m.rot_dim, "value_dim": m.vdim, "q_rank": None,
            "kv_rank": m.kv_rank, "scale": m.scale, "window": None, "norm_eps": self.eps, "position": m.rot.spec(m.rot_dim),
            "sink": "learned", "head_gate": True})

    def _feed_forward_spec(self, f) -> Optional[PartSpec]:
        D = self.width
        if f is None:
            return None
        if isinstance(f, DenseSizes):
            return PartSpec("mlp", {"hidden_size": D, "intermediate_size": f.ff, "activation": "relu2"})
        shared = None if f.shared_ff is None else {"hidden_size": D, "intermediate_size": f.shared_ff, "activation": "silu"}
        return PartSpec("routed_experts", {
            "hidden_size": D, "intermediate_size": f.ff, "experts": f.experts, "top": f.top, "activation": "silu", "scores": "sigmoid",
            "weigh_input": True, "shared": shared, "shared_gate": shared is not None})

    def model_spec(self) -> ModelSpec:
        D = self.width
        norm = PartSpec("dynamic_tanh", {"size": D})
        specs = []
        for layer in self.layers:
            ff = self._feed_forward_spec(layer.mlp)
            extra = {"mixer_out_norm": norm}
            if ff is not None:
                extra["feed_forward_out_norm"] = norm
            specs.append(LayerSpec(mixer=self._mixer_spec(layer), feed_forward=ff, mixer_norm=norm,
                                   feed_forward_norm=None if ff is None else norm, block="sandwich", extra=extra))
        # a further pass of a looped layer: a layer of its own for the cache manager, the owner's parts and weights
        schedule, shared = [], {}
        for i, p, starts in self.runs():
            cache_of = None
            if p > 0:
                specs.append(specs[i])
                cache_of = len(specs) - 1
                shared[cache_of] = i
            schedule.append(ScheduleEntry(i, cache_of=cache_of, stream_input=starts))
        again = any(e.stream_input for e in schedule)
        return ModelSpec(architecture=self.architecture, hidden_size=D, vocab_size=self.vocab, max_position=self.max_position,
                         layers=specs, schedule=schedule, final_norm=norm, tie_word_embeddings=True,
                         stream_input=PartSpec("embedding_add", {"hidden_size": D}) if again else None,
                         logit_transform=None if self.logit_scale == 1.0 else PartSpec("scale", {"factor": self.logit_scale}),
                         open_ended=True, shared_layers=shared)
