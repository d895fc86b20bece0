"""Configuration of the Mimolix design, read from its own config.json keys.

Keys: ``architecture`` ("Mimolix"), ``width``, ``vocab``, ``norm.eps``, ``embedding.scale`` (1 when absent), ``residual_mult`` (1
when absent), ``loop`` (``start``, ``stop``, ``times``: layers start .. stop-1 run that many times in a row on the same weights,
every pass with a cache or state of its own, and the stream is replaced by a product over itself and the embedding's output
ahead of each; absent: every layer once and no such product) and ``layers``, a list whose entries give ``type``, the mixer's
sizes under ``mixer`` and the feed-forward under ``mlp`` (null for none):

* "attention": ``heads``, ``kv_heads``, ``dim`` (of one score map), ``vdim``, ``scale``, ``diff`` and optionally ``q_temp``
  (``coef``, ``every``);
* "delta": ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``;
* ``mlp``: ``kind`` "moe", ``expert.ff``, ``router`` (``experts``, ``top`` and optionally ``scale``) and optionally ``shared.ff``.

Every size and constant that the file gives is kept as it stands, layer by layer; nothing is assumed equal to anything else.
The design has no context length of its own: ``max_position`` (optional) only sets the engine's default.

Translation into parts (``model_spec``): every layer is a ``parallel`` block with one ``layernorm`` and ``residual_mult`` on the
sum of its sublayers. "attention" becomes the ``attention`` mixer with two score maps, "delta" the ``gated_delta`` mixer; the
feed-forward is ``routed_experts`` with ungated squared-ReLU experts, softmax scores and renormalised weights. A layer that the
loop runs again gets one further (weightless) layer per extra pass, which runs the owner's parts on a cache of its own; the
schedule entries that start a pass name the ``embedding_mix`` stream input. The head is a matrix of its own.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .nipadra import DEFAULT_CONTEXT, _int, _num, _obj

MIXER_TYPES = ("attention", "delta")


@dataclass(frozen=True)
class MapAttentionSizes:
    heads: int
    kv_heads: int
    dim: int                                # of one score map
    vdim: int
    scale: float
    diff: float
    temperature: Optional[Tuple[float, float]] = None      # coef, every

    def to_json(self):
        out: Dict[str, Any] = {"diff": self.diff, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
                               "vdim": self.vdim}
        if self.temperature is not None:
            coef, every = self.temperature
            out["q_temp"] = {"coef": coef, "every": int(every) if every == int(every) else every}
        return out


@dataclass(frozen=True)
class DeltaSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def to_json(self):
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}


@dataclass(frozen=True)
class ExpertSizes:
    ff: int
    experts: int
    top: int
    scale: float = 1.0
    shared_ff: Optional[int] = None         # None: no shared expert

    def to_json(self):
        out: Dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "scale": self.scale, "top": self.top}}
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class MimolixLayer:
    type: str                               # one of MIXER_TYPES
    mixer: Any
    mlp: Optional[ExpertSizes]              # None: the layer has no feed-forward

    def to_json(self):
        return {"type": self.type, "mixer": self.mixer.to_json(), "mlp": None if self.mlp is None else self.mlp.to_json()}


def _heads(m: Dict[str, Any], what: str):
    heads, kv_heads, dim, vdim = (_int(m, k, what) for k in ("heads", "kv_heads", "dim", "vdim"))
    if heads % kv_heads:
        raise ConfigError(f"config.json: {what}: heads must be a multiple of kv_heads")
    return heads, kv_heads, dim, vdim


def _attention(m: Dict[str, Any], what: str) -> MapAttentionSizes:
    temperature = None
    if m.get("q_temp") is not None:
        t = _obj(m["q_temp"], what + ".q_temp")
        temperature = (_num(t, "coef", what + ".q_temp"), _num(t, "every", what + ".q_temp"))
        if not temperature[1] > 0:
            raise ConfigError(f"config.json: {what}.q_temp.every must be positive")
    return MapAttentionSizes(*_heads(m, what), _num(m, "scale", what), _num(m, "diff", what), temperature)


def _experts(f: Dict[str, Any], what: str) -> ExpertSizes:
    if f.get("kind") != "moe":
        raise ConfigError(f"config.json: {what} has the unknown kind {f.get('kind')!r} (known: moe)")
    ff = _int(_obj(f.get("expert"), what + ".expert"), "ff", what + ".expert")
    r = _obj(f.get("router"), what + ".router")
    experts, top = _int(r, "experts", what + ".router"), _int(r, "top", what + ".router")
    if top > experts:
        raise ConfigError(f"config.json: {what}.router.top exceeds the {experts} experts")
    scale = 1.0 if r.get("scale") is None else _num(r, "scale", what + ".router")
    shared = None if f.get("shared") is None else _int(_obj(f["shared"], what + ".shared"), "ff", what + ".shared")
    return ExpertSizes(ff, experts, top, scale, shared)


@dataclass(frozen=True)
class MimolixConfig:
    width: int
    vocab: int
    eps: float
    layers: Tuple[MimolixLayer, ...]
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None         # start, stop, times
    max_position: int = DEFAULT_CONTEXT

    architecture = "Mimolix"
    model_type = "mimolix"

    @classmethod
    def from_json(cls, j: Any) -> "MimolixConfig":
        j = _obj(j, "the configuration")
        width, vocab = _int(j, "width", "the model"), _int(j, "vocab", "the model")
        eps = _num(_obj(j.get("norm"), "norm"), "eps", "norm")
        if not eps >= 0:
            raise ConfigError("config.json: norm.eps must be >= 0")
        raw = j.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[MimolixLayer] = []
        for i, entry in enumerate(raw):
            what = f"layer {i}"
            entry = _obj(entry, what)
            kind = entry.get("type")
            m = _obj(entry.get("mixer"), what + ".mixer")
            if kind == "attention":
                mixer = _attention(m, what + ".mixer")
            elif kind == "delta":
                mixer = DeltaSizes(*_heads(m, what + ".mixer"), _int(m, "conv", what + ".mixer"))
            else:
                raise ConfigError(f"config.json: {what} has the unknown type {kind!r} (known: {', '.join(MIXER_TYPES)})")
            mlp = None if entry.get("mlp") is None else _experts(_obj(entry["mlp"], what + ".mlp"), what + ".mlp")
            layers.append(MimolixLayer(kind, mixer, mlp))
        scale = 1.0
        if j.get("embedding") is not None:
            emb = _obj(j["embedding"], "embedding")
            scale = 1.0 if emb.get("scale") is None else _num(emb, "scale", "embedding")
        mult = 1.0 if j.get("residual_mult") is None else _num(j, "residual_mult", "the model")
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
        return cls(width, vocab, eps, tuple(layers), scale, mult, loop, max_position)

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
                               "layers": [l.to_json() for l in self.layers]}
        if self.embedding_scale != 1.0:
            out["embedding"] = {"scale": self.embedding_scale}
        if self.residual_mult != 1.0:
            out["residual_mult"] = self.residual_mult
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.max_position != DEFAULT_CONTEXT:
            out["max_position"] = self.max_position
        return out

    # ------------------------------------------------------------------ the order of runs
    def runs(self) -> List[Tuple[int, int, bool]]:
        """(layer, pass, whether a pass of the loop starts with it) in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, 0, False) for i in range(n)]
        start, stop, times = self.loop
        return [(i, 0, False) for i in range(start)] + [(i, p, i == start) for p in range(times) for i in range(start, stop)] + \
               [(i, 0, False) for i in range(stop, n)]

    # ------------------------------------------------------------------ translation into parts
    def _mixer_spec(self, layer: MimolixLayer) -> PartSpec:
        D, m = self.width, layer.mixer
        if layer.type == "attention":
            return PartSpec("attention", {
                "hidden_size": D, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim,
                "scale": m.scale, "window": None, "position": PartSpec("none", {}), "qk_norm_eps": self.eps, "maps": 2,
                "map_weight": m.diff, "map_factor": 1.0 - m.diff, "query_temperature": m.temperature})
        return PartSpec("gated_delta", {
            "hidden_size": D, "num_heads": m.heads, "num_key_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
            "conv_taps": m.conv, "norm_eps": self.eps})

    def _feed_forward_spec(self, f: Optional[ExpertSizes]) -> Optional[PartSpec]:
        if f is None:
            return None
        shared = None if f.shared_ff is None else {"hidden_size": self.width, "intermediate_size": f.shared_ff, "activation": "relu2"}
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": f.ff, "experts": f.experts, "top": f.top, "gated": False,
            "activation": "relu2", "scores": "softmax", "renormalise": True, "router_scale": f.scale, "shared": shared})

    def model_spec(self) -> ModelSpec:
        D = self.width
        norm = PartSpec("layernorm", {"size": D, "eps": self.eps})
        specs = [LayerSpec(mixer=self._mixer_spec(layer), feed_forward=self._feed_forward_spec(layer.mlp), mixer_norm=norm,
                           feed_forward_norm=None, block="parallel", block_params={"residual_mult": self.residual_mult})
                 for layer in self.layers]
        # a further pass of a looped layer: a layer of its own for the cache manager, the owner's parts and weights
        schedule, shared = [], {}
        for i, p, starts in self.runs():
            cache_of = None
            if p > 0:
                specs.append(specs[i])
                cache_of = len(specs) - 1
                shared[cache_of] = i
            schedule.append(ScheduleEntry(i, cache_of=cache_of, stream_input=starts))
        return ModelSpec(architecture=self.architecture, hidden_size=D, vocab_size=self.vocab, max_position=self.max_position,
                         layers=specs, schedule=schedule, final_norm=norm, tie_word_embeddings=False,
                         embedding_scale=self.embedding_scale,
                         stream_input=None if self.loop is None else PartSpec("embedding_mix", {"hidden_size": D}),
                         open_ended=True, shared_layers=shared)
