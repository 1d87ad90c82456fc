"""Typed configuration of the Setenex decoder, read from config.json.

config.json gives ``architecture`` ("Setenex"), ``vocab``, ``width``, ``norm`` {eps},
``embedding`` {scale}, ``loop`` {start, stop, times} (optional) and ``layers``: a list whose entries
name the layer's mixer (``type``: "attention" or "latent_attention"), the mixer's sizes and constants
(``mixer``) and its feed-forward (``mlp``: ``kind`` "moe" with ``expert`` {ff} and ``router``
{experts, top, groups {count, keep}}; or null for no feed-forward).  Every size and every constant that
may differ between models comes from there, layer by layer; the number of rows of an attention
layer's distance table is its stored tensor's.

The model.  Embedding: table row times ``scale``.  Every norm of the stream is an RMS norm whose
stored weight lies around zero (multiplier 1 + w).  Layers are parallel over one norm,
x += mixer(norm1(x)) + ff(norm1(x)).  Layers ``start .. stop - 1`` run ``times`` times in a row with the
same weights and a cache per pass; before every pass row t of ``loop.step`` is added to the stream.
"attention": grouped-query attention without rotation, every q and k head normed with a weight per
value, a learned bias per head and bucket of distances added to the scores, a sliding window that keeps
a sequence's first tokens.  "latent_attention": keys and values from one normed latent per position,
queries straight from the input, neighbouring pairs of the rotated part turned by position, a sliding
window, a sigmoid gate per head.  Experts: down(gelu(up(x))), the erf gelu, chosen by sigmoid scores
plus a correction within the best groups (a group's rank the sum of its two largest), weighed by the
chosen scores divided by their sum.  Head: the model's norm, a matrix of its own.

Tensor names: ``embed``, ``loop.step``, ``final.norm``, ``head`` and ``l<i>.norm1``,
``l<i>.mix.{q,k,v,o,q.norm,k.norm,rel}`` or ``l<i>.mix.{q,dkv,dkv.norm,uk,uv,g,o}``,
``l<i>.mlp.{router,correction,e<j>.{up,down}}``, with no ``.weight`` ending; weights are stored in
bfloat16.  Positions have no bound of the model's own.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .llama import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, StreamEnter

# angles are float32 products position * frequency; beyond 2^24 a position is no exact float32
MAX_POSITIONS = 1 << 24
# constants that the design fixes
NORM_OFFSET = 1.0  # a norm's multiplier is NORM_OFFSET + the stored weight
GROUP_TOP = 2      # an expert group's rank is the sum of this many of its largest choice scores
# rows of a distance table where weights are made at random (a stored table brings its own number)
RANDOM_TABLE_ROWS = 32


def _int(raw: Mapping[str, Any], key: str, where: str, least: int = 1) -> int:
    value = raw.get(key)
    if isinstance(value, bool) or not isinstance(value, int) or value < least:
        raise ConfigError(f"config.json: {where}.{key} must be an integer >= {least}; got {value!r}")
    return value


def _number(raw: Mapping[str, Any], key: str, where: str, positive: bool = True) -> float:
    value = raw.get(key)
    if isinstance(value, bool) or not isinstance(value, (int, float)) or not math.isfinite(value) \
            or (positive and value <= 0):
        raise ConfigError(f"config.json: {where}.{key} must be a finite{' positive' if positive else ''} number; "
                          f"got {value!r}")
    return float(value)


def _object(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return value


def _check_attention(m: Mapping[str, Any], where: str) -> None:
    heads, kv_heads = _int(m, "heads", where), _int(m, "kv_heads", where)
    _int(m, "dim", where)
    _int(m, "vdim", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.heads={heads} is no multiple of kv_heads={kv_heads}")
    _number(m, "scale", where, positive=False)
    _number(m, "bias_max", where)
    mask = _object(m, "mask", where)
    _int(mask, "size", where + ".mask")
    _int(mask, "keep_first", where + ".mask", 0)


def _check_latent(m: Mapping[str, Any], where: str) -> None:
    for key in ("heads", "dim", "vdim", "kv_rank"):
        _int(m, key, where)
    rot_dim = _int(m, "rot_dim", where, 0)
    _number(m, "scale", where, positive=False)
    _int(_object(m, "mask", where), "size", where + ".mask")
    rot = _object(m, "rot", where)
    dims = rot.get("dims")
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > rot_dim:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most {rot_dim}; got {dims!r}")
    _number(rot, "base", where + ".rot")


_MIXERS = {"attention": _check_attention, "latent_attention": _check_latent}


def _check_mlp(mlp: Mapping[str, Any], where: str) -> None:
    if mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}.kind {mlp.get('kind')!r} is not a feed-forward of this design (moe)")
    _int(_object(mlp, "expert", where), "ff", where + ".expert")
    r = _object(mlp, "router", where)
    experts, top = _int(r, "experts", where + ".router"), _int(r, "top", where + ".router")
    g = _object(r, "groups", where + ".router")
    count, keep = _int(g, "count", where + ".router.groups"), _int(g, "keep", where + ".router.groups")
    if experts % count or keep > count or top > keep * (experts // count):
        raise ConfigError(f"config.json: {where}.router: {experts} experts in {count} groups (keep {keep}) cannot "
                          f"give top={top}")


@dataclass(frozen=True)
class SetenexLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]


@dataclass(frozen=True)
class SetenexConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    loop: Optional[Tuple[int, int, int]]  # start, stop, times
    layers: Tuple[SetenexLayer, ...]
    raw: Mapping[str, Any]

    architecture = "Setenex"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "SetenexConfig":
        if raw.get("architecture") != cls.architecture:
            raise ConfigError(f"config.json: architecture must be {cls.architecture!r}; "
                              f"got {raw.get('architecture')!r}")
        vocab, width = _int(raw, "vocab", "config"), _int(raw, "width", "config")
        eps = _number(_object(raw, "norm", "config"), "eps", "norm")
        scale = _number(_object(raw, "embedding", "config"), "scale", "embedding", positive=False)
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: layers must be a list of at least one layer")
        layers: List[SetenexLayer] = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping) or not isinstance(entry.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where} must be an object with type, mixer and mlp")
            kind, mixer = entry.get("type"), entry["mixer"]
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design "
                                  f"({', '.join(sorted(_MIXERS))})")
            _MIXERS[kind](mixer, where + ".mixer")
            mlp = entry.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, Mapping):
                    raise ConfigError(f"config.json: {where}.mlp must be null or an object")
                _check_mlp(mlp, where + ".mlp")
            layers.append(SetenexLayer(kind, mixer, mlp))
        loop = None
        if raw.get("loop") is not None:
            lp = _object(raw, "loop", "config")
            start, stop = _int(lp, "start", "loop", 0), _int(lp, "stop", "loop", 0)
            times = _int(lp, "times", "loop", 1)
            if not start < stop <= len(layers):
                raise ConfigError(f"config.json: loop {start}..{stop} does not lie within {len(layers)} layers")
            loop = (start, stop, times)
        return cls(vocab, width, eps, scale, loop, tuple(layers), dict(raw))

    def to_dict(self) -> Dict[str, Any]:
        """The config.json that reads back as this configuration."""
        def plain(x):
            return {k: plain(v) for k, v in x.items()} if isinstance(x, Mapping) else x
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
               "layers": [{"type": l.type, "mixer": plain(l.mixer),
                           "mlp": None if l.mlp is None else plain(l.mlp)} for l in self.layers]}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return out

    # ------------------------------------------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "name": name, "leaf": "",
                                    "offset": NORM_OFFSET})

    def _mixer(self, layer: SetenexLayer) -> PartSpec:
        m = layer.mixer
        window = min(m["mask"]["size"], MAX_POSITIONS)
        if layer.type == "attention":
            return PartSpec("sink_attention", {
                "hidden_size": self.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"],
                "vdim": m["vdim"], "scale": m["scale"], "window": window,
                "keep_first": min(m["mask"]["keep_first"], MAX_POSITIONS),
                "distance_bias": {"far": m["bias_max"], "rows": RANDOM_TABLE_ROWS}, "qk_norm": "head_weight",
                "eps": self.norm_eps, "pad_heads": True,
                # no rotation: a position shows in the distance bias alone
                "position": PartSpec("rope_frequencies", {"dims": 0, "base": 1.0, "pairing": "half"}), "leaf": "",
                "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "q_norm": "mix.q.norm",
                          "k_norm": "mix.k.norm", "distance_bias": "mix.rel"}})
        return PartSpec("latent_attention", {
            "hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"],
            "vdim": m["vdim"], "q_rank": 0, "kv_rank": m["kv_rank"], "scale": m["scale"], "eps": self.norm_eps,
            "window": window, "gate": "head",
            "position": PartSpec("rope_frequencies", {"dims": m["rot"]["dims"], "base": m["rot"]["base"],
                                                      "pairing": "neighbours"}), "leaf": "",
            "names": {"q": "mix.q", "dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm", "uk": "mix.uk", "uv": "mix.uv",
                      "gate": "mix.g", "o": "mix.o"}})

    def _ffn(self, mlp: Mapping[str, Any]) -> PartSpec:
        r = mlp["router"]
        return PartSpec("moe", {
            "hidden_size": self.width, "experts": r["experts"], "top": r["top"], "ff": mlp["expert"]["ff"],
            "activation": "gelu", "scores": "sigmoid_all", "weight_on": "output", "groups": r["groups"]["count"],
            "keep": r["groups"]["keep"], "group_top": GROUP_TOP, "renormalise": True, "leaf": "",
            "names": {"router": "mlp.router", "correction": "mlp.correction", "expert": "mlp.e{e}", "up": "up",
                      "down": "down"}})

    def run_order(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass number if it is the first layer of a pass through the loop) in run order."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        order: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(start)]
        for t in range(times):
            order += [(i, t if i == start else None) for i in range(start, stop)]
        return order + [(i, None) for i in range(stop, n)]

    def to_spec(self) -> ModelSpec:
        layers = []
        for i, layer in enumerate(self.layers):
            parts = {"norm": self._norm("norm1"), "mixer": self._mixer(layer)}
            if layer.mlp is not None:
                parts["ffn"] = self._ffn(layer.mlp)
            layers.append(LayerSpec(prefix=f"l{i}", block="parallel", parts=parts, params={}))
        times = self.loop[2] if self.loop is not None else 0
        schedule = [ScheduleEntry(i, enter=None if t is None else StreamEnter(tensor="loop.step", rows=times, row=t))
                    for i, t in self.run_order()]
        spec = ModelSpec(
            architecture=self.architecture,
            hidden_size=self.width,
            vocab_size=self.vocab,
            max_positions=MAX_POSITIONS,
            embedding=PartSpec("scaled_token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width,
                                                          "name": "embed", "leaf": "",
                                                          "scale": self.embedding_scale}),
            layers=tuple(layers),
            schedule=tuple(schedule),
            final_norm=self._norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": self.width, "name": "head",
                                          "leaf": ""}),
            stop_token_ids=(),
            stored_dtype="bfloat16",
        )
        spec.validate()
        return spec
