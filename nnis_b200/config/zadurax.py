"""Typed configuration of the Zadurax decoder, read from config.json.

config.json gives ``architecture`` ("Zadurax"), ``vocab``, ``width``, ``norm`` {eps} and
``layers``: a list whose entries name the layer's mixer (``type``: "attention", "latent_attention"
or "mlstm"), the mixer's sizes and constants (``mixer``), its feed-forward (``mlp``: ``kind``
"dense" with ``ff``; or null for none) and, optionally, ``weights_of``: the layer whose tensors
this one uses (it has none of its own, and a cache or state of its own all the same).  Every size
and every constant that may differ between models comes from there, layer by layer.

The model.  Embedding: a table row, normed.  Layers with a norm before and a norm after each
sub-layer: x += norm1b(mixer(norm1(x))), then x += norm2b(ff(norm2(x))).  "attention":
grouped-query attention over a sliding window, every q and k head normed with a weight per value
that all heads share and then turned in neighbouring pairs, the values the keys as they were
before both, the joined heads gated value by value.  "latent_attention": keys and values from one
normed latent per position, queries straight from the input, frequencies blended by index and
cosines and sines with a magnitude, a sink in the softmax, the joined heads gated value by value.
"mlstm": a matrix memory with exponential gates.  Feed-forward: down(gelu(gate(x)) * up(x)), gelu
in its tanh form.  Head: the model's norm, a matrix of its own.

Tensor names: ``embed``, ``embed.norm``, ``final.norm``, ``head`` and ``l<i>.norm1``,
``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.{q,k,q.norm,k.norm,g,o}``,
``l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,g,o}`` or ``l<i>.mix.{q,k,v,g,o,norm,i,i.b,f,f.b}``,
``l<i>.mlp.{gate,up,down}``, with no ``.weight`` ending; weights are stored in bfloat16.
Positions have no bound of the model's own.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

from .llama import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

# angles are float32 products position * frequency; beyond 2^24 a position is no exact float32
MAX_POSITIONS = 1 << 24
# constants that the design fixes
MEMORY_FLOOR = 1e-6  # added to the matrix memory's denominator


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


def _check_rotation(m: Mapping[str, Any], where: str, most: int) -> None:
    rot = _object(m, "rot", where)
    where += ".rot"
    dims = rot.get("dims")
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > most:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {most}; got {dims!r}")
    base = _number(rot, "base", where)
    if rot.get("scaling") is not None:
        scaling = _object(rot, "scaling", where)
        for key in ("factor", "original", "fast", "slow"):
            _number(scaling, key, where + ".scaling")
        if base <= 1.0:
            raise ConfigError(f"config.json: {where}.base must be above 1 with scaling; got {base}")


def _check_attention(m: Mapping[str, Any], where: str) -> None:
    heads, kv_heads = _int(m, "heads", where), _int(m, "kv_heads", where)
    dim = _int(m, "dim", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.heads={heads} is no multiple of kv_heads={kv_heads}")
    if _int(m, "vdim", where) != dim:
        raise ConfigError(f"config.json: {where}.vdim={m['vdim']} must be dim={dim}: the values are the keys")
    _number(m, "scale", where, positive=False)
    if m.get("mask") is not None:
        _int(_object(m, "mask", where), "size", where + ".mask")
    _check_rotation(m, where, dim)


def _check_latent(m: Mapping[str, Any], where: str) -> None:
    for key in ("heads", "dim", "vdim", "kv_rank"):
        _int(m, key, where)
    rot_dim = _int(m, "rot_dim", where, 0)
    _number(m, "scale", where, positive=False)
    _check_rotation(m, where, rot_dim)


def _check_mlstm(m: Mapping[str, Any], where: str) -> None:
    for key in ("heads", "dim", "vdim"):
        _int(m, key, where)
    _number(m, "gate_cap", where)


_MIXERS = {"attention": _check_attention, "latent_attention": _check_latent, "mlstm": _check_mlstm}


@dataclass(frozen=True)
class ZaduraxLayer:
    type: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]
    weights_of: Optional[int] = None


@dataclass(frozen=True)
class ZaduraxConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[ZaduraxLayer, ...]
    raw: Mapping[str, Any]

    architecture = "Zadurax"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "ZaduraxConfig":
        if raw.get("architecture") != cls.architecture:
            raise ConfigError(f"config.json: architecture must be {cls.architecture!r}; "
                              f"got {raw.get('architecture')!r}")
        vocab, width = _int(raw, "vocab", "config"), _int(raw, "width", "config")
        eps = _number(_object(raw, "norm", "config"), "eps", "norm")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: layers must be a list of at least one layer")
        layers: List[ZaduraxLayer] = []
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
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind {mlp.get('kind')!r} is not a feed-forward of "
                                      f"this design (dense)")
                _int(mlp, "ff", where + ".mlp")
            source = entry.get("weights_of")
            if source is not None:
                if isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < len(entries) \
                        or source == i:
                    raise ConfigError(f"config.json: {where}.weights_of must name another layer; got {source!r}")
                other = entries[source]
                if not isinstance(other, Mapping) or any(other.get(key) != entry.get(key)
                                                         for key in ("type", "mixer", "mlp")):
                    raise ConfigError(f"config.json: {where} uses the weights of layer {source} but differs from it")
            layers.append(ZaduraxLayer(kind, mixer, mlp, source))
        config = cls(vocab, width, eps, tuple(layers), dict(raw))
        for i in range(len(layers)):
            config.owner(i)
        return config

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses (itself, or the end of its chain of ``weights_of``)."""
        seen = [i]
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
            if i in seen:
                raise ConfigError(f"config.json: layers {seen} name each other's weights")
            seen.append(i)
        return i

    def to_dict(self) -> Dict[str, Any]:
        """The config.json that reads back as this configuration."""
        def plain(x):
            return {k: plain(v) for k, v in x.items()} if isinstance(x, Mapping) else x
        layers = []
        for l in self.layers:
            entry = {"type": l.type, "mixer": plain(l.mixer), "mlp": None if l.mlp is None else plain(l.mlp)}
            if l.weights_of is not None:
                entry["weights_of"] = l.weights_of
            layers.append(entry)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "layers": layers}

    # ------------------------------------------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "name": name, "leaf": ""})

    @staticmethod
    def _position(rot: Mapping[str, Any]) -> PartSpec:
        params = {"dims": rot["dims"], "base": rot["base"], "pairing": "neighbours"}
        if rot.get("scaling") is not None:
            params["scaling"] = {"ramp": "index", **rot["scaling"]}
        return PartSpec("rope_frequencies", params)

    def _mixer(self, layer: ZaduraxLayer) -> PartSpec:
        m = layer.mixer
        if layer.type == "attention":
            return PartSpec("sink_attention", {
                "hidden_size": self.width, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"],
                "vdim": m["vdim"], "scale": m["scale"],
                "window": min(m["mask"]["size"], MAX_POSITIONS) if m.get("mask") else 0, "values": "keys",
                "qk_norm": "head_weight", "gate": "value", "eps": self.norm_eps, "pad_heads": True,
                "position": self._position(m["rot"]), "leaf": "",
                "names": {"q": "mix.q", "k": "mix.k", "o": "mix.o", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm",
                          "gate": "mix.g"}})
        if layer.type == "latent_attention":
            return PartSpec("latent_attention", {
                "hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"],
                "vdim": m["vdim"], "q_rank": 0, "kv_rank": m["kv_rank"], "scale": m["scale"], "eps": self.norm_eps,
                "sink": True, "gate": "value", "position": self._position(m["rot"]), "leaf": "",
                "names": {"q": "mix.q", "dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm", "uk": "mix.uk", "uv": "mix.uv",
                          "sink": "mix.sink", "gate": "mix.g", "o": "mix.o"}})
        return PartSpec("matrix_memory", {
            "hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"],
            "gate_cap": m["gate_cap"], "floor": MEMORY_FLOOR, "eps": self.norm_eps, "leaf": "",
            "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "g": "mix.g", "o": "mix.o", "norm": "mix.norm",
                      "i": "mix.i", "i_bias": "mix.i.b", "f": "mix.f", "f_bias": "mix.f.b"}})

    def to_spec(self) -> ModelSpec:
        owners = [self.owner(i) for i in range(len(self.layers))]
        place: Dict[int, int] = {}  # a layer with tensors -> its place among those
        layers = []
        for i in sorted(set(owners)):
            layer = self.layers[i]
            parts = {"mixer_norm": self._norm("norm1"), "mixer": self._mixer(layer),
                     "mixer_post_norm": self._norm("norm1b")}
            if layer.mlp is not None:
                parts["ffn_norm"], parts["ffn_post_norm"] = self._norm("norm2"), self._norm("norm2b")
                parts["ffn"] = PartSpec("gated_mlp", {
                    "hidden_size": self.width, "intermediate_size": layer.mlp["ff"], "activation": "gelu_tanh",
                    "bias": False, "leaf": "", "names": {"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"}})
            place[i] = len(layers)
            layers.append(LayerSpec(prefix=f"l{i}", block="sandwich", parts=parts,
                                    params={"tolerated": () if layer.mlp is not None else ("norm2", "norm2b")}))
        spec = ModelSpec(
            architecture=self.architecture,
            hidden_size=self.width,
            vocab_size=self.vocab,
            max_positions=MAX_POSITIONS,
            embedding=PartSpec("normed_token_embedding", {"vocab_size": self.vocab, "hidden_size": self.width,
                                                          "name": "embed", "leaf": "",
                                                          "norm": self._norm("embed.norm")}),
            layers=tuple(layers),
            schedule=tuple(ScheduleEntry(place[i]) for i in owners),
            final_norm=self._norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": self.width, "name": "head",
                                          "leaf": ""}),
            stop_token_ids=(),
            stored_dtype="bfloat16",
        )
        spec.validate()
        return spec
