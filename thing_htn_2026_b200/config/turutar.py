"""Typed configuration of the Turutar decoder: a stack of layers given one by one over a float32 residual
stream, some of which may run several times in a row with the same weights.

The stream starts as the token's embedding behind an RMS norm.  A layer has one norm that both sublayers
read, and adds each sublayer's output times a vector of its own; then it adds what the token itself
brings to the layer::

    n = norm1(x),  x <- x + ls1 * mixer(n) + ls2 * ff(n)
    x <- x + norm(proj(gelu(gate x) * side[token, i * dim : (i + 1) * dim]))

The model's norms are RMS norms whose gain is stored around zero; the norms inside a mixer and the one of
the token's part have plain gains.

config.json keys::

    architecture      "Turutar"
    vocab, width      sizes of the embedding table ``embed`` [vocab, width] and the head ``head``
    norm.eps          eps of every norm of the model
    loop              {"start", "stop", "times"} (optional): layers start .. stop - 1 run times times in a row;
                      every pass has its own cache, and every pass but the first adds the stream's start first
    token_side.dim    columns of ``side.embed`` [vocab, layers * dim] per layer (absent: no such part)
    layers            a list; entry i has
        type   "attention" or "latent_attention"
        mixer  the mixer's sizes and constants, see below
        mlp    {"kind": "dense", "ff", "limit"} or null (no feed-forward in this layer)

    mixer of "attention":         heads, kv_heads, dim, vdim (= dim), scale, mask {"size"} (the window; absent: every
                                  earlier position).  No rotation; values are the keys as projected; biases of q
                                  and k; an RMS norm over all heads of q and one over all of k; one added to the
                                  softmax's denominator; a logistic gate per head.
    mixer of "latent_attention":  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {"base", "dims"} (dims =
                                  rot_dim; neighbouring entries make a pair): a learned sink and a logistic
                                  gate per head.

Tensor names: layer i's start with ``l<i>.``: ``norm1``, ``mix.*``, ``mlp.gate / up / down``, ``ls1``, ``ls2``,
``side.gate / proj / norm``; the embedding's norm is ``embed.norm``, the last one ``final.norm``.

One constant is the design's own and stands here: the slope of the feed-forward's logistic gate.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .base import ConfigError, LayerSpec, ModelConfig, ModelPlan, PartSpec, _freeze, looped_schedule, require

ATTENTION = "attention"
LATENT = "latent_attention"
KINDS = (ATTENTION, LATENT)
GLU_SLOPE = 1.702
UNIT_SINK = 0.0     # the score of the attention layers' sink: exp(0) = 1 is added to the denominator


def _section(data: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = data.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return value


def _int(data: Mapping[str, Any], key: str, where: str, minimum: int = 1) -> int:
    value = data.get(key)
    if isinstance(value, bool) or not isinstance(value, int) or value < minimum:
        raise ConfigError(f"config.json: {where}'{key}' must be an integer >= {minimum}, got {value!r}")
    return value


def _float(data: Mapping[str, Any], key: str, where: str) -> float:
    value = data.get(key)
    if isinstance(value, bool) or not isinstance(value, (int, float)) or not value > 0:
        raise ConfigError(f"config.json: {where}'{key}' must be a positive number, got {value!r}")
    return float(value)


@dataclass(frozen=True)
class TurutarConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    side_dim: int                                  # 0: no token input beside the layers
    loop: Optional[Tuple[int, int, int]]           # start, stop, times
    layers: Tuple[Mapping[str, Any], ...]
    max_positions: int = 1 << 20

    architecture = "Turutar"

    # ------------------------------------------------------------------ reading

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "TurutarConfig":
        layers = data.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        loop = None
        if data.get("loop") is not None:
            section = _section(data, "loop", "")
            loop = (_int(section, "start", "loop.", 0), _int(section, "stop", "loop."), _int(section, "times", "loop."))
        config = cls(
            vocab=require(data, "vocab", int),
            width=require(data, "width", int),
            norm_eps=_float(_section(data, "norm", ""), "eps", "norm."),
            side_dim=_int(_section(data, "token_side", ""), "dim", "token_side.") if data.get("token_side") is not None else 0,
            loop=loop,
            layers=tuple(_freeze(dict(layer)) for layer in layers),
            max_positions=int(data.get("max_positions", 1 << 20)),
        )
        config.validate()
        return config

    def validate(self) -> None:
        if self.loop is not None and not self.loop[0] < self.loop[1] <= len(self.layers):
            raise ConfigError(f"config.json: loop.start {self.loop[0]} and loop.stop {self.loop[1]} must name a run of the "
                              f"{len(self.layers)} layers")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            kind = layer.get("type")
            if kind not in KINDS:
                raise ConfigError(f"config.json: {where}'type' must be one of {', '.join(KINDS)}, got {kind!r}")
            mixer, at = _section(layer, "mixer", where), where + "mixer."
            heads = _int(mixer, "heads", at)
            _float(mixer, "scale", at)
            if kind == ATTENTION:
                kv_heads, dim, vdim = _int(mixer, "kv_heads", at), _int(mixer, "dim", at), _int(mixer, "vdim", at)
                if heads % kv_heads:
                    raise ConfigError(f"config.json: {at}heads {heads} is not a multiple of kv_heads {kv_heads}")
                if vdim != dim:
                    raise ConfigError(f"config.json: {at}vdim {vdim} differs from dim {dim}; the values of this attention "
                                      f"are its keys")
                if mixer.get("mask") is not None:
                    _int(_section(mixer, "mask", at), "size", at + "mask.")
                if mixer.get("rot") is not None:
                    raise ConfigError(f"config.json: {at}rot: positions do not enter the scores of this attention")
            else:
                for key in ("dim", "vdim", "q_rank", "kv_rank"):
                    _int(mixer, key, at)
                rot_dim = _int(mixer, "rot_dim", at, 0)
                if rot_dim:
                    rot = _section(mixer, "rot", at)
                    if rot_dim % 2 or _int(rot, "dims", at + "rot.") != rot_dim:
                        raise ConfigError(f"config.json: {at}rot.dims {rot['dims']} must be even and rot_dim, {rot_dim}")
                    _float(rot, "base", at + "rot.")
                if mixer.get("mask") is not None:
                    raise ConfigError(f"config.json: {at}mask: this mixer sees every earlier position")
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind must be 'dense', got {mlp.get('kind')!r}")
                _int(mlp, "ff", where + "mlp."), _float(mlp, "limit", where + "mlp.")

    def to_dict(self) -> dict:
        def thaw(value):
            if isinstance(value, Mapping):
                return {k: thaw(v) for k, v in value.items()}
            if isinstance(value, tuple):
                return [thaw(v) for v in value]
            return value
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": [thaw(layer) for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        return out

    # ------------------------------------------------------------------ the plan

    def _norm(self, name: str, offset: float = 1.0) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "gain_offset": offset, "residual": "float32"},
                        {"weight": name})

    def _mixer(self, layer: Mapping[str, Any], prefix: str) -> PartSpec:
        m = layer["mixer"]

        def names(**own):
            return {key: f"{prefix}mix.{name}" for key, name in own.items()}

        common = {"hidden_size": self.width, "n_heads": m["heads"], "scale": float(m["scale"]), "softmax_weights": "float32"}
        if layer["type"] == ATTENTION:
            mask = m.get("mask")
            return PartSpec("attention", {**common, "n_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                                          "window": None if mask is None else mask["size"], "qk_norm_eps": self.norm_eps,
                                          "qk_norm_scope": "projection", "values": "keys", "biases": ["q", "k"],
                                          "sinks": UNIT_SINK, "gate": "head", "position": None},
                            names(q_proj="q", q_bias="q.b", k_proj="k", k_bias="k.b", q_norm="q.norm", k_norm="k.norm",
                                  g_proj="g", o_proj="o"))
        position = None
        if m["rot_dim"]:
            position = PartSpec("rope", {"head_dim": m["rot_dim"], "rotary_dim": m["rot_dim"], "theta": float(m["rot"]["base"]),
                                         "layout": "interleaved", "frequency_precision": "float64",
                                         "angle_precision": "float64"})
        return PartSpec("latent_attention", {**common, "plain_dim": m["dim"], "rot_dim": m["rot_dim"], "value_dim": m["vdim"],
                                             "q_rank": m["q_rank"], "latent_rank": m["kv_rank"], "norm_eps": self.norm_eps,
                                             "position": position, "sinks": "learned", "gated": True, "gate_scope": "head"},
                        names(q_down="dq", q_norm="dq.norm", q_proj="uq", down_proj="dkv", latent_norm="dkv.norm", up_k="uk",
                              up_v="uv", sink="sink", g_proj="g", o_proj="o"))

    def _side(self, i: int, prefix: str) -> PartSpec:
        return PartSpec("token_rows", {"hidden_size": self.width, "vocab_size": self.vocab, "dim": self.side_dim,
                                       "column": i * self.side_dim, "table_width": len(self.layers) * self.side_dim,
                                       "norm": self._norm(prefix + "side.norm", offset=0.0)},
                        {"table": "side.embed", "gate": prefix + "side.gate", "proj": prefix + "side.proj"})

    def plan(self) -> ModelPlan:
        layers: List[LayerSpec] = []
        for i, layer in enumerate(self.layers):
            prefix = f"l{i}."
            mlp = layer.get("mlp")
            parts = dict(norm=self._norm(prefix + "norm1"), mixer=self._mixer(layer, prefix), layer_scale=True)
            tensors = {"mixer_scale": prefix + "ls1"}
            if mlp is not None:
                parts["ffn"] = PartSpec("clamped_glu", {"hidden_size": self.width, "intermediate_size": mlp["ff"],
                                                        "limit": float(mlp["limit"]), "slope": GLU_SLOPE},
                                        {"gate_proj": prefix + "mlp.gate", "up_proj": prefix + "mlp.up",
                                         "down_proj": prefix + "mlp.down"})
                tensors["ffn_scale"] = prefix + "ls2"
            if self.side_dim:
                parts["side"] = self._side(i, prefix)
            layers.append(LayerSpec(PartSpec("parallel", parts, tensors)))
        return ModelPlan(
            hidden_size=self.width,
            vocab_size=self.vocab,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": self.width, "stream": "float32",
                                             "norm": self._norm("embed.norm")}, {"weight": "embed"}),
            layers=tuple(layers),
            schedule=looped_schedule(len(layers), *(self.loop or ())),
            final_norm=self._norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False}, {"weight": "head"}),
            max_positions=self.max_positions,
        )
