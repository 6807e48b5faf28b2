"""Typed configuration of the Futepel decoder: a stack of layers given one by one over a plain float32
residual stream, each layer with a token mixer of one of three kinds and an optional feed-forward,
dense or a mixture of experts.

The stream starts as the token's embedding times ``embedding.scale``, plus a row for the pair of the
token before and the token, plus a learned vector for the position.  A layer does
``x <- x + mixer(norm1(x))`` and, where it has a feed-forward, ``x <- x + ff(norm2(x))``, both norms RMS
norms; the model ends with such a norm and the head.

config.json keys::

    architecture      "Futepel"
    vocab, width      sizes of the embedding table ``embed`` [vocab, width] and the head ``head``
    embedding.scale   the factor on the embedding (default 1)
    embedding.bigram  {"buckets", "mul_prev", "mul_cur"}: the pair (b, t) takes row
                      (b mul_prev + t mul_cur) mod buckets of ``bigram`` [buckets + 1, width], a first
                      token the last row (absent: no pairs)
    max_positions     rows of the position table ``pos``; no sequence is longer
    norm.eps          eps of every norm of the model
    layers            a list; entry i has
        type   "wkv", "latent_attention" or "mamba2"
        mixer  the mixer's sizes and constants, see below
        mlp    {"kind": "dense", "ff"}, {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"},
                "shared": {"ff"} (optional)} or null (no feed-forward in this layer)

    mixer of "wkv":               heads, dim: time mixing.  ``rank`` (optional): the channels between the decay's two
                                  projections; without it the shapes of the checkpoint's two tensors give it
                                  (random weights need it).
    mixer of "latent_attention":  heads, dim, rot_dim, vdim, kv_rank, scale, rot {"base", "dims", "scaling" (optional)
                                  {"factor", "original", "fast", "slow"}}: latent attention over all earlier
                                  positions, rotation of entry i with entry i + dims/2 of the rotated parts
                                  (dims = rot_dim), a logistic gate per head.
    mixer of "mamba2":            heads, vdim, state, groups, conv, norm_groups: state-space duality.

Tensor names: layer i's start with ``l<i>.``; its norms are ``norm1`` and ``norm2``, its mixer's tensors
``mix.*``, its feed-forward's ``mlp.up / down`` or ``mlp.router``, ``mlp.e<j>.gate / up / down``,
``mlp.shared.gate / up / down``; the model's last norm is ``final.norm``.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .base import ConfigError, LayerSpec, ModelConfig, ModelPlan, PartSpec, ScheduleEntry, _freeze, require

WKV = "wkv"
LATENT = "latent_attention"
MAMBA2 = "mamba2"
KINDS = (WKV, LATENT, MAMBA2)


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
class FutepelConfig(ModelConfig):
    vocab: int
    width: int
    embedding_scale: float
    bigram: Optional[Mapping[str, int]]
    max_positions: int
    norm_eps: float
    layers: Tuple[Mapping[str, Any], ...]

    architecture = "Futepel"

    # ------------------------------------------------------------------ reading

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "FutepelConfig":
        layers = data.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        embedding = data.get("embedding") or {}
        bigram = None
        if embedding.get("bigram") is not None:
            section, at = _section(embedding, "bigram", "embedding."), "embedding.bigram."
            bigram = _freeze({"buckets": _int(section, "buckets", at), "mul_prev": _int(section, "mul_prev", at, 0),
                              "mul_cur": _int(section, "mul_cur", at, 0)})
        config = cls(
            vocab=require(data, "vocab", int),
            width=require(data, "width", int),
            embedding_scale=_float(embedding, "scale", "embedding.") if "scale" in embedding else 1.0,
            bigram=bigram,
            max_positions=require(data, "max_positions", int),
            norm_eps=_float(_section(data, "norm", ""), "eps", "norm."),
            layers=tuple(_freeze(dict(layer)) for layer in layers),
        )
        config.validate()
        return config

    def validate(self) -> None:
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            kind = layer.get("type")
            if kind not in KINDS:
                raise ConfigError(f"config.json: {where}'type' must be one of {', '.join(KINDS)}, got {kind!r}")
            mixer, at = _section(layer, "mixer", where), where + "mixer."
            if kind == WKV:
                _int(mixer, "heads", at), _int(mixer, "dim", at)
                if mixer.get("rank") is not None:
                    _int(mixer, "rank", at)
            elif kind == LATENT:
                for key in ("heads", "dim", "vdim", "kv_rank"):
                    _int(mixer, key, at)
                rot_dim = _int(mixer, "rot_dim", at, 0)
                _float(mixer, "scale", at)
                if rot_dim:
                    rot = _section(mixer, "rot", at)
                    if rot_dim % 2 or _int(rot, "dims", at + "rot.") != rot_dim:
                        raise ConfigError(f"config.json: {at}rot.dims {rot['dims']} must be even and rot_dim, {rot_dim}")
                    _float(rot, "base", at + "rot.")
                    if rot.get("scaling") is not None:
                        for key in ("factor", "original", "fast", "slow"):
                            _float(_section(rot, "scaling", at + "rot."), key, at + "rot.scaling.")
                for key in ("mask", "window"):
                    if mixer.get(key) is not None:
                        raise ConfigError(f"config.json: {at}{key}: this mixer sees every earlier position")
            else:
                heads, vdim, groups = _int(mixer, "heads", at), _int(mixer, "vdim", at), _int(mixer, "groups", at)
                _int(mixer, "state", at), _int(mixer, "conv", at)
                if heads % groups:
                    raise ConfigError(f"config.json: {at}heads {heads} is not a multiple of groups {groups}")
                if heads * vdim % _int(mixer, "norm_groups", at):
                    raise ConfigError(f"config.json: {at}norm_groups {mixer['norm_groups']} does not divide heads * vdim, {heads * vdim}")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            at = where + "mlp."
            if mlp.get("kind") == "dense":
                _int(mlp, "ff", at)
            elif mlp.get("kind") == "moe":
                _int(_section(mlp, "expert", at), "ff", at + "expert.")
                router = _section(mlp, "router", at)
                experts, top = _int(router, "experts", at + "router."), _int(router, "top", at + "router.")
                if top > experts:
                    raise ConfigError(f"config.json: {at}router.top {top} is more than the {experts} experts")
                if mlp.get("shared") is not None:
                    _int(_section(mlp, "shared", at), "ff", at + "shared.")
            else:
                raise ConfigError(f"config.json: {at}kind must be 'dense' or 'moe', got {mlp.get('kind')!r}")

    def to_dict(self) -> dict:
        def thaw(value):
            if isinstance(value, Mapping):
                return {k: thaw(v) for k, v in value.items()}
            if isinstance(value, tuple):
                return [thaw(v) for v in value]
            return value
        embedding = {"scale": self.embedding_scale}
        if self.bigram is not None:
            embedding["bigram"] = thaw(self.bigram)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": embedding,
                "max_positions": self.max_positions, "norm": {"eps": self.norm_eps},
                "layers": [thaw(layer) for layer in self.layers]}

    # ------------------------------------------------------------------ the plan

    def _norm(self, name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": self.width, "eps": self.norm_eps, "residual": "float32"}, {"weight": name})

    def _mixer(self, layer: Mapping[str, Any], prefix: str) -> PartSpec:
        m, kind = layer["mixer"], layer["type"]

        def names(**own):
            return {key: f"{prefix}mix.{name}" for key, name in own.items()}

        if kind == WKV:
            return PartSpec("time_mixing", {"hidden_size": self.width, "n_heads": m["heads"], "dim": m["dim"],
                                            "rank": m.get("rank"), "norm_eps": self.norm_eps},
                            names(mu_r="mu.r", mu_k="mu.k", mu_v="mu.v", mu_g="mu.g", mu_w="mu.w", r="r", k="k", v="v", g="g",
                                  w1="w1", w2="w2", w0="w0", u="u", norm="norm", o="o"))
        if kind == MAMBA2:
            return PartSpec("state_space", {"hidden_size": self.width, "n_heads": m["heads"], "value_dim": m["vdim"],
                                            "state": m["state"], "groups": m["groups"], "conv_taps": m["conv"],
                                            "norm_groups": m["norm_groups"], "norm_eps": self.norm_eps},
                            names(**{"in": "in"}, conv="conv", conv_bias="conv.b", dt_bias="dt_bias", A_log="A_log", D="D",
                                  norm="norm", o="o"))
        position = None
        if m["rot_dim"]:
            rot = m["rot"]
            position = PartSpec("rope", {"head_dim": m["rot_dim"], "rotary_dim": m["rot_dim"], "theta": float(rot["base"]),
                                         "layout": "half", "frequency_precision": "float64", "angle_precision": "float64",
                                         "scaling": rot.get("scaling")})
        return PartSpec("latent_attention", {"hidden_size": self.width, "n_heads": m["heads"], "plain_dim": m["dim"],
                                             "rot_dim": m["rot_dim"], "value_dim": m["vdim"], "latent_rank": m["kv_rank"],
                                             "scale": float(m["scale"]), "norm_eps": self.norm_eps, "position": position,
                                             "gated": True, "gate_scope": "head", "softmax_weights": "float32"},
                        names(q_proj="q", down_proj="dkv", latent_norm="dkv.norm", up_k="uk", up_v="uv", g_proj="g", o_proj="o"))

    def _ffn(self, mlp: Mapping[str, Any], prefix: str) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("squared_relu", {"hidden_size": self.width, "intermediate_size": mlp["ff"]},
                            {"up_proj": prefix + "mlp.up", "down_proj": prefix + "mlp.down"})
        router, shared = mlp["router"], mlp.get("shared")
        tensors = {"router": prefix + "mlp.router"}
        for e in range(router["experts"]):
            for name in ("gate", "up", "down"):
                tensors[f"{name}.{e}"] = f"{prefix}mlp.e{e}.{name}"
        if shared is not None:
            tensors.update(shared_gate_proj=prefix + "mlp.shared.gate", shared_up=prefix + "mlp.shared.up",
                           shared_down=prefix + "mlp.shared.down")
        return PartSpec("routed_glu_experts",
                        {"hidden_size": self.width, "n_experts": router["experts"], "expert_ff": mlp["expert"]["ff"],
                         "top": router["top"], "shared_ff": 0 if shared is None else shared["ff"]}, tensors)

    def plan(self) -> ModelPlan:
        layers: List[LayerSpec] = []
        for i, layer in enumerate(self.layers):
            prefix = f"l{i}."
            parts = dict(norm_mixer=self._norm(prefix + "norm1"), mixer=self._mixer(layer, prefix))
            if layer.get("mlp") is not None:
                parts.update(norm_ffn=self._norm(prefix + "norm2"), ffn=self._ffn(layer["mlp"], prefix))
            layers.append(LayerSpec.of("pre_norm", **parts))
        embedding = {"vocab_size": self.vocab, "hidden_size": self.width, "scale": self.embedding_scale, "stream": "float32",
                     "positions": {"kind": "learned", "size": self.max_positions}}
        tensors = {"weight": "embed", "positions": "pos"}
        if self.bigram is not None:
            embedding["pairs"] = {"buckets": self.bigram["buckets"], "mul_before": self.bigram["mul_prev"],
                                  "mul_token": self.bigram["mul_cur"]}
            tensors["pairs"] = "bigram"
        return ModelPlan(
            hidden_size=self.width,
            vocab_size=self.vocab,
            embedding=PartSpec("embedding", embedding, tensors),
            layers=tuple(layers),
            schedule=tuple(ScheduleEntry(layer=i, cache=i) for i in range(len(layers))),
            final_norm=self._norm("final.norm"),
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": self.width, "tied": False}, {"weight": "head"}),
            max_positions=self.max_positions,
        )
