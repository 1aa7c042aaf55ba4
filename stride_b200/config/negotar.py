"""Typed configuration of the Negotar decoder.

config.json gives ``vocab``, ``width``, ``norm.eps``, ``logit_scale`` and a list ``layers``; each entry has ``type`` (``attention`` or
``mamba2``), the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``: ``kind`` ``moe`` with ``expert.ff`` and
``router.experts``, ``router.top``; or null). Nothing else is read, and no size stands in code. The architecture is laid out from
the package's parts:

* a layer is the ``output_norm`` arrangement, ``x += norm(sublayer(x))``; norms are ``rmsnorm`` whose factor is one plus the stored
  weight;
* ``attention`` is the paged attention part with biases, a rotation of the first ``rot.dims`` entries of a head (halves paired,
  optionally with Llama 3.1's rescaled frequencies), unit norms on queries and keys behind the rotation, and optionally a cap on the
  scores; layers with ``v_mix`` blend their values with those of the first such layer;
* ``mamba2`` is the selective state space mixer;
* the mixture is ``routed_experts`` with plain gated units, sigmoid scores used as they are, on the experts' inputs;
* the head shares the embedding table; ``logit_scale`` is a factor of the final norm, which stands right in front of it.

The design names no longest sequence; ``max_positions`` only sizes the rotation tables and is grown on demand
(``with_max_positions``).
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass, field

from .registry import ConfigError, register_architecture
from .specs import FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, RopeScaling, default_schedule

MIXERS = ("attention", "mamba2")
DEFAULT_MAX_POSITIONS = 32768
MAX_HEAD, MAX_STATE, MAX_TAPS, MAX_EXPERTS, MAX_TOP = 256, 256, 16, 256, 32       # what the kernels take
_KNOWN = ("architecture", "architectures", "vocab", "width", "layers", "norm", "logit_scale", "max_positions")


def _int(d, key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, int) or v < minimum:
        raise ConfigError(f"{where}: `{key}` must be an integer >= {minimum}, got {v!r}")
    return v


def _num(d, key: str, where: str) -> float:
    v = d.get(key) if isinstance(d, dict) else None
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"{where}: `{key}` must be a number, got {v!r}")
    return float(v)


def _check_attention(m: dict, where: str) -> None:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"{where}: {heads} heads do not group into {kv} kv_heads")
    dim, vdim = _int(m, "dim", where), _int(m, "vdim", where)
    if dim > MAX_HEAD or vdim > MAX_HEAD:
        raise ConfigError(f"{where}: head sizes up to {MAX_HEAD} are supported, got dim {dim} and vdim {vdim}")
    _num(m, "scale", where)
    if m.get("softcap") is not None and not _num(m, "softcap", where) > 0:
        raise ConfigError(f"{where}: softcap must be positive")
    if not isinstance(m.get("v_mix", False), bool):
        raise ConfigError(f"{where}: v_mix must be true or false")
    rot = m.get("rot")
    if rot is None:             # no rotation
        return
    if not isinstance(rot, dict):
        raise ConfigError(f"{where}: `rot` must be an object with `base` and `dims`, or null")
    dims = _int(rot, "dims", where + ".rot", minimum=0)
    if dims % 2 or dims > dim or not _num(rot, "base", where + ".rot") > 0:
        raise ConfigError(f"{where}: rot.dims must be even and at most dim, rot.base positive")
    sc = rot.get("scaling")
    if sc is not None:
        for key in ("factor", "low", "high", "original"):
            if not _num(sc, key, where + ".rot.scaling") > 0:
                raise ConfigError(f"{where}.rot.scaling: `{key}` must be positive")
        if not sc["high"] >= sc["low"]:
            raise ConfigError(f"{where}.rot.scaling: high must not lie below low")


def _check_mamba2(m: dict, where: str) -> None:
    heads, groups = _int(m, "heads", where), _int(m, "groups", where)
    if heads % groups:
        raise ConfigError(f"{where}: {heads} heads do not divide into {groups} groups")
    if _int(m, "state", where) > MAX_STATE:
        raise ConfigError(f"{where}: a state of up to {MAX_STATE} is supported, got {m['state']}")
    if _int(m, "conv", where) > MAX_TAPS:
        raise ConfigError(f"{where}: up to {MAX_TAPS} taps are supported, got {m['conv']}")
    inner = heads * _int(m, "vdim", where)
    if inner % _int(m, "norm_groups", where):
        raise ConfigError(f"{where}: {inner} inner channels do not divide into {m['norm_groups']} norm_groups")


def _check_mlp(mlp, where: str) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"{where}: `mlp` must be null or have `kind` 'moe'")
    _int(mlp.get("expert"), "ff", where + ".expert")
    experts, top = _int(mlp.get("router"), "experts", where + ".router"), _int(mlp.get("router"), "top", where + ".router")
    if top > experts or experts > MAX_EXPERTS or top > MAX_TOP:
        raise ConfigError(f"{where}.router: up to {MAX_TOP} of up to {MAX_EXPERTS} experts are supported, got {top} of {experts}")


@dataclass(frozen=True)
class NegotarConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers_json: str                        # the ``layers`` list as canonical JSON (keeps the record hashable)
    max_position_embeddings: int = DEFAULT_MAX_POSITIONS
    extra: dict = field(default_factory=dict, compare=False)

    @property
    def layers(self) -> list:
        return json.loads(self.layers_json)

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: dict) -> "NegotarConfig":
        for key in ("vocab", "width", "layers", "norm", "logit_scale"):
            if key not in d:
                raise ConfigError(f"config.json is missing `{key}`")
        if not isinstance(d["norm"], dict):
            raise ConfigError("`norm` must be an object with `eps`")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("`layers` must be a list with at least one layer")
        cfg = cls(vocab=_int(d, "vocab", "config.json"), width=_int(d, "width", "config.json"), norm_eps=_num(d["norm"], "eps", "norm"),
                  logit_scale=_num(d, "logit_scale", "config.json"), layers_json=json.dumps(d["layers"], sort_keys=True),
                  max_position_embeddings=int(d.get("max_positions", DEFAULT_MAX_POSITIONS)),
                  extra={k: v for k, v in d.items() if k not in _KNOWN})
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.norm_eps >= 0:
            raise ConfigError("norm.eps must not be negative")
        first_values = None         # (layer, sizes) of the first layer that takes part in the value mixing
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXERS:
                raise ConfigError(f"{where}: `type` must be one of {MIXERS}, got {layer.get('type') if isinstance(layer, dict) else layer!r}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"{where}: `mixer` must be an object")
            if layer["type"] == "mamba2":
                _check_mamba2(m, where)
            else:
                _check_attention(m, where)
                if m.get("v_mix"):
                    sizes = (m["kv_heads"], m["vdim"])
                    if first_values is None:
                        first_values = (i, sizes)
                    elif sizes != first_values[1]:
                        raise ConfigError(f"{where}: values of {sizes[0]} x {sizes[1]} cannot be mixed with those of layer {first_values[0]}, "
                                          f"{first_values[1][0]} x {first_values[1][1]}")
            _check_mlp(layer.get("mlp"), where + ".mlp")

    def to_dict(self) -> dict:
        d = {"architecture": "Negotar", "layers": self.layers, "logit_scale": self.logit_scale, "norm": {"eps": self.norm_eps},
             "vocab": self.vocab, "width": self.width}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_position_embeddings
        d.update(copy.deepcopy(self.extra))
        return d

    def with_max_positions(self, count: int) -> "NegotarConfig":
        import dataclasses
        return dataclasses.replace(self, max_position_embeddings=int(count))

    # ------------------------------------------------------------------- layout
    def _norm(self, name: str, *params) -> NormSpec:
        return NormSpec(kind="rmsnorm", width=self.width, eps=self.norm_eps, prefix=name, params=(("tensor", name), ("weight_offset", 1.0), *params))

    def _attention(self, m: dict, prefix: str, mixing: str | None) -> MixerSpec:
        rot, scaling = m.get("rot") or {"base": 1.0, "dims": 0}, None
        sc = rot.get("scaling")
        if sc:
            scaling = RopeScaling(rope_type="llama3", factor=float(sc["factor"]), low_freq_factor=float(sc["low"]),
                                  high_freq_factor=float(sc["high"]), original_max_position_embeddings=sc["original"])
        position = PositionSpec(kind="rope", head_dim=m["dim"], theta=float(rot["base"]), max_positions=self.max_position_embeddings,
                                scaling=scaling, params=(("angles", "float64"), ("rotated", int(rot["dims"]))))
        params = [("names", "short"), ("value_dim", m["vdim"]), ("qk_norm", "unit_rotated"), ("norm_eps", self.norm_eps), ("padded_heads", True)]
        if m.get("softcap") is not None:
            params += [("softcap", float(m["softcap"])), ("precise_cap", True)]
        if mixing is not None:
            params.append(("value_mix", mixing))
        return MixerSpec(kind="attention", hidden=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                         scale=float(m["scale"]), bias=True, position=position, prefix=prefix, params=tuple(params))

    def _mamba2(self, m: dict, prefix: str) -> MixerSpec:
        return MixerSpec(kind="mamba2", hidden=self.width, num_heads=m["heads"], head_dim=m["vdim"], prefix=prefix,
                         params=(("groups", m["groups"]), ("state", m["state"]), ("taps", m["conv"]), ("norm_groups", m["norm_groups"]),
                                 ("norm_eps", self.norm_eps)))

    def to_model_spec(self) -> ModelSpec:
        layers, ignorable, values_seen = [], [], False
        for i, layer in enumerate(self.layers):
            p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
            if layer["type"] == "mamba2":
                mixer = self._mamba2(m, p + "mix.")
            else:
                mixing = ("later" if values_seen else "first") if m.get("v_mix") else None
                values_seen = values_seen or mixing is not None
                mixer = self._attention(m, p + "mix.", mixing)
                if mixing is None:
                    ignorable.append(p + "mix.vmix")
            ffn = None
            if mlp is not None:
                r = mlp["router"]
                ffn = FeedForwardSpec(kind="routed_experts", hidden=self.width, intermediate=mlp["expert"]["ff"], activation="silu",
                                      prefix=p + "mlp.", params=(("experts", r["experts"]), ("top", r["top"]), ("router", "sigmoid_scores"),
                                                                 ("weigh", "inputs")))
            else:
                ignorable.append(p + "norm2")
            layers.append(LayerSpec(kind="output_norm", mixer=mixer, feed_forward=ffn, mixer_norm=self._norm(p + "norm1"),
                                    ffn_norm=self._norm(p + "norm2") if ffn is not None else None))
        return ModelSpec(architecture="Negotar", hidden=self.width, vocab=self.vocab, layers=tuple(layers), schedule=default_schedule(len(layers)),
                         final_norm=self._norm("final.norm", ("factor", self.logit_scale)), embed_name="embed", head_name=None,
                         max_positions=self.max_position_embeddings, ignorable_tensors=tuple(ignorable), extra=self)


register_architecture("Negotar", NegotarConfig)
