"""Typed configuration of the Dopudra decoder.

config.json gives ``vocab``, ``width``, ``streams``, ``max_positions``, ``embedding.scale``, ``norm.eps`` and a list ``layers``. A
layer entry has ``type`` (``lightning`` or ``parallel``), the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``:
``kind`` ``dense`` with ``ff``, or null). Sizes that no key names are read off the checkpoint: the rows of a distance table, the
inner width of a low-rank product, and the longest sequence where ``max_positions`` is left out. Nothing else is read, and no size
stands in code. The architecture is laid out from the package's parts:

* the embedding is ``lookup`` with a factor and a learned vector per position (tensor ``pos``); ``max_positions`` is therefore a
  hard limit;
* the residual stream is kept in ``streams`` copies and a layer is the ``copies`` arrangement: a norm before either sublayer, a
  learned vector (``ls1``, ``ls2``) on what it gives, and learned numbers (``hc1``, ``hc2``) for what it reads of the copies and how
  the copies mix and take its output;
* ``lightning`` is the matrix memory with a constant decay per head;
* ``parallel`` is two mixers on one input: paged attention without rotation (a short convolution, norms over whole projections,
  queries that grow with the position, a learned number per head and distance) beside a matrix memory whose key channels fade
  by factors of the token's own;
* the feed-forward is ``mlp`` with the square of relu;
* final norm ``final.norm``, an output head of its own (``head``).
"""

from __future__ import annotations

import copy
import json
from dataclasses import dataclass, field

from .registry import ConfigError, register_architecture
from .specs import EmbeddingSpec, FeedForwardSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec, default_schedule

MIXERS = ("lightning", "parallel")
_KNOWN = ("architecture", "architectures", "vocab", "width", "layers", "norm", "embedding", "streams", "max_positions")


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


def _check_memory(m: dict, where: str) -> None:
    _int(m, "heads", where), _int(m, "vdim", where)
    if _int(m, "dim", where) > 256:
        raise ConfigError(f"{where}: dim up to 256 is supported, got {m['dim']}")


def _check_lightning(m: dict, where: str) -> None:
    _check_memory(m, where)
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != m["heads"] or any(
            isinstance(x, bool) or not isinstance(x, (int, float)) or not 0 <= x <= 1 for x in decay):
        raise ConfigError(f"{where}: `decay` must list one number from 0 to 1 for each of the {m['heads']} heads")


def _check_attention(m: dict, where: str) -> None:
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"{where}: {heads} heads do not group into {kv} kv_heads")
    if _int(m, "dim", where) > 256 or _int(m, "vdim", where) > 256:
        raise ConfigError(f"{where}: head sizes up to 256 are supported, got dim {m['dim']} and vdim {m['vdim']}")
    if not _num(m, "scale", where) > 0:
        raise ConfigError(f"{where}: scale must be positive")
    if m.get("conv") is not None and _int(m, "conv", where) > 16:
        raise ConfigError(f"{where}: up to 16 taps are supported")
    if m.get("q_temp") is not None:
        _num(m["q_temp"], "coef", where + ".q_temp"), _int(m["q_temp"], "every", where + ".q_temp")
    _int(m, "bias_max", where)
    if "buckets" in m:
        buckets = _int(m, "buckets", where, minimum=2)
        if m["bias_max"] <= buckets // 2:
            raise ConfigError(f"{where}: bias_max {m['bias_max']} must lie beyond half of the {buckets} buckets")


def _check_channel_decay(m: dict, where: str) -> None:
    _check_memory(m, where)
    if not _num(m, "tau", where) > 0:
        raise ConfigError(f"{where}: tau must be positive")
    if "decay_rank" in m:
        _int(m, "decay_rank", where)


@dataclass(frozen=True)
class DopudraConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    embedding_scale: float
    max_position_embeddings: int            # rows of the table of learned position vectors: no longer sequence can run
    layers_json: str                        # the ``layers`` list as canonical JSON (keeps the record hashable)
    extra: dict = field(default_factory=dict, compare=False)

    @property
    def layers(self) -> list:
        return json.loads(self.layers_json)

    # ------------------------------------------------------------------ reading
    @staticmethod
    def complete_from_checkpoint(d: dict, tensor_names: set, tensor_shapes: dict | None = None) -> dict:
        """Fills in what only a tensor's shape gives: the buckets of ``rel``, the rank of ``a1``, the positions of ``pos``."""
        if not tensor_shapes or not isinstance(d.get("layers"), list):
            return d
        d = copy.deepcopy(d)

        def rows(name):
            shape = tensor_shapes.get(name)
            return int(shape[0]) if shape else None

        if "max_positions" not in d and rows("pos"):
            d["max_positions"] = rows("pos")
        for i, layer in enumerate(d["layers"]):
            m = layer.get("mixer") if isinstance(layer, dict) else None
            if not isinstance(m, dict) or layer.get("type") != "parallel":
                continue
            for side, key, tensor in (("left", "buckets", "rel"), ("right", "decay_rank", "a1")):
                count = rows(f"l{i}.mix.{side}.{tensor}")
                if isinstance(m.get(side), dict) and key not in m[side] and count:
                    m[side][key] = count
        return d

    @classmethod
    def from_dict(cls, d: dict) -> "DopudraConfig":
        for key in ("vocab", "width", "layers", "norm", "embedding", "streams", "max_positions"):
            if key not in d:
                raise ConfigError(f"config.json is missing `{key}`")
        for key, inner in (("norm", "eps"), ("embedding", "scale")):
            if not isinstance(d[key], dict):
                raise ConfigError(f"`{key}` must be an object with `{inner}`")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("`layers` must be a list with at least one layer")
        cfg = cls(vocab=_int(d, "vocab", "config.json"), width=_int(d, "width", "config.json"), streams=_int(d, "streams", "config.json"),
                  norm_eps=_num(d["norm"], "eps", "norm"), embedding_scale=_num(d["embedding"], "scale", "embedding"),
                  max_position_embeddings=_int(d, "max_positions", "config.json"), layers_json=json.dumps(d["layers"], sort_keys=True),
                  extra={k: v for k, v in d.items() if k not in _KNOWN})
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.norm_eps >= 0:
            raise ConfigError("norm.eps must not be negative")
        if self.streams > 16:
            raise ConfigError(f"up to 16 streams are supported, got {self.streams}")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or layer.get("type") not in MIXERS:
                raise ConfigError(f"{where}: `type` must be one of {MIXERS}, got {layer.get('type') if isinstance(layer, dict) else layer!r}")
            m = layer.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"{where}: `mixer` must be an object")
            if layer["type"] == "lightning":
                _check_lightning(m, where)
            else:
                if not isinstance(m.get("left"), dict) or not isinstance(m.get("right"), dict):
                    raise ConfigError(f"{where}: a parallel mixer needs `left` and `right`")
                _check_attention(m["left"], where + ".left")
                _check_channel_decay(m["right"], where + ".right")
                _num(m, "left_scale", where), _num(m, "right_scale", where)
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"{where}: `mlp` must be null or have `kind` 'dense'")
                _int(mlp, "ff", where + ".mlp")

    def to_dict(self) -> dict:
        d = {"architecture": "Dopudra", "layers": self.layers, "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
             "streams": self.streams, "max_positions": self.max_position_embeddings, "vocab": self.vocab, "width": self.width}
        d.update(copy.deepcopy(self.extra))
        return d

    # ------------------------------------------------------------------- layout
    def _norm(self, name: str) -> NormSpec:
        return NormSpec(kind="rmsnorm", width=self.width, eps=self.norm_eps, prefix=name, params=(("tensor", name),))

    def _attention(self, m: dict, prefix: str) -> MixerSpec:
        params = [("names", "short"), ("value_dim", m["vdim"]), ("qk_norm", "rows"), ("norm_eps", self.norm_eps),
                  ("distance_table", (int(m.get("buckets", 0)), m["bias_max"], self.max_position_embeddings))]
        if m.get("conv"):
            params.append(("conv", m["conv"]))
        if m.get("q_temp"):
            params.append(("query_factor", (float(m["q_temp"]["coef"]), m["q_temp"]["every"])))
        return MixerSpec(kind="attention", hidden=self.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"],
                         scale=float(m["scale"]), position=PositionSpec(kind="none"), prefix=prefix, params=tuple(params))

    def _mixer(self, layer: dict, prefix: str) -> MixerSpec:
        m = layer["mixer"]
        if layer["type"] == "lightning":
            return MixerSpec(kind="lightning", hidden=self.width, num_heads=m["heads"], head_dim=m["dim"], prefix=prefix,
                             params=(("value_dim", m["vdim"]), ("decay", tuple(float(x) for x in m["decay"])), ("norm_eps", self.norm_eps)))
        r = m["right"]
        right = MixerSpec(kind="channel_decay", hidden=self.width, num_heads=r["heads"], head_dim=r["dim"], prefix=prefix + "right.",
                          params=(("value_dim", r["vdim"]), ("tau", float(r["tau"])), ("norm_eps", self.norm_eps),
                                  ("decay_rank", int(r.get("decay_rank", 0)))))
        left = self._attention(m["left"], prefix + "left.")
        return MixerSpec(kind="parallel", hidden=self.width, prefix=prefix,
                         params=(("branches", ((left, float(m["left_scale"])), (right, float(m["right_scale"])))),))

    def to_model_spec(self) -> ModelSpec:
        layers = []
        for i, layer in enumerate(self.layers):
            p, mlp = f"l{i}.", layer.get("mlp")
            ffn = None
            params = [("copies", self.streams), ("mixer_copies", p + "hc1."), ("mixer_scale", p + "ls1")]
            if mlp is not None:
                ffn = FeedForwardSpec(kind="mlp", hidden=self.width, intermediate=mlp["ff"], activation="relu2", prefix=p + "mlp.")
                params += [("ffn_copies", p + "hc2."), ("ffn_scale", p + "ls2")]
            layers.append(LayerSpec(kind="copies", mixer=self._mixer(layer, p + "mix."), feed_forward=ffn, mixer_norm=self._norm(p + "norm1"),
                                    ffn_norm=self._norm(p + "norm2") if ffn is not None else None, params=tuple(params)))
        embedding = EmbeddingSpec("lookup", self.vocab, self.width, "embed",
                                  params=(("scale", self.embedding_scale), ("positions", ("pos", self.max_position_embeddings))))
        return ModelSpec(architecture="Dopudra", hidden=self.width, vocab=self.vocab, layers=tuple(layers), schedule=default_schedule(len(layers)),
                         final_norm=self._norm("final.norm"), embed_name="embed", head_name="head", max_positions=self.max_position_embeddings,
                         extra=self, embedding=embedding, copies=self.streams)


register_architecture("Dopudra", DopudraConfig)
