"""Typed configuration of the Pekodra decoder, read from its own config.json keys.

A Pekodra model is a list of layers around a float32 residual stream. A layer norms the stream twice, with two weights
stored around zero (x / sqrt(mean(x^2) + eps) * (1 + w)), and hands one result to its mixer and the other to its
feed-forward; both are added to the stream at once: x += mixer(norm1(x)) + ff(norm2(x)). The mixer is ``attention``:
grouped-query softmax attention inside a sliding window (position i sees the ``mask.size`` tokens up to itself), without
biases, value heads of a size of their own, rotate-half rotary positions on the first ``rot.dims`` channels of a head
with rates blended by the pair's index (``rot.scaling``) and tables scaled by 0.1 ln(factor) + 1, every head of q and k
divided by its root mean square after the rotation (no weight), the score scale of the configuration. The feed-forward
is ``dense`` (W_down (gelu(W_gate h + b) * (W_up h + b)) + b with the tanh form of gelu), ``moe`` (a float32 router,
the ``top`` largest logits, weights the softmax over those alone, ungated experts W_down relu(W_up h)^2, and one more
of them that every token passes), or none. The embedding's rows are multiplied by ``embedding.scale``. ``loop`` runs the
layers ``start .. stop - 1`` ``times`` times in a row with the same weights, every pass with a cache of its own, and in
front of every pass the stream x becomes W_in [x; x0] with x0 the embedding's output. The head is a tensor of its own;
the logits are multiplied by ``logit_scale``.

Checkpoint names: ``embed``, ``loop.in``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.{q,k,v,o}``,
``l<i>.mlp.{gate,up,down}`` (each with ``.b``), ``l<i>.mlp.{router,e<j>.{up,down},shared.{up,down}}``, ``final.norm``,
``head``.
"""

from __future__ import annotations

import json
import math
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping, Optional, Tuple

from .girelix import _freeze, _int, _number, _thaw
from .kidarax import _rope, _rot
from .lfm2 import ConfigError
from .specs import AttentionSpec, GatedMLPSpec, LayerSpec, ModelSpec, RMSNormSpec, RoutedExpertsSpec, ScheduleEntry

ARCHITECTURE = "Pekodra"
MIXER_TYPES = ("attention",)
MLP_KINDS = ("dense", "moe")
JOIN = "loop.in"


@dataclass(frozen=True)
class PekodraLayer:
    """One entry of ``layers``: its type and what config.json gives for its mixer and its feed-forward (None: none),
    kept as nested tuples so that the layer can be hashed."""

    type: str
    mixer: tuple
    mlp: Optional[tuple]

    @property
    def mixer_options(self) -> dict:
        return _thaw(self.mixer)

    @property
    def mlp_options(self) -> Optional[dict]:
        return None if self.mlp is None else _thaw(self.mlp)


@dataclass(frozen=True)
class PekodraConfig:
    width: int
    vocab: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[PekodraLayer, ...]
    loop: Optional[Tuple[int, int, int]] = None  # (start, stop, times)
    eos_token_id: Optional[int] = None

    architecture = ARCHITECTURE

    # ------------------------------------------------------------------ reading

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "PekodraConfig":
        if data.get("architecture") != ARCHITECTURE:
            raise ConfigError(f"architecture {data.get('architecture')!r} is not {ARCHITECTURE!r}")
        width = _int("config", data, "width")
        vocab = _int("config", data, "vocab")
        eps = _number("norm", data.get("norm") or {}, "eps")
        embedding = data.get("embedding") or {}
        multiplier = 1.0 if embedding.get("scale") is None else _number("embedding", embedding, "scale", positive=False)
        scale = 1.0 if data.get("logit_scale") is None else _number("config", data, "logit_scale", positive=False)
        listed = data.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = entry.get("type") if isinstance(entry, Mapping) else None
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{where}.type {kind!r} is none of {list(MIXER_TYPES)}")
            m = entry.get("mixer")
            if not isinstance(m, Mapping):
                raise ConfigError(f"{where}.mixer must be an object")
            cls._check_attention(where + ".mixer", m)
            mlp = entry.get("mlp")
            if mlp is not None:
                cls._check_mlp(where + ".mlp", mlp)
            layers.append(PekodraLayer(kind, _freeze(m), None if mlp is None else _freeze(mlp)))
        loop = data.get("loop")
        if loop is not None:
            if not isinstance(loop, Mapping):
                raise ConfigError("loop must be an object")
            start, stop = _int("loop", loop, "start", least=0), _int("loop", loop, "stop", least=0)
            times = _int("loop", loop, "times", least=1)
            if not start < stop <= len(layers):
                raise ConfigError(f"loop: start {start} .. stop {stop} is no stretch of {len(layers)} layers")
            loop = (start, stop, times)
        eos = data.get("eos_token_id")
        return cls(width=width, vocab=vocab, norm_eps=eps, embedding_scale=multiplier, logit_scale=scale, layers=tuple(layers),
                   loop=loop, eos_token_id=eos if type(eos) is int else None)

    @staticmethod
    def _check_attention(where: str, m: Mapping[str, Any]) -> None:
        heads, dim = _int(where, m, "heads"), _int(where, m, "dim")
        if heads % _int(where, m, "kv_heads"):
            raise ConfigError(f"{where}: {heads} heads are not a multiple of {m['kv_heads']} kv_heads")
        _int(where, m, "vdim")
        _number(where, m, "scale", positive=False)
        if not isinstance(m.get("mask"), Mapping):
            raise ConfigError(f"{where}.mask must be an object")
        _int(where + ".mask", m["mask"], "size")
        _rot(where, m, dim, blended=True)
        scaling = m["rot"].get("scaling")
        if scaling is not None:
            for key in ("original", "fast", "slow"):
                _number(where + ".rot.scaling", scaling, key)

    @staticmethod
    def _check_mlp(where: str, mlp: Any) -> None:
        kind = mlp.get("kind") if isinstance(mlp, Mapping) else None
        if kind not in MLP_KINDS:
            raise ConfigError(f"{where}.kind {kind!r} is none of {list(MLP_KINDS)}")
        if kind == "dense":
            _int(where, mlp, "ff")
            return
        _int(where + ".expert", mlp.get("expert"), "ff")
        experts = _int(where + ".router", mlp.get("router"), "experts")
        top = _int(where + ".router", mlp.get("router"), "top")
        if top > experts:
            raise ConfigError(f"{where}.router: top {top} exceeds the {experts} experts")
        if mlp.get("shared") is not None:
            _int(where + ".shared", mlp.get("shared"), "ff")

    @classmethod
    def from_json(cls, path) -> "PekodraConfig":
        path = Path(path)
        if path.is_dir():
            path = path / "config.json"
        return cls.from_dict(json.loads(path.read_text()))

    # ------------------------------------------------------------------ writing

    def to_dict(self) -> dict:
        """A config.json that reads back as this configuration."""
        data = dict(
            architecture=ARCHITECTURE,
            embedding=dict(scale=self.embedding_scale),
            layers=[dict(type=l.type, mixer=l.mixer_options, mlp=l.mlp_options) for l in self.layers],
            logit_scale=self.logit_scale,
            norm=dict(eps=self.norm_eps),
            vocab=self.vocab,
            width=self.width,
        )
        if self.loop is not None:
            data["loop"] = dict(start=self.loop[0], stop=self.loop[1], times=self.loop[2])
        if self.eos_token_id is not None:
            data["eos_token_id"] = self.eos_token_id
        return data

    # ------------------------------------------------------------------ the model it describes

    def mixer_spec(self, layer: PekodraLayer):
        m = layer.mixer_options
        rot = m["rot"]
        names = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "out_proj.weight": "o"}
        return AttentionSpec(
            self.width, m["heads"], m["kv_heads"], m["dim"], position=_rope(m["dim"], rot, rot["dims"], blended=True),
            window=m["mask"]["size"], scale=float(m["scale"]), v_head_dim=m["vdim"], qk_unit_eps=self.norm_eps, names=names,
        )

    def ffn_spec(self, layer: PekodraLayer):
        mlp = layer.mlp_options
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return GatedMLPSpec(self.width, mlp["ff"], activation="gelu_tanh", bias=True)
        shared = mlp.get("shared")
        return RoutedExpertsSpec(
            self.width, mlp["expert"]["ff"], mlp["router"]["experts"], 0, mlp["router"]["top"], correction=False,
            shared_size=None if shared is None else shared["ff"], gated=False, activation="relu2",
        )

    def run_order(self) -> Tuple[ScheduleEntry, ...]:
        """One entry per layer run; a layer inside the loop runs ``times`` times, each time with a cache of its own, and
        in front of every pass the embedding's output is joined to the stream."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(ScheduleEntry(i) for i in range(n))
        start, stop, times = self.loop
        order = [ScheduleEntry(i) for i in range(start)]
        for _ in range(times):
            order += [ScheduleEntry(i, join=JOIN if i == start else None) for i in range(start, stop)]
        return tuple(order + [ScheduleEntry(i) for i in range(stop, n)])

    def model_spec(self) -> ModelSpec:
        norm = RMSNormSpec(self.width, self.norm_eps, zero_centered=True)
        layers = []
        for i, layer in enumerate(self.layers):
            prefix = f"l{i}."
            ffn = self.ffn_spec(layer)
            layers.append(LayerSpec(
                mixer=self.mixer_spec(layer),
                ffn=ffn,
                mixer_norm=norm,
                ffn_norm=None if ffn is None else norm,
                mixer_prefix=prefix + "mix.",
                ffn_prefix=prefix + "mlp.",
                mixer_norm_name=prefix + "norm1",
                ffn_norm_name=prefix + "norm2",
                arrangement="parallel",
            ))
        return ModelSpec(
            architecture=ARCHITECTURE,
            hidden_size=self.width,
            vocab_size=self.vocab,
            layers=tuple(layers),
            final_norm=norm,
            embedding_name="embed",
            final_norm_name="final.norm",
            head_name="head",
            schedule=self.run_order(),
            embedding_multiplier=self.embedding_scale,
            logit_scale=self.logit_scale,
        )
