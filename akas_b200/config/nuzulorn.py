"""Typed configuration of the Nuzulorn decoder, read from its own config.json keys.

A Nuzulorn model is a list of layers around a float32 residual stream. A token's embedding is its own row plus a row that
a hash of the token in front of it and of itself picks from a second table (``embedding.bigram``); a sequence's first
token takes that table's last row. A layer adds ``residual_mult`` times its mixer's result and then ``residual_mult``
times its feed-forward's, each read through an RMSNorm; what goes on to the next layer is a learned weighted sum of the
embedding's output and of the results of all layers so far. Mixers: ``attention`` (grouped-query attention inside a
sliding window of ``mask.size`` tokens and, in front of it, over whole blocks of ``mask.pool`` tokens as their mean key
and mean value; rotate-half rotary positions on the first ``rot.dims`` channels, exp(0) in the softmax's denominator, a
sigmoid gate per head, biases on all four projections), ``attention_2`` (causal grouped-query attention without rotation:
queries times 1 + ``q_temp.coef`` ln(floor((p + 1) / ``q_temp.every``) + 1), scores capped by a tanh at ``softcap``, less
2^(-8 (h + 1) / heads) times the distance, exp of a learned logit per head in the denominator, biases on q, k and v) and
``hgrn2`` (a matrix state per head whose forget gate, bounded from below by a tensor, also decides what is written). The
feed-forward is a mixture of SwiGLU experts with sigmoid scores, a correction in the choice, a limit to the best groups
of experts (by the sum of a group's two largest choice scores) and weights that are the scores times ``router.scale``; or
none. The head is the embedding.

Checkpoint names: ``embed``, ``bigram``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.{q,k,v,o}`` (with ``.b`` where biased),
``l<i>.mix.{g,sink}``, ``l<i>.mix.{f,f.b,lower,norm}``, ``l<i>.mlp.{router,correction,e<j>.{gate,up,down}}``, ``l<i>.dwa``,
``final.norm``.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping, Optional, Tuple

from .girelix import _freeze, _int, _number, _thaw
from .kidarax import _rope, _rot
from .lfm2 import ConfigError
from .specs import AttentionSpec, BigramSpec, HGRN2Spec, LayerSpec, ModelSpec, RMSNormSpec, RoutedExpertsSpec, ScheduleEntry

ARCHITECTURE = "Nuzulorn"
MIXER_TYPES = ("attention", "attention_2", "hgrn2")
MLP_KINDS = ("moe",)
GROUP_BEST = 2  # a group of experts is judged by the sum of its two largest choice scores


@dataclass(frozen=True)
class NuzulornLayer:
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
class NuzulornConfig:
    width: int
    vocab: int
    norm_eps: float
    residual_mult: float
    bigram: Tuple[int, int, int]  # (buckets, mul_prev, mul_cur)
    layers: Tuple[NuzulornLayer, ...]
    eos_token_id: Optional[int] = None

    architecture = ARCHITECTURE

    # ------------------------------------------------------------------ reading

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "NuzulornConfig":
        if data.get("architecture") != ARCHITECTURE:
            raise ConfigError(f"architecture {data.get('architecture')!r} is not {ARCHITECTURE!r}")
        width = _int("config", data, "width")
        vocab = _int("config", data, "vocab")
        eps = _number("norm", data.get("norm") or {}, "eps")
        mult = _number("config", data, "residual_mult", positive=False)
        big = (data.get("embedding") or {}).get("bigram")
        if not isinstance(big, Mapping):
            raise ConfigError("embedding.bigram must be an object")
        bigram = (_int("embedding.bigram", big, "buckets"), _int("embedding.bigram", big, "mul_prev", least=0),
                  _int("embedding.bigram", big, "mul_cur", least=0))
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
            getattr(cls, "_check_" + kind)(where + ".mixer", m)
            mlp = entry.get("mlp")
            if mlp is not None:
                cls._check_mlp(where + ".mlp", mlp)
            layers.append(NuzulornLayer(kind, _freeze(m), None if mlp is None else _freeze(mlp)))
        eos = data.get("eos_token_id")
        return cls(width=width, vocab=vocab, norm_eps=eps, residual_mult=mult, bigram=bigram, layers=tuple(layers),
                   eos_token_id=eos if type(eos) is int else None)

    @staticmethod
    def _check_heads(where: str, m: Mapping[str, Any]) -> None:
        if _int(where, m, "heads") % _int(where, m, "kv_heads"):
            raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
        _int(where, m, "dim"), _int(where, m, "vdim")
        _number(where, m, "scale", positive=False)

    @classmethod
    def _check_attention(cls, where: str, m: Mapping[str, Any]) -> None:
        cls._check_heads(where, m)
        if not isinstance(m.get("mask"), Mapping):
            raise ConfigError(f"{where}.mask must be an object")
        _int(where + ".mask", m["mask"], "size"), _int(where + ".mask", m["mask"], "pool")
        _rot(where, m, m["dim"], blended=False)

    @classmethod
    def _check_attention_2(cls, where: str, m: Mapping[str, Any]) -> None:
        cls._check_heads(where, m)
        _number(where, m, "softcap")
        temp = m.get("q_temp")
        if not isinstance(temp, Mapping):
            raise ConfigError(f"{where}.q_temp must be an object")
        _number(where + ".q_temp", temp, "coef", positive=False)
        _int(where + ".q_temp", temp, "every")

    @staticmethod
    def _check_hgrn2(where: str, m: Mapping[str, Any]) -> None:
        for key in ("heads", "dim", "vdim"):
            _int(where, m, key)

    @staticmethod
    def _check_mlp(where: str, mlp: Any) -> None:
        kind = mlp.get("kind") if isinstance(mlp, Mapping) else None
        if kind not in MLP_KINDS:
            raise ConfigError(f"{where}.kind {kind!r} is none of {list(MLP_KINDS)}")
        _int(where + ".expert", mlp.get("expert"), "ff")
        router = mlp.get("router")
        w = where + ".router"
        experts, top = _int(w, router, "experts"), _int(w, router, "top")
        if router.get("scale") is not None:
            _number(w, router, "scale", positive=False)
        groups = router.get("groups")
        count, keep = 1, 1
        if groups is not None:
            count, keep = _int(w + ".groups", groups, "count"), _int(w + ".groups", groups, "keep")
        if experts % count:
            raise ConfigError(f"{w}: {experts} experts do not form {count} equal groups")
        if keep > count:
            raise ConfigError(f"{w}.groups: keep {keep} exceeds count {count}")
        if top > keep * (experts // count):
            raise ConfigError(f"{w}: top {top} exceeds the {keep * (experts // count)} experts of {keep} groups")

    @classmethod
    def from_json(cls, path) -> "NuzulornConfig":
        path = Path(path)
        if path.is_dir():
            path = path / "config.json"
        return cls.from_dict(json.loads(path.read_text()))

    # ------------------------------------------------------------------ writing

    def to_dict(self) -> dict:
        """A config.json that reads back as this configuration."""
        buckets, mul_prev, mul_cur = self.bigram
        data = dict(
            architecture=ARCHITECTURE,
            embedding=dict(bigram=dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)),
            layers=[dict(type=l.type, mixer=l.mixer_options, mlp=l.mlp_options) for l in self.layers],
            norm=dict(eps=self.norm_eps),
            residual_mult=self.residual_mult,
            vocab=self.vocab,
            width=self.width,
        )
        if self.eos_token_id is not None:
            data["eos_token_id"] = self.eos_token_id
        return data

    # ------------------------------------------------------------------ the model it describes

    def mixer_spec(self, layer: NuzulornLayer):
        m = layer.mixer_options
        if layer.type == "hgrn2":
            return HGRN2Spec(self.width, m["heads"], m["dim"], m["vdim"], self.norm_eps)
        names = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "out_proj.weight": "o", "gate.weight": "g"}
        common = dict(scale=float(m["scale"]), v_head_dim=m["vdim"], bias=True, names=names)
        if layer.type == "attention":
            rot = m["rot"]
            return AttentionSpec(self.width, m["heads"], m["kv_heads"], m["dim"], position=_rope(m["dim"], rot, rot["dims"], blended=False),
                                 window=m["mask"]["size"], pool=m["mask"]["pool"], sink=True, gate="head", out_bias=True, **common)
        temp = m["q_temp"]
        return AttentionSpec(self.width, m["heads"], m["kv_heads"], m["dim"], softcap=float(m["softcap"]), distance_bias="linear",
                             sink="learned", q_temperature=(float(temp["coef"]), temp["every"]), **common)

    def ffn_spec(self, layer: NuzulornLayer):
        mlp = layer.mlp_options
        if mlp is None:
            return None
        router = mlp["router"]
        groups = router.get("groups") or dict(count=1, keep=1)
        scale = router.get("scale")
        return RoutedExpertsSpec(
            self.width, mlp["expert"]["ff"], router["experts"], 0, router["top"], groups["count"], groups["keep"], scoring="sigmoid",
            correction=True, renormalize=False, group_best=GROUP_BEST, weight_scale=1.0 if scale is None else float(scale),
        )

    def model_spec(self) -> ModelSpec:
        norm = RMSNormSpec(self.width, self.norm_eps)
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
                residual_multiplier=self.residual_mult,
            ))
        return ModelSpec(
            architecture=ARCHITECTURE,
            hidden_size=self.width,
            vocab_size=self.vocab,
            layers=tuple(layers),
            final_norm=norm,
            embedding_name="embed",
            final_norm_name="final.norm",
            head_name=None,
            schedule=tuple(ScheduleEntry(i, average=f"l{i}.dwa") for i in range(len(self.layers))),
            bigram=BigramSpec("bigram", *self.bigram),
        )
