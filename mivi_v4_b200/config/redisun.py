"""Typed configuration of the Redisun decoder, read from its config.json.

The file names its architecture with one string, ``"architecture": "Redisun"``, and gives the model's sizes
(``vocab``, ``width``), the norm's eps (``norm.eps``), the weight of what the stream held in every residual sum
(``postln_alpha``), the hashed bigram table of the embedding (``embedding.bigram``: ``buckets``, ``mul_prev``,
``mul_cur``) and a list ``layers`` whose entries say which mixer the layer has (``type``: latent_attention), the
mixer's sizes and constants (``mixer``) and the feed-forward (``mlp``: ``kind`` dense | moe, or null for none; a
mixture's shared expert, ``shared``, may be absent).  Every size and constant is taken from there; nothing is assumed
equal between layers.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .errors import ConfigError
from .puzorax import _check_latent, _int, _num, _obj

MIXER_TYPES = ("latent_attention",)
MLP_KINDS = ("dense", "moe")


def _check_mixer(where: str, m: dict) -> None:
    _check_latent(where, m)
    _int(where, m, "q_rank")
    if m["rot_dim"] % 2:
        raise ConfigError(f"{where}: key 'rot_dim' must be even, got {m['rot_dim']!r}")
    if m["rot_dim"] and (m.get("rot") or {}).get("dims") != m["rot_dim"]:
        raise ConfigError(f"{where}.rot: 'dims' must be the rotated size 'rot_dim' ({m['rot_dim']}), got {m.get('rot')!r}")


def _check_mlp(where: str, mlp: dict) -> None:
    kind = mlp.get("kind")
    if kind not in MLP_KINDS:
        raise ConfigError(f"{where}: 'kind' must be one of {', '.join(MLP_KINDS)}, got {kind!r}")
    if kind == "dense":
        _int(where, mlp, "ff")
        return
    for name in ("expert", "shared"):
        if name == "shared" and mlp.get("shared") is None:
            continue
        d = _obj(where, mlp, name)
        _int(f"{where}.{name}", d, "ff")
        _num(f"{where}.{name}", d, "limit", positive=True)
    r = _obj(where, mlp, "router")
    E, top = _int(where + ".router", r, "experts"), _int(where + ".router", r, "top")
    if top > E:
        raise ConfigError(f"{where}.router: {top} of {E} experts cannot be chosen")


@dataclass
class RedisunLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclass
class RedisunConfig:
    vocab: int
    width: int
    norm_eps: float
    alpha: float
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: List[RedisunLayer] = field(default_factory=list)
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict) -> "RedisunConfig":
        vocab, width = _int("config", d, "vocab"), _int("config", d, "width")
        eps = _num("config key 'norm'", _obj("config", d, "norm"), "eps")
        alpha = _num("config", d, "postln_alpha")
        bg = _obj("config key 'embedding'", _obj("config", d, "embedding"), "bigram")
        buckets = _int("config embedding.bigram", bg, "buckets")
        mul_prev, mul_cur = _int("config embedding.bigram", bg, "mul_prev", 0), _int("config embedding.bigram", bg, "mul_cur", 0)
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config key 'layers' must be a non-empty list")
        layers = []
        for i, e in enumerate(raw):
            where = f"config layers[{i}]"
            if not isinstance(e, dict) or e.get("type") not in MIXER_TYPES:
                raise ConfigError(f"{where}: 'type' must be one of {', '.join(MIXER_TYPES)}, got "
                                  f"{e.get('type') if isinstance(e, dict) else e!r}")
            m = dict(_obj(where, e, "mixer"))
            _check_mixer(where + ".mixer", m)
            mlp = e.get("mlp")
            if mlp is not None:
                mlp = dict(_obj(where, e, "mlp"))
                _check_mlp(where + ".mlp", mlp)
            layers.append(RedisunLayer(e["type"], m, mlp))
        eos = d.get("eos_token_id")
        return cls(vocab, width, eps, alpha, buckets, mul_prev, mul_cur, layers, None if eos is None else int(eos))

    def to_dict(self) -> dict:
        return {"vocab": self.vocab, "width": self.width, "norm_eps": self.norm_eps, "postln_alpha": self.alpha,
                "bigram": {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur},
                "layers": [f"{l.type} {l.mixer}" + (f" + mlp {l.mlp}" if l.mlp else "") for l in self.layers]}
