"""Typed configuration of the Mevulix decoder, read from its config.json.

The file names its architecture with one string, ``"architecture": "Mevulix"``, and gives the model's sizes
(``vocab``, ``width``), the norms' eps (``norm.eps``), the factor on the logits (``logit_scale``) and a list ``layers``
whose entries say which mixer the layer has (``type``: attention | latent_attention), the mixer's sizes and constants
(``mixer``) and the feed-forward (``mlp``: ``kind`` dense | moe, or null for none; a mixture's shared expert,
``shared``, may be absent).  An attention layer with ``kv_from`` reads the keys and values of that earlier attention
layer.  Every size and constant is taken from there; nothing is assumed equal between layers.  How many distance buckets
a layer's bias has, the checkpoint says; ``bias_rows`` (optional) says it too, which random weights need.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .errors import ConfigError
from .puzorax import _check_latent, _int, _num, _obj

MIXER_TYPES = ("attention", "latent_attention")
MLP_KINDS = ("dense", "moe")


def _check_attention(where: str, m: dict) -> None:
    for k in ("heads", "kv_heads", "dim", "vdim"):
        _int(where, m, k)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
    _num(where, m, "scale")
    _num(where, m, "softcap", positive=True)
    _num(where, m, "bias_max", positive=True)
    q = _obj(where, m, "q_temp")
    _num(where + ".q_temp", q, "coef")
    _num(where + ".q_temp", q, "every", positive=True)
    for k, low in (("kv_from", 0), ("bias_rows", 2)):
        if m.get(k) is not None:
            _int(where, m, k, low)


def _check_latent_mixer(where: str, m: dict) -> None:
    _check_latent(where, m)
    _int(where, m, "q_rank")
    if not m["rot_dim"]:
        return
    rot = _obj(where, m, "rot")
    if rot.get("dims") != m["rot_dim"]:
        raise ConfigError(f"{where}.rot: 'dims' must be the rotated size 'rot_dim' ({m['rot_dim']}), got {rot.get('dims')!r}")
    if rot.get("scaling") is not None:
        s = _obj(where + ".rot", rot, "scaling")
        for k in ("factor", "original", "fast", "slow"):
            _num(where + ".rot.scaling", s, k, positive=True)


def _check_mlp(where: str, mlp: dict) -> None:
    kind = mlp.get("kind")
    if kind not in MLP_KINDS:
        raise ConfigError(f"{where}: 'kind' must be one of {', '.join(MLP_KINDS)}, got {kind!r}")
    if kind == "dense":
        _int(where, mlp, "ff")
        return
    _int(where + ".expert", _obj(where, mlp, "expert"), "ff")
    if mlp.get("shared") is not None:
        _int(where + ".shared", _obj(where, mlp, "shared"), "ff")
    r = _obj(where, mlp, "router")
    E, top = _int(where + ".router", r, "experts"), _int(where + ".router", r, "top")
    if top > E:
        raise ConfigError(f"{where}.router: {top} of {E} experts cannot be chosen")


@dataclass
class MevulixLayer:
    type: str
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]

    @property
    def kv_from(self) -> Optional[int]:
        return self.mixer.get("kv_from")


@dataclass
class MevulixConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: List[MevulixLayer] = field(default_factory=list)
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict) -> "MevulixConfig":
        vocab, width = _int("config", d, "vocab"), _int("config", d, "width")
        eps = _num("config key 'norm'", _obj("config", d, "norm"), "eps")
        logit_scale = _num("config", d, "logit_scale")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config key 'layers' must be a non-empty list")
        layers: List[MevulixLayer] = []
        for i, e in enumerate(raw):
            where = f"config layers[{i}]"
            if not isinstance(e, dict) or e.get("type") not in MIXER_TYPES:
                raise ConfigError(f"{where}: 'type' must be one of {', '.join(MIXER_TYPES)}, got "
                                  f"{e.get('type') if isinstance(e, dict) else e!r}")
            m = dict(_obj(where, e, "mixer"))
            (_check_attention if e["type"] == "attention" else _check_latent_mixer)(where + ".mixer", m)
            src = m.get("kv_from") if e["type"] == "attention" else None
            if src is not None:
                if src >= i or layers[src].type != "attention" or layers[src].kv_from is not None:
                    raise ConfigError(f"{where}.mixer: 'kv_from' must name an earlier attention layer with keys and values of "
                                      f"its own, got {src}")
                for k in ("heads", "kv_heads", "dim", "vdim"):
                    if layers[src].mixer[k] != m[k]:
                        raise ConfigError(f"{where}.mixer: {k!r} is {m[k]}, but layer {src}, whose keys and values it reads, "
                                          f"has {layers[src].mixer[k]}")
            mlp = e.get("mlp")
            if mlp is not None:
                mlp = dict(_obj(where, e, "mlp"))
                _check_mlp(where + ".mlp", mlp)
            layers.append(MevulixLayer(e["type"], m, mlp))
        eos = d.get("eos_token_id")
        return cls(vocab, width, eps, logit_scale, layers, None if eos is None else int(eos))

    def to_dict(self) -> dict:
        return {"vocab": self.vocab, "width": self.width, "norm_eps": self.norm_eps, "logit_scale": self.logit_scale,
                "layers": [f"{l.type} {l.mixer}" + (f" + mlp {l.mlp}" if l.mlp else "") for l in self.layers]}
