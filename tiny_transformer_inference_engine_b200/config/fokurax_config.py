"""Configuration of the Fokurax design: a decoder whose attention and feed-forward read the same normed rows, and to whose layers every
token's id adds an input of its own; the layers are listed one by one.

config.json keys: ``architecture`` ("Fokurax"), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``residual_mult``,
``logit_softcap`` (optional or null: none), ``token_side.dim`` (optional or null: no such input) and ``layers``, a list with one entry
per layer: ``type`` (``attention``), ``mixer`` (its sizes and constants; ``kv_from``: the layer whose keys and values it reads) and
``mlp`` (``kind`` ``dense`` with ``ff``, or ``moe`` with ``expert.ff``, ``router.experts`` and ``router.top``; null or absent: no
feed-forward).  Every size and every constant that can differ between models is read from there; nothing has a default in code,
except what an absent option means: no mask, no rotation, no rescaled frequencies, one kv head per head, values of the keys' size.
The design names no longest sequence; ``max_seq_len`` is this engine's own bound on positions (an optional key, else
``DEFAULT_MAX_SEQ_LEN``).
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .model_config import ConfigError, register_config
from .munevik_config import _need, _pos_int, DEFAULT_MAX_SEQ_LEN
from .mizupel_config import _pos_num
from .dabilorn_config import _check_rot

MIXERS = ("attention",)
MLPS = ("dense", "moe")


def _number(v, where: str):
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"{where} must be a number, got {v!r}")


def _kv_sizes(m: dict):
    return m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])


def _check_attention(m: dict, where: str):
    _need(m, ("heads", "dim", "scale"), where)                          # (kv_heads absent: one per head; vdim absent: dim)
    for k in ("heads", "kv_heads", "dim", "vdim"):
        if k in m:
            _pos_int(m[k], f"{where}.{k}")
    if m["heads"] % m.get("kv_heads", m["heads"]):
        raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
    _number(m["scale"], f"{where}.scale")
    if m.get("mask") is not None:
        _need(m["mask"], ("size",), f"{where}.mask")
        _pos_int(m["mask"]["size"], f"{where}.mask.size")
    _check_rot(m, where, m["dim"], scaling=True)


def _check_mlp(f: dict, where: str):
    _need(f, ("kind",), where)
    if f["kind"] == "dense":
        _need(f, ("ff",), where)
        _pos_int(f["ff"], f"{where}.ff")
    elif f["kind"] == "moe":
        _need(f, ("expert", "router"), where)
        _need(f["expert"], ("ff",), f"{where}.expert")
        _pos_int(f["expert"]["ff"], f"{where}.expert.ff")
        _need(f["router"], ("experts", "top"), f"{where}.router")
        for k in ("experts", "top"):
            _pos_int(f["router"][k], f"{where}.router.{k}")
        if f["router"]["top"] > f["router"]["experts"]:
            raise ConfigError(f"{where}.router: top={f['router']['top']} of {f['router']['experts']} experts")
    else:
        raise ConfigError(f"{where}.kind {f['kind']!r} unknown; known: {MLPS}")


@register_config("Fokurax")
@dataclass(frozen=True)
class FokuraxConfig:
    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    logit_softcap: Optional[float] = None
    side_dim: Optional[int] = None
    max_seq_len: int = DEFAULT_MAX_SEQ_LEN
    eos_token_id: Optional[int] = None
    architecture: str = "Fokurax"
    extra: Dict[str, Any] = field(default_factory=dict, compare=False)

    def __post_init__(self):
        _pos_int(self.vocab, "vocab"); _pos_int(self.width, "width"); _pos_int(self.max_seq_len, "max_seq_len")
        _number(self.embedding_scale, "embedding.scale"); _number(self.residual_mult, "residual_mult")
        if self.logit_softcap is not None:
            _pos_num(self.logit_softcap, "logit_softcap")
        if self.side_dim is not None:
            _pos_int(self.side_dim, "token_side.dim")
        if not self.layers:
            raise ConfigError("'layers' must list at least one layer")
        for i, L in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(L, ("type", "mixer"), where)
            if L["type"] not in MIXERS:
                raise ConfigError(f"{where}.type {L['type']!r} unknown; known: {MIXERS}")
            m = L["mixer"]
            _check_attention(m, f"{where}.mixer")
            j = m.get("kv_from")
            if j is not None:
                if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < i:
                    raise ConfigError(f"{where}.mixer.kv_from={j!r} must name an earlier layer")
                other = self.layers[j]["mixer"]
                if other.get("kv_from") is not None:
                    raise ConfigError(f"{where}.mixer.kv_from={j}: that layer has no keys and values of its own")
                if _kv_sizes(other)[1:] != _kv_sizes(m)[1:]:
                    raise ConfigError(f"{where}.mixer.kv_from={j}: kv heads and head sizes {_kv_sizes(m)[1:]} differ from that layer's {_kv_sizes(other)[1:]}")
            if L.get("mlp") is not None:
                _check_mlp(L["mlp"], f"{where}.mlp")

    # the names the engine asks every configuration for
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def d_model(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "FokuraxConfig":
        raw = dict(raw)
        _need(raw, ("vocab", "width", "layers", "norm", "embedding", "residual_mult"), "config.json")
        _need(raw["norm"], ("eps",), "config.json 'norm'")
        _need(raw["embedding"], ("scale",), "config.json 'embedding'")
        raw.pop("architecture", None)
        side = raw.pop("token_side", None)
        if side is not None:
            _need(side, ("dim",), "config.json 'token_side'")
        kw = dict(vocab=raw.pop("vocab"), width=raw.pop("width"), layers=tuple(raw.pop("layers")), norm_eps=float(raw.pop("norm")["eps"]),
                  embedding_scale=raw.pop("embedding")["scale"], residual_mult=raw.pop("residual_mult"),
                  logit_softcap=raw.pop("logit_softcap", None), side_dim=None if side is None else side["dim"])
        if "max_seq_len" in raw:
            kw["max_seq_len"] = raw.pop("max_seq_len")
        if "eos_token_id" in raw:
            kw["eos_token_id"] = raw.pop("eos_token_id")
        return cls(extra=raw, **kw)

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "layers": list(self.layers),
             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult,
             "logit_softcap": self.logit_softcap, "token_side": None if self.side_dim is None else {"dim": self.side_dim}}
        if self.max_seq_len != DEFAULT_MAX_SEQ_LEN:
            d["max_seq_len"] = self.max_seq_len
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        d.update({k: v for k, v in self.extra.items() if k not in d})
        return d

    def save(self, folder: str) -> str:
        os.makedirs(folder, exist_ok=True)
        path = os.path.join(folder, "config.json")
        with open(path, "w", encoding="utf-8") as f:
            json.dump(self.to_dict(), f, indent=2, sort_keys=True)
        return path
