"""Configuration of the Renanex design: a decoder with norms on both sides of every sub-layer that mixes windowed attention with
two kinds of recurrence; its layers are listed one by one.

config.json keys: ``architecture`` ("Renanex"), ``vocab``, ``width``, ``norm.eps``, ``logit_scale``, ``logit_softcap`` and
``layers``, a list with one entry per layer: ``type`` (the mixer: ``lightning``, ``mamba1`` or ``attention``), ``mixer`` (its sizes
and constants) and ``mlp`` (``kind`` ``dense`` with ``ff``; null or absent: no feed-forward).  Every size and every constant that
can differ between models is read from there; nothing has a default in code, except what an absent option means: no mask, no
rotation, no rescaled frequencies, no kept first tokens, no mixed values, no cap.  The design names no longest sequence;
``max_seq_len`` is this engine's own bound on positions (an optional key, else ``DEFAULT_MAX_SEQ_LEN``).
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

MIXERS = ("lightning", "mamba1", "attention")
MLPS = ("dense",)


def _check_lightning(m: dict, where: str):
    _need(m, ("heads", "dim", "vdim", "decay"), where)
    for k in ("heads", "dim", "vdim"):
        _pos_int(m[k], f"{where}.{k}")
    if not isinstance(m["decay"], (list, tuple)) or len(m["decay"]) != m["heads"]:
        raise ConfigError(f"{where}.decay must list one number per head ({m['heads']})")
    for x in m["decay"]:
        if isinstance(x, bool) or not isinstance(x, (int, float)) or not 0.0 <= x <= 1.0:
            raise ConfigError(f"{where}.decay: {x!r} is not in [0, 1]")


def _check_attention(m: dict, where: str):
    _need(m, ("heads", "dim", "scale"), where)                          # (kv_heads absent: one per head; vdim absent: dim)
    for k in ("heads", "kv_heads", "dim", "vdim"):
        if k in m:
            _pos_int(m[k], f"{where}.{k}")
    if m["heads"] % m.get("kv_heads", m["heads"]):
        raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
    _pos_num(m["scale"], f"{where}.scale")
    mask = m.get("mask")
    if mask is not None:
        _need(mask, ("size",), f"{where}.mask")
        _pos_int(mask["size"], f"{where}.mask.size")
        keep = mask.get("keep_first", 0)
        if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
            raise ConfigError(f"{where}.mask.keep_first={keep!r} must be an integer of 0 or more")
    if not isinstance(m.get("v_mix", False), bool):
        raise ConfigError(f"{where}.v_mix={m['v_mix']!r} must be true or false")
    _check_rot(m, where, m["dim"], scaling=True)


@register_config("Renanex")
@dataclass(frozen=True)
class RenanexConfig:
    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm_eps: float
    logit_scale: float
    logit_softcap: Optional[float] = None
    max_seq_len: int = DEFAULT_MAX_SEQ_LEN
    eos_token_id: Optional[int] = None
    architecture: str = "Renanex"
    extra: Dict[str, Any] = field(default_factory=dict, compare=False)

    def __post_init__(self):
        _pos_int(self.vocab, "vocab"); _pos_int(self.width, "width"); _pos_int(self.max_seq_len, "max_seq_len")
        if isinstance(self.logit_scale, bool) or not isinstance(self.logit_scale, (int, float)):
            raise ConfigError(f"logit_scale must be a number, got {self.logit_scale!r}")
        if self.logit_softcap is not None:
            _pos_num(self.logit_softcap, "logit_softcap")
        if not self.layers:
            raise ConfigError("'layers' must list at least one layer")
        values = None                                                   # value channels of the layers whose values are mixed
        for i, L in enumerate(self.layers):
            where = f"layers[{i}]"
            _need(L, ("type", "mixer"), where)
            m, mw = L["mixer"], f"{where}.mixer"
            if L["type"] == "lightning":
                _check_lightning(m, mw)
            elif L["type"] == "mamba1":
                _need(m, ("inner", "state", "dt_rank", "conv"), mw)
                for k in ("inner", "state", "dt_rank", "conv"):
                    _pos_int(m[k], f"{mw}.{k}")
            elif L["type"] == "attention":
                _check_attention(m, mw)
                if m.get("v_mix"):
                    n = m.get("kv_heads", m["heads"]) * m.get("vdim", m["dim"])
                    if values is not None and n != values:
                        raise ConfigError(f"{mw}: {n} value channels cannot be mixed with the {values} of the first layer with v_mix")
                    values = n
            else:
                raise ConfigError(f"{where}.type {L['type']!r} unknown; known: {MIXERS}")
            f = L.get("mlp")
            if f is not None:
                _need(f, ("kind",), f"{where}.mlp")
                if f["kind"] != "dense":
                    raise ConfigError(f"{where}.mlp.kind {f['kind']!r} unknown; known: {MLPS}")
                _need(f, ("ff",), f"{where}.mlp")
                _pos_int(f["ff"], f"{where}.mlp.ff")

    # the names the engine asks every configuration for
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def d_model(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "RenanexConfig":
        raw = dict(raw)
        _need(raw, ("vocab", "width", "layers", "norm", "logit_scale"), "config.json")
        _need(raw["norm"], ("eps",), "config.json 'norm'")
        raw.pop("architecture", None)
        kw = dict(vocab=raw.pop("vocab"), width=raw.pop("width"), layers=tuple(raw.pop("layers")), norm_eps=float(raw.pop("norm")["eps"]),
                  logit_scale=raw.pop("logit_scale"), logit_softcap=raw.pop("logit_softcap", None))
        if "max_seq_len" in raw:
            kw["max_seq_len"] = raw.pop("max_seq_len")
        if "eos_token_id" in raw:
            kw["eos_token_id"] = raw.pop("eos_token_id")
        return cls(extra=raw, **kw)

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "layers": list(self.layers),
             "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
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
