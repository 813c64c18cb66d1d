"""The Fokurax design as data: a decoder of parallel layers over chunked attention, with an input to every layer from the token's id.

Token embedding times ``embedding.scale``; a layer is ``x += m (attention(h) + ff(h))`` with ``h`` the normed stream, then
``x += m n(proj(gelu_tanh(gate x) * e))`` with ``e`` the layer's own part of the token's row in a second table and ``n`` an RMS norm;
``m`` is ``residual_mult``.  The model's norms store their weights around zero; ``n`` has a plain weight.  Logits from an untied
head, soft-capped.

* ``attention``: grouped-query attention, a rotation of the first ``rot.dims`` values of every head in half-split pairs with
  YaRN-rescaled frequencies, every rotated query and key head over its root mean square (no weight), a chunked mask.  A layer with
  ``kv_from`` has queries only and reads the cache of the layer named there, with its own mask and scale
  (``parts/attention.py``).
* feed-forward: a gelu-gated unit with biases (``parts/ffn.py``), or SwiGLU experts that a table names for every token id, all
  of one weight (``parts/moe.py``).

Tensor names: ``embed``, ``side.embed``, ``l<i>.norm1``, ``l<i>.mix.q`` / ``.k`` / ``.v`` / ``.o``, ``l<i>.mlp.gate`` / ``.up`` / ``.down`` (each
with ``.b``) or ``l<i>.mlp.table``, ``.e<j>.gate`` / ``.up`` / ``.down``, ``l<i>.side.gate`` / ``.proj`` / ``.norm``, ``final.norm``, ``head``.

Constants the design fixes (not in config.json): the activations, the pairing of rotated values, equal weights of the chosen
experts, YaRN's magnitude ``0.1 ln(factor) + 1`` (in the rotation part).
"""
from __future__ import annotations

from ..config.fokurax_config import FokuraxConfig
from ..parts.base import PartSpec, LayerSpec, RunEntry, ModelSpec
from ..registry import register_model

ROTARY_STYLE = "half"
DENSE_ACT = "gelu_tanh"


def _norm(prefix: str, name: str, d: int, eps: float) -> PartSpec:
    return PartSpec("rmsnorm", prefix, {"dim": d, "eps": eps, "name": name, "zero_centered": True})


def _position(m: dict) -> PartSpec:
    rot = m.get("rot")
    if rot is None or not rot["dims"]:
        return PartSpec("none", "", {})
    sc = rot.get("scaling")
    scaling = None if sc is None else {"kind": "yarn", "factor": sc["factor"], "original": sc["original"],
                                       "fast": sc["fast"], "slow": sc["slow"]}
    return PartSpec("rope", "", {"dim": rot["dims"], "base": rot["base"], "style": ROTARY_STYLE, "scaling": scaling})


def _chunk(m: dict):
    mask = m.get("mask")
    return None if mask is None else mask["size"]


def _mixer(m: dict, p: str, d: int, eps: float, readers=()) -> PartSpec:
    """``readers``: the mixers of the layers that read this layer's keys and values."""
    return PartSpec("attention", f"{p}.mix", {
        "d_model": d, "num_heads": m["heads"], "num_kv_heads": m.get("kv_heads", m["heads"]), "head_dim": m["dim"],
        "v_head_dim": m.get("vdim", m["dim"]), "position": _position(m), "chunk": _chunk(m), "scale": m["scale"], "norm_after": eps,
        "shares_kv": m.get("kv_from") is not None, "cache_chunks": tuple(_chunk(r) for r in readers),
        "names": {"q": "q", "k": "k", "v": "v", "o": "o"}, "weight_suffix": ""})


def _ffn(f, p: str, d: int, vocab: int):
    if f is None:
        return None
    if f["kind"] == "dense":
        return PartSpec("glu", f"{p}.mlp", {"d_model": d, "hidden": f["ff"], "act": DENSE_ACT, "bias": True, "bias_suffix": ".b", "defer_bias": True})
    return PartSpec("grouped_moe", f"{p}.mlp", {"d_model": d, "hidden": f["expert"]["ff"], "experts": f["router"]["experts"],
                                                "top": f["router"]["top"], "table": vocab, "defer_combine": True})


@register_model("Fokurax")
def fokurax(config: FokuraxConfig) -> ModelSpec:
    d, eps, side = config.width, config.norm_eps, config.side_dim
    layers, run_order = [], []
    for i, L in enumerate(config.layers):
        p, m = f"l{i}", L["mixer"]
        readers = [r["mixer"] for r in config.layers if r["mixer"].get("kv_from") == i]
        args = {"norm": _norm(p, "norm1", d, eps), "mixer": _mixer(m, p, d, eps, readers), "ffn": _ffn(L.get("mlp"), p, d, config.vocab),
                "mult": config.residual_mult}
        if side is not None:
            args["side"] = PartSpec("token_gated", f"{p}.side", {"d_model": d, "dim": side, "column": i * side})
            args["side_norm"] = PartSpec("rmsnorm", f"{p}.side", {"dim": d, "eps": eps, "name": "norm", "gain": config.residual_mult})
        layers.append(LayerSpec(PartSpec("parallel", p, args)))
        run_order.append(RunEntry(i, m.get("kv_from")))
    table = None if side is None else {"name": "side.embed", "dim": side, "layers": len(config.layers)}
    return ModelSpec(
        d_model=d, vocab_size=config.vocab, max_seq_len=config.max_seq_len,
        embedding=PartSpec("token", "", {"vocab_size": config.vocab, "dim": d, "name": "embed", "scale": config.embedding_scale, "side": table}),
        layers=tuple(layers), run_order=tuple(run_order),
        final_norm=_norm("final", "norm", d, eps),
        head=PartSpec("linear", "", {"dim": d, "vocab_size": config.vocab, "name": "head", "softcap": config.logit_softcap}),
        eos_token_id=config.eos_token_id,
    )
