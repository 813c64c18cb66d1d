"""The Renanex design as data: a decoder with a norm on both sides of every sub-layer, of windowed attention and two recurrences.

Token embedding; a layer is ``x += n1b(mixer(n1(x)))`` and, where it has a feed-forward, ``x += n2b(ff(n2(x)))``: RMS norms whose
weight is a single number; the model's norm of the same kind; logits from an untied head, scaled and soft-capped.  The mixer is

* ``lightning``: linear attention with one fixed decay per head; q, k and v pass silu, nothing is scaled, the concatenated heads are
  RMS-normed together with a weight per value and gated by a sigmoid (``parts/retention.py``);
* ``mamba1``: the selective scan (``parts/selective_scan.py``);
* ``attention``: grouped-query attention with one RMS norm over all of q and one over all of k, a rotation in half-split pairs with
  YaRN-rescaled frequencies, scores mixed over the heads before the softmax, a sliding window that keeps the first tokens, and
  values blended with those of the first such layer (``parts/attention.py``).

The feed-forward is SwiGLU.  Tensor names: ``embed``, ``l<i>.norm1`` / ``.norm1b`` / ``.norm2`` / ``.norm2b``, ``l<i>.mix.*``,
``l<i>.mlp.gate`` / ``.up`` / ``.down``, ``final.norm``, ``head``.

Constants the design fixes (not in config.json): silu on q, k and v of the linear attention and its sigmoid gate, the pairing of
rotated values, silu as the feed-forward's activation, YaRN's magnitude ``0.1 ln(factor) + 1`` (in the rotation part).
"""
from __future__ import annotations

from ..config.renanex_config import RenanexConfig
from ..parts.base import PartSpec, LayerSpec, RunEntry, ModelSpec
from ..registry import register_model

ROTARY_STYLE = "half"
LIGHTNING_ACT, LIGHTNING_GATE = "silu", "sigmoid"


def _norm(prefix: str, name: str, d: int, eps: float) -> PartSpec:
    return PartSpec("rmsnorm", prefix, {"dim": d, "eps": eps, "name": name, "scalar": True})


def _position(m: dict) -> PartSpec:
    rot = m.get("rot")
    if rot is None or not rot["dims"]:
        return PartSpec("none", "", {})
    sc = rot.get("scaling")
    scaling = None if sc is None else {"kind": "yarn", "factor": sc["factor"], "original": sc["original"],
                                       "fast": sc["fast"], "slow": sc["slow"]}
    return PartSpec("rope", "", {"dim": rot["dims"], "base": rot["base"], "style": ROTARY_STYLE, "scaling": scaling})


def _mixer(L: dict, p: str, d: int, eps: float, v_mix: str = None) -> PartSpec:
    """``v_mix``: "first" or "mix" for an attention layer whose values are mixed, None otherwise."""
    m = L["mixer"]
    if L["type"] == "lightning":
        return PartSpec("retention", f"{p}.mix", {
            "d_model": d, "num_heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "decay": tuple(m["decay"]), "eps": eps,
            "qkv_act": LIGHTNING_ACT, "key_scale": 1.0, "norm_over": "all", "norm_weight": "norm", "gate_act": LIGHTNING_GATE})
    if L["type"] == "mamba1":
        return PartSpec("selective_scan", f"{p}.mix", {"d_model": d, "inner": m["inner"], "state": m["state"], "dt_rank": m["dt_rank"],
                                                       "taps": m["conv"]})
    mask = m.get("mask")
    return PartSpec("attention", f"{p}.mix", {
        "d_model": d, "num_heads": m["heads"], "num_kv_heads": m.get("kv_heads", m["heads"]), "head_dim": m["dim"],
        "v_head_dim": m.get("vdim", m["dim"]), "position": _position(m), "window": None if mask is None else mask["size"],
        "keep_first": 0 if mask is None else mask.get("keep_first", 0), "scale": m["scale"], "qk_norm": eps, "qk_norm_over": "projection",
        "head_mix": "talk", "v_mix": v_mix, "v_mix_name": "vmix",
        "names": {"q": "q", "k": "k", "v": "v", "o": "o"}, "weight_suffix": "", "norm_suffix": ".norm"})


@register_model("Renanex")
def renanex(config: RenanexConfig) -> ModelSpec:
    d, eps = config.width, config.norm_eps
    layers, run_order, first_values = [], [], True
    for i, L in enumerate(config.layers):
        p, f, v_mix = f"l{i}", L.get("mlp"), None
        if L["type"] == "attention" and L["mixer"].get("v_mix"):
            v_mix, first_values = ("first" if first_values else "mix"), False
        args = {"mixer_norm": _norm(p, "norm1", d, eps), "mixer": _mixer(L, p, d, eps, v_mix), "mixer_out_norm": _norm(p, "norm1b", d, eps)}
        if f is not None:
            args.update({"ffn_norm": _norm(p, "norm2", d, eps), "ffn": PartSpec("glu", f"{p}.mlp", {"d_model": d, "hidden": f["ff"]}),
                         "ffn_out_norm": _norm(p, "norm2b", d, eps)})
        layers.append(LayerSpec(PartSpec("sandwich_norm", p, args)))
        run_order.append(RunEntry(i))
    return ModelSpec(
        d_model=d, vocab_size=config.vocab, max_seq_len=config.max_seq_len,
        embedding=PartSpec("token", "", {"vocab_size": config.vocab, "dim": d, "name": "embed"}),
        layers=tuple(layers), run_order=tuple(run_order),
        final_norm=_norm("final", "norm", d, eps),
        head=PartSpec("linear", "", {"dim": d, "vocab_size": config.vocab, "name": "head", "softcap": config.logit_softcap,
                                     "scale": config.logit_scale}),
        eos_token_id=config.eos_token_id,
    )
