"""The Fokurax configuration, its model as data, what its layers ask of the cache manager, and pages that layers of several chunk
sizes read (no GPU)."""
import copy

import pytest
import torch

import plain_fokurax as pf
from fokurax_configs import ALL, FOK_A, FOK_B, FOK_C, FOK_D, attn, dense, layer, model, moe

from tiny_transformer_inference_engine_b200 import ModelConfig
from tiny_transformer_inference_engine_b200.cache import CacheManager
from tiny_transformer_inference_engine_b200.config import ConfigError
from tiny_transformer_inference_engine_b200.config.fokurax_config import FokuraxConfig
from tiny_transformer_inference_engine_b200.models.model import Model
from tiny_transformer_inference_engine_b200.parts.base import PagedKVNeed, PartSpec
from tiny_transformer_inference_engine_b200.registry import model_spec, build_part
from tiny_transformer_inference_engine_b200.weights import random_tensors, write_random_model, read_safetensors


def test_architecture_picks_the_config_class_and_round_trips(tmp_path):
    cfg = ModelConfig.from_dict(FOK_A)
    assert isinstance(cfg, FokuraxConfig)
    assert (cfg.vocab_size, cfg.d_model, cfg.norm_eps, cfg.embedding_scale, cfg.residual_mult, cfg.logit_softcap, cfg.side_dim) == \
        (131, 64, 1e-5, 4.0, 0.6, 12.0, 10)
    write_random_model(cfg, 3, str(tmp_path))
    again = ModelConfig.from_json(str(tmp_path))
    assert again == cfg and again.to_dict() == cfg.to_dict()
    stored = read_safetensors(str(tmp_path))
    assert set(stored) == set(Model(model_spec(cfg)).param_specs())
    assert stored["l2.mlp.table"].dtype == torch.int32 and (stored["l2.mlp.table"] < 7).all() and (stored["l2.mlp.table"] >= 0).all()
    assert all(len(set(row)) == 3 for row in stored["l2.mlp.table"].tolist())                     # the experts of a token differ
    assert ModelConfig.from_dict(FOK_B).logit_softcap is None and ModelConfig.from_dict(FOK_D).side_dim is None
    for name, c in ALL.items():
        assert ModelConfig.from_dict(ModelConfig.from_dict(c).to_dict()) == ModelConfig.from_dict(c), name
    without = {k: v for k, v in FOK_D.items() if k != "token_side"}
    assert ModelConfig.from_dict(without) == ModelConfig.from_dict(FOK_D)


def test_tensor_names_and_shapes():
    specs = {k: tuple(v[2].shape) for k, v in Model(model_spec(ModelConfig.from_dict(FOK_A))).param_specs().items()}
    assert specs["embed"] == (131, 64) and specs["head"] == (131, 64) and specs["final.norm"] == (64,) and specs["side.embed"] == (131, 50)
    for i in range(5):
        assert specs[f"l{i}.norm1"] == (64,) and f"l{i}.norm2" not in specs
        assert specs[f"l{i}.side.gate"] == (10, 64) and specs[f"l{i}.side.proj"] == (64, 10) and specs[f"l{i}.side.norm"] == (64,)
    assert specs["l0.mix.q"] == (64, 64) and specs["l0.mix.k"] == (32, 64) and specs["l0.mix.v"] == (48, 64) and specs["l0.mix.o"] == (64, 96)
    assert specs["l1.mix.q"] == (72, 64) and specs["l1.mix.k"] == (24, 64) and specs["l1.mix.v"] == (12, 64)
    for i in (2, 3, 4):                                                     # queries of their own, another layer's keys and values
        assert f"l{i}.mix.q" in specs and f"l{i}.mix.o" in specs and f"l{i}.mix.k" not in specs and f"l{i}.mix.v" not in specs
    assert specs["l0.mlp.gate"] == (80, 64) and specs["l0.mlp.gate.b"] == specs["l0.mlp.up.b"] == (80,) and specs["l0.mlp.down.b"] == (64,)
    assert specs["l2.mlp.table"] == (131, 3) and specs["l2.mlp.e6.gate"] == (36, 64) and specs["l2.mlp.e6.down"] == (64, 36)
    assert "l2.mlp.e7.gate" not in specs and "l2.mlp.router" not in specs and "l2.mlp.e0.gate.b" not in specs
    assert not any(k.startswith("l3.mlp") for k in specs)                   # no feed-forward
    none = set(Model(model_spec(ModelConfig.from_dict(FOK_D))).param_specs())
    assert not any("side" in k for k in none)


def test_cache_needs_follow_the_readers_of_a_cache():
    model = Model(model_spec(ModelConfig.from_dict(FOK_A)))
    needs = model.cache_needs()
    assert needs[0] == [PagedKVNeed(2, 32, chunk=13, also_chunks=(21,))]     # keys of 16 and values of 24 in rows of 32
    assert needs[1] == [PagedKVNeed(1, 32, chunk=29)] and needs[2] == needs[3] == needs[4] == []
    assert [e.cache_from for e in model.run_order] == [None, None, 0, 0, 1]
    d = Model(model_spec(ModelConfig.from_dict(FOK_D))).cache_needs()
    assert d[0] == [PagedKVNeed(4, 32)] and d[2] == [PagedKVNeed(1, 16)]     # whoever reads without chunks keeps every page


def test_pages_stay_while_any_reader_needs_them():
    """Chunks of 6 and of 10 positions on one cache, pages of two: a page leaves when both have passed it."""
    cfg = model(32, 16, 1e-5, 1.0, 1.0, None, 4, [layer(attn(1, 1, 8, 8, 1.0, chunk=6)), layer(attn(1, 1, 8, 8, 1.0, chunk=10, kv_from=0))])
    m = Model(model_spec(ModelConfig.from_dict(cfg)))
    mgr = CacheManager(m.cache_needs(), m.run_order, 2, 24, 2, "float32", "cpu", max_step_tokens=4)
    assert len(mgr.groups) == 1 and mgr.groups[0].reach == 10
    mgr.admit("r")
    for pos in range(45):
        mgr.extend("r", pos, pos + 1)
        first = min(pos - pos % 6, pos - pos % 10) // 2
        table = mgr.table(0, "r")
        assert [p != 0 for p in table] == [i >= first for i in range(len(table))], pos
    mgr.check()
    views = mgr.views({0: torch.zeros((1, 1), dtype=torch.int32)})
    assert views[1][0].k_pages.data_ptr() == views[0][0].k_pages.data_ptr() and views[0][0].writable and not views[1][0].writable
    mgr.release("r")
    mgr.check()
    assert mgr.num_free_pages == mgr.num_usable_pages


@pytest.mark.parametrize("edit,text", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(kv_from=0), "earlier"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "no keys and values"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=0), "differ"),
    (lambda c: c["layers"][0]["mlp"].update(kind="mlp"), "unknown"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c["token_side"].update(dim=0), "token_side"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.pop("embedding"), "embedding"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "at least one"),
])
def test_bad_configs_are_refused(edit, text):
    cfg = copy.deepcopy(FOK_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        ModelConfig.from_dict(cfg)


def test_a_table_that_names_a_missing_expert_is_refused():
    part = build_part("ffn", PartSpec("grouped_moe", "f", {"d_model": 8, "hidden": 4, "experts": 3, "top": 2, "table": 5}))
    w = {k: torch.zeros(ps.shape, dtype=torch.int32 if ps.storage == "table" else torch.float32) for k, ps in part.param_specs().items()}
    part.load(w)
    w["table"][4, 1] = 3
    with pytest.raises(ValueError, match="experts 0 .. 3"):
        part.load(w)
    with pytest.raises(ValueError, match="router"):
        build_part("ffn", PartSpec("grouped_moe", "f", {"d_model": 8, "hidden": 4, "experts": 3, "top": 2, "table": 5, "identity": 1}))


def test_norm_weights_are_stored_around_zero():
    norm = build_part("norm", PartSpec("rmsnorm", "n", {"dim": 4, "eps": 1e-5, "name": "w", "zero_centered": True}))
    norm.load({"w": torch.tensor([0.0, 0.5, -1.0, 2.0], dtype=torch.bfloat16)})
    assert norm.weight.tolist() == [1.0, 1.5, 0.0, 3.0] and norm.weight.dtype == torch.float32
    gained = build_part("norm", PartSpec("rmsnorm", "n", {"dim": 2, "eps": 1e-5, "name": "w", "gain": 0.5}))
    gained.load({"w": torch.tensor([1.0, 3.0])})
    assert gained.weight.tolist() == [0.5, 1.5] == gained.weight32.tolist()


def test_plain_implementation_sees_every_mechanism():
    """Leaving any one mechanism out of the plain model moves its logits: the tests that compare with it would notice."""
    cfg = copy.deepcopy(FOK_A)
    w = random_tensors(ModelConfig.from_dict(cfg), 4, std=0.2)
    w["embed"] = w["embed"] * 4
    toks = torch.randint(0, 131, (40,), generator=torch.Generator().manual_seed(1)).tolist()
    base = pf.forward(cfg, w, toks)

    def moved(edit_cfg=None, edit_w=None):
        c, ww = copy.deepcopy(cfg), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(ww)
        return ((pf.forward(c, ww, toks) - base).abs().max() / base.abs().max()).item()

    edits = {"chunk": lambda c: c["layers"][2]["mixer"]["mask"].update(size=22), "scale": lambda c: c["layers"][3]["mixer"].update(scale=0.5),
             "yarn": lambda c: c["layers"][1]["mixer"]["rot"].pop("scaling"), "rotated values": lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6),
             "multiplier": lambda c: c.update(residual_mult=0.65), "embedding": lambda c: c["embedding"].update(scale=3.0),
             "soft cap": lambda c: c.update(logit_softcap=None), "side": lambda c: c.update(token_side=None), "eps": lambda c: c["norm"].update(eps=0.05)}
    for name, e in edits.items():
        assert moved(edit_cfg=e) > 1e-3, name
    for key in ("l0.mlp.gate.b", "l0.mlp.up.b", "l0.mlp.down.b", "l4.side.norm", "l3.norm1", "final.norm"):
        assert moved(edit_w=lambda ww: ww.update({key: torch.zeros_like(ww[key])})) > 1e-3, key
    assert moved(edit_w=lambda ww: ww.update({"l2.mlp.table": (ww["l2.mlp.table"] + 1) % 7})) > 1e-3
    assert moved(edit_w=lambda ww: ww.update({"side.embed": ww["side.embed"].roll(10, dims=1)})) > 1e-3
