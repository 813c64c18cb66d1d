"""The Renanex configuration, its model as data, what its layers ask of the cache manager, and pages that a window keeps (no GPU)."""
import copy
import random

import pytest
import torch

import plain_renanex as pr
from renanex_configs import ALL, REN_A, REN_B, REN_D, yarn

from tiny_transformer_inference_engine_b200 import ModelConfig
from tiny_transformer_inference_engine_b200.cache import CacheManager, OutOfPages
from tiny_transformer_inference_engine_b200.config import ConfigError
from tiny_transformer_inference_engine_b200.config.renanex_config import RenanexConfig
from tiny_transformer_inference_engine_b200.engine.batch import BatchPacker, StepEntry
from tiny_transformer_inference_engine_b200.models.model import Model
from tiny_transformer_inference_engine_b200.ops import CudaOps
from tiny_transformer_inference_engine_b200.parts.base import PagedKVNeed, FixedStateNeed, PartSpec, RunEntry
from tiny_transformer_inference_engine_b200.registry import model_spec, build_part
from tiny_transformer_inference_engine_b200.weights import write_random_model, read_safetensors


def test_architecture_picks_the_config_class_and_round_trips(tmp_path):
    cfg = ModelConfig.from_dict(REN_A)
    assert isinstance(cfg, RenanexConfig)
    assert (cfg.vocab_size, cfg.d_model, cfg.norm_eps, cfg.logit_scale, cfg.logit_softcap) == (131, 64, 1e-5, 1.5, 12.0)
    write_random_model(cfg, 3, str(tmp_path))
    again = ModelConfig.from_json(str(tmp_path))
    assert again == cfg and again.to_dict() == cfg.to_dict()
    assert set(read_safetensors(str(tmp_path))) == set(Model(model_spec(cfg)).param_specs())
    assert ModelConfig.from_dict(REN_B).logit_softcap is None and "logit_softcap" not in ModelConfig.from_dict(REN_B).to_dict()
    for name, c in ALL.items():
        assert ModelConfig.from_dict(ModelConfig.from_dict(c).to_dict()) == ModelConfig.from_dict(c), name


def test_tensor_names_and_shapes():
    specs = {k: tuple(v[2].shape) for k, v in Model(model_spec(ModelConfig.from_dict(REN_A))).param_specs().items()}
    assert specs["embed"] == (131, 64) and specs["head"] == (131, 64) and specs["final.norm"] == ()
    for i in range(5):
        assert specs[f"l{i}.norm1"] == () and specs[f"l{i}.norm1b"] == ()
    assert specs["l0.norm2"] == specs["l0.norm2b"] == () and specs["l0.mlp.gate"] == (80, 64) and specs["l0.mlp.down"] == (64, 80)
    assert not any(k.startswith(("l2.norm2", "l2.mlp")) for k in specs)                                  # no feed-forward
    assert specs["l0.mix.q"] == (64, 64) and specs["l0.mix.k"] == (32, 64) and specs["l0.mix.v"] == (48, 64) and specs["l0.mix.o"] == (64, 96)
    assert specs["l0.mix.q.norm"] == (64,) and specs["l0.mix.k.norm"] == (32,) and specs["l0.mix.talk"] == (4, 4)
    assert specs["l0.mix.vmix"] == specs["l4.mix.vmix"] == () and "l3.mix.vmix" not in specs
    assert specs["l1.mix.in"] == (144, 64) and specs["l1.mix.conv"] == (72, 4) and specs["l1.mix.conv.b"] == (72,)
    assert specs["l1.mix.x"] == (25, 72) and specs["l1.mix.dt"] == (72, 5) and specs["l1.mix.dt.b"] == (72,)
    assert specs["l1.mix.A_log"] == (72, 10) and specs["l1.mix.D"] == (72,) and specs["l1.mix.o"] == (64, 72)
    assert specs["l2.mix.q"] == (36, 64) and specs["l2.mix.v"] == (60, 64) and specs["l2.mix.g"] == (60, 64) and specs["l2.mix.norm"] == (60,)


def test_which_values_are_mixed_with_which():
    def kinds(cfg):
        return [layer.block.args["mixer"].args.get("v_mix") for layer in model_spec(ModelConfig.from_dict(cfg)).layers]

    assert kinds(REN_A) == ["first", None, None, None, "mix"]
    assert kinds(REN_B) == [None, "first", None, None, None, "mix", None]
    one = copy.deepcopy(REN_A)
    one["layers"][0]["mixer"]["v_mix"] = False
    assert kinds(one) == [None, None, None, None, "first"]


def test_cache_needs():
    needs = Model(model_spec(ModelConfig.from_dict(REN_A))).cache_needs()
    assert needs[0] == [PagedKVNeed(1, 48, 13, keep_first=3)]                     # two kv heads' values of 24 side by side
    assert needs[1] == [FixedStateNeed((72, 16), "float32"), FixedStateNeed((3, 72), "float32")]
    assert needs[2] == [FixedStateNeed((3, 20, 16), "float32")]
    assert needs[3] == [PagedKVNeed(1, 24, 29, keep_first=6)] and needs[4] == [PagedKVNeed(1, 48, 8, keep_first=1)]
    b = Model(model_spec(ModelConfig.from_dict(REN_B))).cache_needs()
    assert b[2] == [FixedStateNeed((54, 4), "float32")] and len(b[4]) == 2         # one tap keeps no rows
    d = Model(model_spec(ModelConfig.from_dict(REN_D))).cache_needs()
    assert d[0] == [PagedKVNeed(1, 320)]                                           # no mask: every page stays


def test_joint_rows_are_padded_to_what_the_kernels_take():
    width = lambda dtype, *a: CudaOps.joint_width(None, dtype, *a)
    bf = torch.bfloat16
    assert [width(bf, *a) for a in ((2, 24, 8), (2, 10, 12), (1, 128, 64), (2, 65, 8), (3, 80, 90), (8, 64, 64), (3, 87, 1), (4, 100, 128), (5, 100, 100))] == \
        [48, 32, 128, 256, 272, 512, 264, 512, 504]
    assert width(torch.float32, 3, 7, 5) == 24 and width(torch.float32, 1, 6, 30) == 32


def test_planned_keys_of_windows():
    vis = CudaOps.visible_keys
    assert vis(1, 5000, 0, 0, 0) == 5000
    assert vis(1, 5000, 1024, 0, 4) == 128 + 1024 + 1 + 127 and vis(1, 700, 1024, 0, 4) == 700
    assert vis(300, 5000, 1024, 0, 0) == 1024 + 300 + 127 and vis(1, 5000, 0, 256, 0) == 256 + 1 + 127
    # never fewer than a tile of rows walks: kept tiles, the window, the rows' own span and the rounding of its first key
    rng = random.Random(1)
    for _ in range(500):
        window, keep, n, L = rng.choice([1, 5, 100, 1000]), rng.choice([0, 1, 130, 300]), rng.choice([1, 2, 70, 500]), rng.randint(500, 4000)
        for tile in (32, 64, 128):
            first = max(0, L - n - window + 1) // tile * tile
            kept = min(-(-keep // tile) * tile, first)
            assert kept + L - first <= vis(n, L, window, 0, keep)


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="wkv"), "unknown"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0), "scale"),
    (lambda c: c["layers"][4]["mixer"].update(vdim=8), "value channels"),
    (lambda c: c["layers"][1]["mixer"].pop("dt_rank"), "dt_rank"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5]), "one number per head"),
    (lambda c: c["layers"][2]["mixer"].update(decay=[0.5, 0.5, 1.5]), "not in"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "at least one")])
def test_bad_configurations_are_refused(edit, message):
    cfg = copy.deepcopy(REN_A)
    edit(cfg)
    with pytest.raises(ConfigError, match=message):
        ModelConfig.from_dict(cfg)


def test_parts_refuse_what_they_do_not_compute():
    args = dict(d_model=32, num_heads=4, num_kv_heads=2, head_dim=8, position=PartSpec("none", "", {}), head_mix="talk")
    for more in (dict(conv_taps=3), dict(gated="value"), dict(qk_norm=1e-5), dict(softcap=5.0), dict(weights="sigmoid"), dict(keep_first=4)):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("attention", "a", dict(args, **more)))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("selective_scan", "a", dict(d_model=8, inner=8, state=129, dt_rank=1, taps=2)))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("retention", "a", dict(d_model=8, num_heads=1, dim=4, vdim=4, decay=[0.5], eps=1e-5, qkv_act="silu")))


def test_plain_masks_and_frequencies():
    """The oracle itself: rows of the mask by hand, and rescaled frequencies at both ends of the ramp."""
    m = pr.visible(9, {"size": 3, "keep_first": 2})
    assert m[8].nonzero().flatten().tolist() == [0, 1, 6, 7, 8] and m[1].nonzero().flatten().tolist() == [0, 1]
    assert pr.visible(5, None).sum() == 15
    f, mag = pr.frequencies({"base": 100.0, "dims": 16, "scaling": yarn(4.0, 64, 8.0, 1.0)})
    assert f[0] == 1.0 and abs(f[-1] - 100.0 ** (-14 / 16) / 4.0) < 1e-12 and abs(mag - (0.1 * 1.3862943611198906 + 1)) < 1e-12


# ------------------------------------------------------------------------------------------ pages of first tokens that a window keeps
def test_kept_pages_stay_and_the_rest_come_back():
    m = CacheManager([PagedKVNeed(1, 8, window=6, keep_first=5)], [RunEntry(0)], 4, 9, 3, "float32", "cpu")
    m.admit("a")
    m.extend("a", 0, 10)
    assert m.table(0, "a") == [1, 2, 3]
    m.extend("a", 10, 18)                                          # keys from 5 on: page 1 would go, but holds kept token 4
    assert m.table(0, "a") == [1, 2, 3, 4, 5]
    m.extend("a", 18, 19)                                          # keys from 13 on: page 2 goes
    assert m.table(0, "a") == [1, 2, 0, 4, 5]
    m.extend("a", 30, 31)                                          # keys from 25 on
    assert m.table(0, "a")[:2] == [1, 2] and m.table(0, "a")[2:6] == [0, 0, 0, 0] and 0 not in m.table(0, "a")[6:]
    m.check()
    m.release("a")
    assert m.num_free_pages == m.num_usable_pages
    g = m.groups[0]
    assert g.kept_pages == 2 and g.needed_pages(30, 8) == [0, 1, 6, 7] and g.needed_pages(0, 3) == [0, 1, 2]
    assert g.pages_of_request(1000, 1) == 2 + 2 + 1


def test_random_requests_with_kept_pages_lose_none():
    rng = random.Random(5)
    for keep, window, page in ((1, 3, 2), (7, 5, 4), (20, 9, 8), (0, 4, 4)):
        need = PagedKVNeed(1, 4, window=window, keep_first=keep)
        m = CacheManager([need], [RunEntry(0)], page, 30, 4, "float32", "cpu", max_step_tokens=8)
        g, live = m.groups[0], {}
        for step in range(400):
            rid = rng.choice("abcd")
            if rid not in live:
                m.admit(rid)
                live[rid] = 0
            n = rng.randint(1, 8)
            try:
                m.extend(rid, live[rid], live[rid] + n)
            except OutOfPages:
                m.release(rid)
                live.pop(rid)
                continue
            for pos in range(live[rid], live[rid] + n):            # every key a new token may see has a page
                for key in list(range(min(keep, pos + 1))) + list(range(max(0, pos - window + 1), pos + 1)):
                    assert m.table(0, rid)[key // page] > 0
            live[rid] += n
            held = sum(p != 0 for p in m.table(0, rid))
            assert held <= g.pages_of_request(live[rid], 8)
            m.check()
            if live[rid] > 90:
                m.release(rid)
                live.pop(rid)


def test_packer_accepts_kept_pages_and_refuses_a_lost_one():
    m = CacheManager([PagedKVNeed(1, 4, window=5, keep_first=3)], [RunEntry(0)], 4, 20, 2, "float32", "cpu")
    m.admit("a")
    m.extend("a", 0, 30)
    m.extend("a", 30, 31)
    packer = BatchPacker(m, None, torch.float32, "cpu", 50, 100)
    packer.validate([StepEntry("a", 30, [1], [0])])
    m.table(0, "a")[0] = 0
    with pytest.raises(ValueError, match="does not cover"):
        packer.validate([StepEntry("a", 30, [1], [0])])
