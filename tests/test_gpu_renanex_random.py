"""Renanex configurations drawn at random (layer order, sizes, head counts, windows, kept tokens, rotated values, rescaled frequencies,
states, taps, decays and constants) through the engine in four cuts and both dtypes, against the plain implementation."""
import random

import pytest

import trace_util as tu
from renanex_configs import attn, lightning, mamba, layer, model, yarn
from test_gpu_renanex import weights_for, engine_for, requests, expected_for, check

pytestmark = pytest.mark.gpu


def draw(seed):
    r = random.Random(seed)
    width = r.choice([24, 40, 50, 56, 64, 72, 96, 128])
    values = r.choice([(1, 16), (2, 12), (2, 32), (4, 16), (3, 20)])              # kv heads and value size of the layers whose values are mixed
    layers = []
    for _ in range(r.randint(2, 7)):
        kind = r.choice(["attention", "attention", "lightning", "mamba1"])
        if kind == "lightning":
            heads = r.choice([1, 2, 3, 4])
            mixer = lightning(heads, r.choice([4, 8, 12, 32, 64, 72]), r.choice([4, 8, 20, 32, 64]), [r.choice([0.2, 0.6, 0.9, 0.99, 0.999]) for _ in range(heads)])
        elif kind == "mamba1":
            mixer = mamba(r.choice([16, 40, 72, 96, 256]), r.choice([1, 4, 6, 16, 24, 33, 64]), r.choice([1, 3, 8, 12]), r.choice([1, 2, 3, 4, 6]))
        else:
            v_mix = r.random() < 0.6
            kv, vdim = values if v_mix else (r.choice([1, 2, 3, 4]), r.choice([4, 8, 16, 20, 32, 64]))
            dim = r.choice([4, 10, 16, 24, 32, 48, 64])
            window = None if r.random() < 0.15 else r.choice([1, 2, 5, 8, 13, 16, 24, 33, 64, 300])
            rot = r.choice([0, 2, 4, dim])
            scaling = None if r.random() < 0.4 else yarn(r.choice([2.0, 4.0, 8.0]), r.choice([16, 64, 256]), r.choice([4.0, 16.0, 32.0]), r.choice([0.5, 1.0, 2.0]))
            mixer = attn(kv * r.choice([1, 2, 4]), kv, dim, vdim, r.choice([1.0, 0.5, 1.5]) * dim ** -0.5, window=window, keep=r.choice([None, 0, 1, 4, 18]),
                         rot=rot, base=r.choice([20.0, 1e3, 1e4, 3e5]), scaling=scaling, v_mix=v_mix)
        layers.append(layer(kind, mixer, r.choice([None, 16, 40, 96])))
    return model(r.choice([50, 97, 128, 300]), width, r.choice([1e-6, 1e-5, 1e-3]), r.choice([0.5, 1.0, 2.0]), r.choice([None, 5.0, 20.0]), layers)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(1, 13))
def test_random_configuration(seed, dtype):
    cfg = draw(seed)
    w = weights_for(cfg, 100 + seed)
    reqs = requests(cfg, [1, 2, 45, 130, 19, 77], seed=seed)
    exp = expected_for(cfg, w, reqs, dtype)
    page = random.Random(seed).choice([2, 4, 8, 16])
    for cut in (tu.whole, tu.prefill_then_decode, tu.portions, tu.mixed):
        steps = cut(reqs)
        tokens = tu.max_live_tokens(steps, rounding=page)
        eng = engine_for(cfg, w, dtype, page=page, pages=tokens // page + 2)
        check(tu.run_steps(eng, steps), exp, dtype, tail16=0.4, worst32=1e-3)
