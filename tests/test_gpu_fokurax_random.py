"""Fokurax configurations drawn at random (layer order, sizes, head counts, chunks, shared caches, rotated values, rescaled frequencies,
experts, side values and constants) through the engine in four cuts and both dtypes, against the plain implementation."""
import random

import pytest

import trace_util as tu
from fokurax_configs import attn, dense, layer, model, moe, yarn
from test_gpu_fokurax import weights_for, engine_for, requests, expected_for, check

pytestmark = pytest.mark.gpu


def draw(seed):
    r = random.Random(seed)
    width = r.choice([24, 40, 50, 56, 64, 72, 96, 128])
    layers, owners = [], []
    for i in range(r.randint(2, 7)):
        chunk = None if r.random() < 0.1 else r.choice([1, 2, 5, 8, 13, 16, 24, 33, 64, 300])
        if owners and r.random() < 0.45:
            j = r.choice(owners)
            mixer = dict(layers[j]["mixer"], kv_from=j, scale=layers[j]["mixer"]["scale"] * r.choice([1.0, 0.5, 1.5]))
            if r.random() < 0.5:                                               # chunks of its own
                mixer.pop("mask", None)
                if chunk is not None:
                    mixer["mask"] = {"size": chunk}
        else:
            kv, dim = r.choice([1, 2, 3, 4]), r.choice([4, 10, 16, 24, 32, 48, 64, 80, 128])
            scaling = None if r.random() < 0.3 else yarn(r.choice([2.0, 4.0, 8.0]), r.choice([16, 64, 256]), r.choice([4.0, 16.0, 32.0]), r.choice([0.5, 1.0, 2.0]))
            mixer = attn(kv * r.choice([1, 2, 4]), kv, dim, r.choice([dim, 4, 8, 20, 64, 128]), r.choice([1.0, 2.0, 4.0]) * dim ** -0.5, chunk=chunk,
                         rot=r.choice([0, 2, 4, dim]), base=r.choice([20.0, 1e3, 1e4, 3e5]), scaling=scaling)
            owners.append(i)
        experts = r.choice([1, 2, 5, 12, 30])
        mlp = r.choice([None, dense(r.choice([16, 30, 96])), moe(r.choice([8, 20, 64]), experts, r.randint(1, min(experts, 6))),
                        moe(r.choice([8, 20, 64]), experts, r.randint(1, min(experts, 6)))])
        layers.append(layer(mixer, mlp))
    return model(r.choice([50, 97, 128, 300]), width, r.choice([1e-6, 1e-5, 1e-3]), r.choice([1.0, 4.0, 16.0]), r.choice([0.3, 0.7, 1.0]),
                 r.choice([None, 5.0, 20.0]), r.choice([1, 6, 16, 24, 30]), layers)


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
        check(tu.run_steps(eng, steps), exp, dtype)
