"""The Renanex design in the engine against the plain implementation (plain_renanex.py): each mechanism alone, whole prompts,
decoding through the cache and the state slots, portions down to two tokens, mixed batches with pages and slots used again,
keys at the edges of windows and pages, the first tokens and keys far back, other sizes, and greedy generation through the
scheduler."""
import json
import os
import subprocess
import sys

import pytest
import torch

import plain_renanex as pr
import trace_util as tu

from tiny_transformer_inference_engine_b200 import Engine, ModelConfig, EngineConfig, CacheConfig, SchedulerConfig, SamplingParams
from tiny_transformer_inference_engine_b200.parts.base import PartSpec, ResidualStream, StepContext, PagedKVView, FixedStateView
from tiny_transformer_inference_engine_b200.registry import build_part
from tiny_transformer_inference_engine_b200.weights import random_tensors
from tiny_transformer_inference_engine_b200.models.renanex import _mixer                     # config.json's layer entry -> the part

from renanex_configs import ALL as CONFIGS, REN_A, REN_B, REN_C, REN_D, REN_E, attn, lightning, mamba, layer, model, yarn

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def ops():
    from tiny_transformer_inference_engine_b200.ops import get_ops
    return get_ops(DEV)


def shaped(k, t, g):
    """Random tensors of a size at which every mechanism shows: norm gains away from 1 and from each other, a mixing matrix with
    weights of both signs beside its diagonal, blended values in between, states that live from two to hundreds of tokens."""
    if k.endswith((".norm1", ".norm2", ".norm1b", ".norm2b", "q.norm", "k.norm", "mix.norm", "final.norm")) or k == "norm":
        return 1.0 + torch.randn(t.shape, generator=g) * 0.3
    if k.endswith("talk"):
        return torch.eye(t.shape[0]) + torch.randn(t.shape, generator=g) * 0.4
    if k.endswith("vmix"):
        return torch.full(t.shape, 0.35)
    if k.endswith("A_log"):
        return torch.log(torch.arange(1, t.shape[1] + 1).float())[None].expand(t.shape) + torch.randn(t.shape, generator=g) * 0.3
    if k.endswith("dt.b"):
        return torch.randn(t.shape, generator=g) * 1.5 - 2.0
    if k.endswith("mix.D") or k == "D":
        return torch.randn(t.shape, generator=g)
    return None


def weights_for(cfg, seed, store="float32"):
    w = random_tensors(ModelConfig.from_dict(cfg), seed, std=0.15, store_dtype=store)
    g = torch.Generator().manual_seed(seed + 1)
    for k in sorted(w):
        t = shaped(k, w[k], g)
        if t is not None:
            w[k] = t.to(w[k].dtype).contiguous()
        elif k == "embed":
            w[k] = w[k] * 6.0
    return w


def engine_for(cfg, w, dtype, page=16, pages=64, max_seqs=4, budget=64, graphs=False):
    ec = EngineConfig(dtype=dtype, device=DEV, use_cuda_graphs=graphs,
                      cache=CacheConfig(block_size=page, num_gpu_blocks=pages),
                      sched=SchedulerConfig(max_num_seqs=max_seqs, max_num_batched_tokens=budget))
    return Engine(ModelConfig.from_dict(cfg), w, ec)


def requests(cfg, lens, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lens)}


def expected_for(cfg, w, reqs, dtype):
    vec = ("norm", "talk", "vmix", "A_log", ".b", ".D", "conv", "norm1", "norm2", "norm1b", "norm2b")    # kept in 32-bit
    ww = {k: (v.to(torch.bfloat16).double() if dtype == "bfloat16" and not k.endswith(vec) else v) for k, v in w.items()}
    return {rid: pr.forward(cfg, ww, toks) for rid, toks in reqs.items()}


def check(got, exp, dtype, tail16=0.2, typical16=6e-2, worst32=2e-4):
    """32-bit: every place within 2e-4 of the row's largest logit and the typical one within 2e-5.  bfloat16: these models are
    narrow and their sharp attention magnifies rounding at single tokens, so the run is held to the typical error and to nine
    rows in ten (every mechanism alone is held to its largest error in both dtypes below)."""
    errs = []
    for (rid, pos), row in got.items():
        ref = exp[rid][pos]
        errs.append((((row.double() - ref).abs().max() / ref.abs().max()).item(), rid, pos))
    errs.sort(reverse=True)
    n = len(errs)
    assert all(e[0] == e[0] for e in errs), "a NaN among the logits"
    if dtype == "float32":
        assert errs[0][0] < worst32 and errs[n // 2][0] < 2e-5, (errs[:3], errs[n // 2])
    else:
        assert errs[n // 2][0] < typical16 and errs[n // 10][0] < tail16, (errs[n // 2], errs[n // 10], errs[:3])


# ------------------------------------------------------------------------------------------ the whole model, four cuts
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
def test_schedules_against_plain_model(name, dtype):
    cfg = CONFIGS[name]
    w = weights_for(cfg, 5 + ord(name))
    reqs = requests(cfg, [1, 2, 37, 70, 101, 23], seed=3)
    exp = expected_for(cfg, w, reqs, dtype)
    page = {"A": 16, "B": 8, "C": 4, "D": 2, "E": 16}[name]
    for cut in (tu.whole, tu.prefill_then_decode, tu.portions, tu.mixed):
        steps = cut(reqs)
        tokens = tu.max_live_tokens(steps, rounding=page)
        eng = engine_for(cfg, w, dtype, page=page, pages=tokens // page + 2)        # no slack: pages and slots are used again
        check(tu.run_steps(eng, steps), exp, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wider_model_with_long_prompts_on_pages_of_16(dtype):
    """Joint rows of 128 and 256 values on pages of 16 keys (the tcgen05 kernels' sizes), prompts of several hundred tokens, windows
    that no page edge meets: whole (the scans walk long prompts in parts), with a decoded tail, and mixed on a pool without slack."""
    cfg = model(200, 224, 1e-5, 1.0, 15.0, [
        layer("attention", attn(8, 2, 64, 64, 0.12, window=150, keep=6, rot=64, base=5e4, v_mix=True), 128),
        layer("mamba1", mamba(384, 16, 12, 4), 128),
        layer("lightning", lightning(3, 64, 64, [0.9, 0.99, 0.999]), 128),
        layer("attention", attn(4, 2, 128, 64, 0.08, window=90, keep=130, rot=128, base=5e4, scaling=yarn(4.0, 256, 16.0, 1.0), v_mix=True), 128)])
    w = weights_for(cfg, 61)
    reqs = requests(cfg, [700, 333, 41, 290], seed=6)
    exp = expected_for(cfg, w, reqs, dtype)
    for cut in (tu.whole, tu.prefill_then_decode, tu.mixed):
        steps = cut(reqs)
        tokens = tu.max_live_tokens(steps, rounding=16)
        eng = engine_for(cfg, w, dtype, page=16, pages=tokens // 16 + 2, budget=1024)
        check(tu.run_steps(eng, steps), exp, dtype)


def test_long_decode_past_windows_and_pages():
    """A short prompt, then 150 tokens one by one: windows of 8, 13 and 29 keys pass over decoded tokens while the first tokens stay,
    pages are given back under way, and the states and the convolution's rows are carried 150 times."""
    w = weights_for(REN_A, 77)
    reqs = requests(REN_A, [160], seed=9)
    exp = expected_for(REN_A, w, reqs, "float32")
    eng = engine_for(REN_A, w, "float32", page=8, pages=9, budget=16)
    check(tu.run_steps(eng, tu.prefill_then_decode(reqs, tail=150)), exp, "float32")


def test_batch_of_unequal_requests_equals_each_alone():
    w = weights_for(REN_A, 21)
    reqs = requests(REN_A, [3, 50, 1, 29], seed=4)
    eng = engine_for(REN_A, w, "float32", pages=40)
    alone = tu.run_steps(eng, tu.whole(reqs))
    together = tu.run_steps(eng, [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()],
                                   "end": list(reqs)}])
    for key, row in alone.items():
        assert (row - together[key]).abs().max() <= 4e-5 * row.abs().max(), key


def test_slots_and_pages_used_again_carry_nothing_over():
    """Two state slots and pages for one long request: the same request replayed after others have used (and dirtied) its slot
    and pages gives the same logits to the bit."""
    w = weights_for(REN_A, 23)
    reqs = requests(REN_A, [40, 33, 40], seed=8)
    reqs["r2"] = list(reqs["r0"])
    eng = engine_for(REN_A, w, "float32", page=8, pages=8, max_seqs=2)
    got = tu.run_steps(eng, tu.portions(reqs))
    for pos in range(40):
        assert torch.equal(got[("r0", pos)], got[("r2", pos)]), pos
    check(got, expected_for(REN_A, w, reqs, "float32"), "float32")


def test_first_tokens_of_a_sequence():
    """Requests of one and two tokens, alone and beside a longer one, and the first positions of a prompt asked for one by one:
    position 0 sees itself only, the convolution finds zeros before it, the states start at zero."""
    for cfg, page in ((REN_B, 2), (REN_C, 4)):
        w = weights_for(cfg, 41)
        reqs = requests(cfg, [1, 2, 3, 30], seed=5)
        exp = expected_for(cfg, w, reqs, "float32")
        eng = engine_for(cfg, w, "float32", page=page, pages=40)
        check(tu.run_steps(eng, tu.whole(reqs)), exp, "float32")
        check(tu.run_steps(eng, tu.prefill_then_decode(reqs, tail=29)), exp, "float32")
        steps = [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()], "end": list(reqs)}]
        check(tu.run_steps(eng, steps), exp, "float32")


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler(graphs):
    cfg = dict(REN_A, max_seq_len=256)
    w = weights_for(cfg, 31)
    prompts = [[5, 9, 2], list(range(10, 41)), [7]]
    want = []
    for p in prompts:
        toks = list(p)
        for _ in range(18):                                           # past a window's edge for every prompt
            toks.append(int(torch.argmax(pr.forward(cfg, w, toks)[-1])))
        want.append(toks[len(p):])
    eng = engine_for(cfg, w, "float32", pages=40, max_seqs=4, budget=16, graphs=graphs)
    got = eng.generate(prompts, SamplingParams(max_new_tokens=18, greedy=True))
    assert got == want


def test_captured_steps_equal_eager_ones_in_bfloat16():
    """Decode steps replayed from graphs (planned for the longest context of their bucket) and eager ones: the same tokens of a
    batch that joins and leaves."""
    cfg = dict(REN_C, max_seq_len=600)
    w = weights_for(cfg, 37)
    prompts = [list(range(3, 90)), [5, 1], list(range(100, 40, -1))]
    outs = []
    for graphs in (False, True):
        eng = engine_for(cfg, w, "bfloat16", pages=80, budget=64, graphs=graphs)
        outs.append(eng.generate(prompts, SamplingParams(max_new_tokens=40, greedy=True)))
    same = sum(a == b for x, y in zip(*outs) for a, b in zip(x, y))
    assert same >= 0.9 * 120, same                                    # (another cut of the key range may flip a near-tie)


def test_command_line_and_trace_runner_with_a_model_folder(tmp_path):
    """A folder written in the random-weights mode (bfloat16 on disk), generated from by the command line and replayed by the
    trace runner: the architecture is picked from config.json by both."""
    import numpy as np
    from safetensors.torch import load_file
    from tiny_transformer_inference_engine_b200 import write_random_model
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = dict(REN_E, max_seq_len=96)
    folder = write_random_model(ModelConfig.from_dict(cfg), 13, str(tmp_path / "model"), std=0.3, perturb_norms=True, store_dtype="bfloat16")
    w = load_file(os.path.join(folder, "model.safetensors"))
    prompt = [4, 60, 7, 7, 23]
    run = subprocess.run([sys.executable, "-m", "tiny_transformer_inference_engine_b200", "--model", folder, "--tokens", "6", "--greedy",
                          "--dtype", "float32", "--num-gpu-blocks", "16", "--prompt-ids", ",".join(map(str, prompt))],
                         cwd=root, capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    toks = list(prompt)
    for _ in range(6):
        toks.append(int(torch.argmax(pr.forward(cfg, w, toks)[-1])))
    assert json.loads(run.stdout.strip().split("\n")[-1])["generated_ids"] == toks[len(prompt):]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:7], "want": [0, 6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[7:9], "want": [1]}, {"id": "b", "tokens": toks[:3], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[3:4], "want": [0]}], "end": ["b"]}]
    out = tmp_path / "out"
    run = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", cwd=root, capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    exp = pr.forward(cfg, w, toks)
    for name, rows in (("0.f32", [0, 6]), ("1.f32", [8]), ("2.f32", [3])):
        got = torch.from_numpy(np.fromfile(str(out / name), dtype="<f4").reshape(len(rows), cfg["vocab"]))
        assert ((got.double() - exp[rows]).abs().max() / exp[rows].abs().max()).item() < 1e-4, name




# ------------------------------------------------------------------------------------------ each mechanism alone
def ctx_for(ops, dtype, seqs, tables=None, slots=None):
    pos = [s + i for s, n in seqs for i in range(n)]
    tseq = [i for i, (_, n) in enumerate(seqs) for _ in range(n)]
    qsl = [0]
    for _, n in seqs:
        qsl.append(qsl[-1] + n)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    return StepContext(ops=ops, dtype=dtype, device=torch.device(DEV), num_tokens=len(pos), num_seqs=len(seqs),
                       max_q_len=max(n for _, n in seqs), max_kv_len=max(s + n for s, n in seqs), token_ids=t([0] * len(pos)),
                       positions=t(pos), token_seq=t(tseq), query_start_loc=t(qsl), seq_lens=t([s + n for s, n in seqs]),
                       slot_ids=t(slots if slots is not None else list(range(len(seqs)))), logit_rows=t([0]), num_logit_rows=0,
                       block_tables={0: tables})


def rel(a, b):
    return ((a.double().cpu() - b.double()).abs().max() / b.double().abs().max()).item()


def whole_sum(o):
    return o.float().sum(0) if o.dim() == 3 else o.float()


def part_with_weights(spec, dtype, ops, seed, page=16, scale=0.15, edit=None):
    """The mixer with random tensors (matrices as the run's dtype stores them) and the same tensors in float64 for the plain
    implementation, under the names of the model folder without the part's prefix."""
    part = build_part("mixer", spec)
    part.validate(ops, DT[dtype], page)
    part.bind(ops, DT[dtype], torch.device(DEV))
    g = torch.Generator().manual_seed(seed)
    w = {}
    for k, ps in part.param_specs().items():
        t = torch.randn(ps.shape, generator=g) * scale
        s = shaped(k, t, g)
        t = t if s is None else s
        w[k] = t.to(DT[dtype]).float() if ps.storage != "vector" else t
    if edit is not None:
        edit(w)
    part.load({k: (w[k].to(DT[dtype]) if ps.storage != "vector" else w[k]).to(DEV) for k, ps in part.param_specs().items()})
    return part, {k: v.double() for k, v in w.items()}


def run_paged(part, ops, dtype, x, cuts, page, table, pool_pages, step_cache=None):
    """One request through an attention part in steps of ``cuts`` tokens, from pages that hold noise where nothing was stored."""
    need = part.cache_needs()[0]
    pages = [torch.randn(pool_pages, need.num_kv_heads, page, need.head_dim, device=DEV).to(DT[dtype]) for _ in range(2)]
    outs, start = [], 0
    for n in cuts:
        ctx = ctx_for(ops, DT[dtype], [(start, n)], table)
        if step_cache is not None:
            ctx.step_cache.update(step_cache(start, n))
        outs.append(whole_sum(part.forward(x[start:start + n].to(DEV), ctx, PagedKVView(pages[0], pages[1], table, page))))
        start += n
    return torch.cat(outs)


def table_for(pages, seed):
    return (torch.randperm(pages, generator=torch.Generator().manual_seed(seed)) + 1).to(torch.int32).to(DEV)[None]


def attention_spec(m, width, eps, v_mix=None):
    return _mixer({"type": "attention", "mixer": m}, "a", width, eps, v_mix)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,keep", [(1, 0), (1, 2), (4, 3), (7, 5), (16, 1), (5, 40), (200, 4), (None, None)])
def test_attention_alone(ops, dtype, window, keep):
    """Whole, in portions and token by token from the pages; windows of one key, a page wide, across pages and wider than the
    prompt, with kept tokens inside a page, over several pages and more than the prompt has; scores mixed over grouped heads
    (without the mixing the output is another); part of every head rotated; a value size above the key size."""
    m = attn(6, 2, 20, 28, 0.25, window=window, keep=keep, rot=6, base=50.0)
    part, w = part_with_weights(attention_spec(m, 72, 2e-5), dtype, ops, 1, page=4)
    S, page = 45, 4
    x = torch.randn(S, 72, generator=torch.Generator().manual_seed(2)).to(DT[dtype])
    exp = pr.attention(x.double(), w, "", m, 2e-5, {})
    plain = pr.attention(x.double(), dict(w, talk=torch.eye(6, dtype=torch.float64)), "", m, 2e-5, {})
    if window != 1 or keep:
        assert (plain - exp).abs().max() > 5e-2 * exp.abs().max()
    for cuts in ([S], [10, 2, 33], [1] * S, [3, 1, 1, 17, 2, 21]):
        got = run_paged(part, ops, dtype, x, cuts, page, table_for(12, 3), 14)
        assert rel(got, exp) < (3e-5 if dtype == "float32" else 3e-2), (cuts, window, keep)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot", [
    (8, 2, 64, 64, 16), (4, 2, 128, 128, 128), (4, 1, 32, 48, 0), (3, 3, 32, 16, 32), (1, 1, 16, 16, 16), (6, 6, 64, 64, 64), (5, 5, 10, 6, 4),
    (16, 8, 96, 40, 48), (8, 4, 40, 13, 40), (4, 4, 100, 300, 20), (2, 1, 250, 64, 10)])
def test_attention_at_other_sizes(ops, dtype, heads, kv_heads, dim, vdim, rot):
    """Joint rows of 16 to 1,200 values: those the tile loop and the decode form take in bfloat16, those the tcgen05 kernels take,
    and those only the general kernel takes; value sizes that are multiples of nothing; one head; one kv head per head."""
    m = attn(heads, kv_heads, dim, vdim, dim ** -0.5, window=70, keep=5, rot=rot, base=500.0)
    part, w = part_with_weights(attention_spec(m, 96, 1e-6), dtype, ops, 3)
    S, page = 200, 16
    x = torch.randn(S, 96, generator=torch.Generator().manual_seed(4)).to(DT[dtype])
    exp = pr.attention(x.double(), w, "", m, 1e-6, {})
    for cuts in ([S], [130, 70], [69, 2, 100] + [1] * 29):
        got = run_paged(part, ops, dtype, x, cuts, page, table_for(14, 5), 16)
        assert rel(got, exp) < (3e-5 if dtype == "float32" else 3e-2), cuts[:3]


@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("window,keep", [(None, None), (200, 4), (333, 150), (64, 64)])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(8, 1, 128, 128), (16, 2, 64, 64), (8, 2, 128, 128), (4, 4, 64, 64), (8, 2, 120, 64), (16, 2, 32, 32), (16, 4, 128, 128),
                                                      (8, 8, 64, 64), (12, 3, 128, 64)])
def test_attention_on_the_tensor_core_kernels(ops, heads, kv_heads, dim, vdim, window, keep, page):
    """Pages of 16 and 64 keys and joint rows of 64, 128 and 256 values in bfloat16: prompt portions of several hundred rows take the
    tcgen05 kernels (two query tiles per CTA, per kv head where there are several), decoded tokens behind a long cache take the
    forms with the key range cut into pieces; the kept tokens lie in tiles of their own, far before the window's."""
    m = attn(heads, kv_heads, dim, vdim, dim ** -0.5, window=window, keep=keep, rot=32)
    part, w = part_with_weights(attention_spec(m, 96, 1e-6), "bfloat16", ops, 21)
    S = 1100
    x = torch.randn(S, 96, generator=torch.Generator().manual_seed(22)).to(torch.bfloat16)
    exp = pr.attention(x.double(), w, "", m, 1e-6, {})
    npages = -(-S // page) + 1
    kernels = set()
    plan = ops.joint_plan

    def noting(*a, **k):
        out = plan(*a, **k)
        kernels.add(out[0] + ("+pieces" if out[1] > 1 else ""))
        return out

    ops.joint_plan = noting
    try:
        for cuts in ([S], [600, 500], [1068] + [1] * 32, [300, 40, 760]):
            got = run_paged(part, ops, "bfloat16", x, cuts, page, table_for(npages, 23), npages + 2).cpu().double()
            err = (got - exp).abs().max(dim=-1).values / exp.abs().max(dim=-1).values.clamp_min(exp.abs().max() * 0.05)
            assert err.max() < 4e-2, (cuts[:3], int(err.argmax()), err.max(), kernels)
    finally:
        del ops.joint_plan
    assert any(k.startswith("tc") for k in kernels), kernels
    if kv_heads > 1 and vdim in (64, 128):
        assert any(k.startswith("tcpg") for k in kernels), kernels


@pytest.mark.parametrize("kernel", ["mma", "mma_c2", "mma_c4", "tc", "tcpp", "tcpg", "joint"])
def test_every_kernel_of_joint_rows_agrees(ops, kernel):
    """The same portion behind a cache through each kernel that takes its sizes, with the key range whole and in pieces."""
    H, G, D, Dv, W, page, window, keep = 8, 2, 64, 64, 128, 16, 90, 20
    lens, news = [260, 33, 150], ([2, 2, 2] if kernel.startswith("mma_c") else [40, 33, 17])
    g = torch.Generator().manual_seed(3)
    kp, vp = (torch.randn(60, 1, page, W, generator=g).to(torch.bfloat16).to(DEV) for _ in range(2))
    tables = torch.zeros(3, 17, dtype=torch.int32)
    perm = (torch.randperm(59, generator=g) + 1).tolist()
    for i, L in enumerate(lens):
        for j in range(-(-L // page)):
            tables[i, j] = perm.pop()
    T = sum(news)
    q = (torch.randn(T, H * W, generator=g) * 0.5).to(torch.bfloat16).to(DEV)
    qsl = torch.tensor([0, news[0], news[0] + news[1], T], dtype=torch.int32, device=DEV)
    exp = torch.zeros(T, H * Dv, dtype=torch.float64)
    for i, (L, n) in enumerate(zip(lens, news)):
        K = torch.cat([kp[p, 0] for p in tables[i]]).double().cpu()[:L]
        V = torch.cat([vp[p, 0] for p in tables[i]]).double().cpu()[:L]
        mask = pr.visible(L, {"size": window, "keep_first": keep})[L - n:]
        for h in range(H):
            s = q[int(qsl[i]):int(qsl[i + 1]), h * W:(h + 1) * W].double().cpu() @ K.T * 0.1
            c = h // (H // G)
            exp[int(qsl[i]):int(qsl[i + 1]), h * Dv:(h + 1) * Dv] = torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ V[:, c * Dv:(c + 1) * Dv]
    for pieces, length in ((1, 1 << 20 if kernel.startswith("mma_c") else 0), (2, 256), (4, 128)):
        out = torch.full((T, H * Dv), 9.0, dtype=torch.bfloat16, device=DEV)
        ops.paged_attention_joint(q, H, G, W, Dv, kp, vp, tables.to(DEV), page, qsl, torch.tensor(lens, dtype=torch.int32, device=DEV), 3,
                                  max(news), max(lens), 0.1, window, out, keep_first=keep, plan=(kernel, pieces, length))
        assert rel(out, exp) < 2e-2, (kernel, pieces)
        ops.check_tc()


def loud(x, at, gain=40.0):
    """Makes the token at ``at`` one that every query which sees it notices: the value it brings is large."""
    x = x.clone()
    x[at] *= gain
    return x


def test_window_edge_and_kept_tokens_show(ops):
    """One token brings a value far larger than the others'.  Every query up to the window's far edge must carry it and none past
    it; as the last kept token every query must, and as the first one behind the kept ones none past the window."""
    S, window, keep = 60, 9, 6
    m = attn(4, 2, 8, 8, 0.3, window=window, keep=keep, rot=4, base=30.0)
    part, w = part_with_weights(attention_spec(m, 72, 2e-5), "float32", ops, 5, page=4)
    base = torch.randn(S, 72, generator=torch.Generator().manual_seed(6)) * 0.3
    for at in (keep - 1, keep, 20):
        x = loud(base, at)
        exp = pr.attention(x.double(), w, "", m, 2e-5, {})
        for other in ({"size": window - 1, "keep_first": keep}, {"size": window + 1, "keep_first": keep}, {"size": window, "keep_first": keep - 1},
                      {"size": window, "keep_first": keep + 1}):
            if at != 20 or other["keep_first"] == keep:               # the oracle itself tells the masks apart
                diff = pr.attention(x.double(), w, "", dict(m, mask=other), 2e-5, {})
                assert (exp - diff).abs().max() > 1e-2 * exp.abs().max(), (at, other)
        for cuts in ([S], [26, 1, 1, 32], [29, 31], [28, 2, 2, 2, 26], [19, 1] + [1] * 40):
            got = run_paged(part, ops, "float32", x, cuts, 4, table_for(15, 7), 17).cpu().double()
            assert (got - exp).abs().max() < 3e-5 * exp.abs().max(), (at, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_among_hundreds(ops, dtype):
    """No window: the third of 700 tokens has a key that stands out for every query (its input is scaled and so is one value
    channel); decoded tokens and short portions run with the key range cut over CTAs, so dropping an early page shows."""
    S, at, page = 700, 2, 16
    m = attn(4, 2, 16, 16, 0.25, rot=16)
    part, w = part_with_weights(attention_spec(m, 72, 2e-5), dtype, ops, 7)
    x = loud(torch.randn(S, 72, generator=torch.Generator().manual_seed(8)) * 0.3, at, 300.0).to(DT[dtype])
    exp = pr.attention(x.double(), w, "", m, 2e-5, {})
    gone = x.clone(); gone[at] = 0
    assert (exp[-1] - pr.attention(gone.double(), w, "", m, 2e-5, {})[-1]).abs().max() > 0.05 * exp[-1].abs().max()
    for cuts in ([S], [650] + [1] * 50, [300, 2, 398]):
        got = run_paged(part, ops, dtype, x, cuts, page, table_for(S // page + 1, 9), S // page + 3).cpu().double()
        tol = 3e-5 if dtype == "float32" else 3e-2
        assert ((got - exp).abs().max(dim=-1).values < tol * exp.abs().max(dim=-1).values.clamp_min(exp.abs().max() * 0.05)).all(), cuts[:3]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("head_mix", [True, False])
def test_blended_values(ops, dtype, head_mix):
    """The first layer of the kind leaves its values, a later one stores (1 - l) v + l v_first; both with mixed scores and in
    the general attention step, whole, cut and token by token (the blended values are what is cached)."""
    m = attn(4, 2, 12, 20, 0.3, window=11, keep=2, rot=4, v_mix=True)
    S, page = 40, 4
    specs = [attention_spec(m, 72, 2e-5, kind) for kind in ("first", "mix")]
    if not head_mix:
        specs = [PartSpec(s.kind, s.prefix, dict(s.args, head_mix=None)) for s in specs]
    (first, w1), (second, w2) = (part_with_weights(s, dtype, ops, 30 + i, page=page) for i, s in enumerate(specs))
    if not head_mix:
        w1, w2 = (dict(w, talk=torch.eye(4, dtype=torch.float64)) for w in (w1, w2))
    g = torch.Generator().manual_seed(12)
    xs = [torch.randn(S, 72, generator=g).to(DT[dtype]) for _ in range(2)]
    shared = {}
    e1 = pr.attention(xs[0].double(), w1, "", m, 2e-5, shared)
    e2 = pr.attention(xs[1].double(), w2, "", m, 2e-5, shared)
    alone = pr.attention(xs[1].double(), w2, "", m, 2e-5, {})
    assert (alone - e2).abs().max() > 0.1 * e2.abs().max()
    for cuts in ([S], [13, 2, 25], [1] * S):
        need = first.cache_needs()[0]
        pools = [[torch.randn(12, need.num_kv_heads, page, need.head_dim, device=DEV).to(DT[dtype]) for _ in range(2)] for _ in range(2)]
        table, start, got = table_for(10, 4), 0, [[], []]
        for n in cuts:
            ctx = ctx_for(ops, DT[dtype], [(start, n)], table)
            for i, part in enumerate((first, second)):
                got[i].append(whole_sum(part.forward(xs[i][start:start + n].to(DEV), ctx, PagedKVView(*pools[i], table, page))))
            start += n
        for out, exp in zip(got, (e1, e2)):
            assert rel(torch.cat(out), exp) < (3e-5 if dtype == "float32" else 3e-2), cuts[:3]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [16, 64, 128])
def test_kept_tokens_without_mixed_scores(ops, dtype, dim):
    """The window that keeps first tokens in plain grouped attention (the kernels of the other designs)."""
    m = attn(8, 2, dim, dim, dim ** -0.5, window=50, keep=10, rot=dim)
    spec = attention_spec(m, 96, 1e-6)
    part, w = part_with_weights(PartSpec(spec.kind, spec.prefix, dict(spec.args, head_mix=None)), dtype, ops, 13)
    w = dict(w, talk=torch.eye(8, dtype=torch.float64))
    S, page = 400, 16
    x = torch.randn(S, 96, generator=torch.Generator().manual_seed(14)).to(DT[dtype])
    exp = pr.attention(x.double(), w, "", m, 1e-6, {})
    for cuts in ([S], [130, 270], [369, 2] + [1] * 29):
        got = run_paged(part, ops, dtype, x, cuts, page, table_for(26, 5), 28)
        assert rel(got, exp) < (3e-5 if dtype == "float32" else 3e-2), cuts[:3]


def run_states(part, ops, dtype, xs, cuts, slots, noise=True):
    """Requests side by side through a recurrent part, each cut as ``cuts`` says (a list per request; 0: left out of the step)."""
    rows = 6
    states = [torch.randn(rows, *n.shape, device=DEV) for n in part.cache_needs()]
    for s in states:
        for slot in slots:
            s[slot].zero_()
    at, outs = [0] * len(xs), [[] for _ in xs]
    for step in zip(*cuts):
        live = [i for i, n in enumerate(step) if n]
        x = torch.cat([xs[i][at[i]:at[i] + step[i]] for i in live]).to(DEV)
        ctx = ctx_for(ops, DT[dtype], [(at[i], step[i]) for i in live], slots=[slots[i] for i in live])
        o = whole_sum(part.forward(x, ctx, [FixedStateView(s) for s in states])).cpu()
        k = 0
        for i in live:
            outs[i].append(o[k:k + step[i]])
            k += step[i]
            at[i] += step[i]
    return [torch.cat(o) for o in outs]


CUTS = [[[60, 0, 0], [0, 35, 0], [0, 0, 7]],
        [[20, 2, 38, 0], [1, 1, 30, 3], [0, 2, 0, 5]],
        [[1] * 60, [1] * 35 + [0] * 25, [1] * 7 + [0] * 53],
        [[3, 0, 1, 16, 40], [17, 1, 2, 0, 15], [0, 7, 0, 0, 0]]]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", [mamba(72, 10, 5, 4), mamba(64, 16, 8, 3), mamba(30, 1, 3, 1), mamba(50, 24, 12, 2), mamba(20, 70, 9, 5),
                               mamba(256, 128, 16, 4), mamba(33, 3, 1, 8), mamba(16, 33, 20, 3)], ids=lambda m: "-".join(map(str, m.values())))
def test_selective_scan_alone(ops, dtype, m):
    """Three requests side by side in scattered slots, whole, in portions, token by token and left out of steps: states of 1 to 128
    values, one to eight taps (more than a portion brings), ranks and channel counts that are multiples of nothing."""
    part, w = part_with_weights(_mixer({"type": "mamba1", "mixer": m}, "a", 48, 1e-5), dtype, ops, 2, scale=0.25)
    g = torch.Generator().manual_seed(3)
    xs = [torch.randn(n, 48, generator=g).to(DT[dtype]) for n in (60, 35, 7)]
    exps = [pr.mamba1(x.double(), w, "", m, 1e-5, {}) for x in xs]
    for cuts in CUTS:
        for got, exp in zip(run_states(part, ops, dtype, xs, cuts, [4, 0, 2]), exps):
            assert rel(got, exp) < (3e-5 if dtype == "float32" else 4e-2), cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", [lightning(3, 12, 20, [0.3, 0.9, 0.99]), lightning(1, 10, 14, [0.0]), lightning(2, 64, 32, [1.0, 0.97]),
                               lightning(4, 8, 200, [0.5, 0.6, 0.7, 0.999]), lightning(2, 160, 24, [0.8, 0.2])], ids=lambda m: f"{m['heads']}-{m['dim']}-{m['vdim']}")
def test_linear_attention_alone(ops, dtype, m):
    """silu on q, k and v, one norm over all heads with a weight per value, a sigmoid gate; decays of zero and one among them."""
    part, w = part_with_weights(_mixer({"type": "lightning", "mixer": m}, "a", 48, 1e-5), dtype, ops, 2, scale=0.25)
    g = torch.Generator().manual_seed(3)
    xs = [torch.randn(n, 48, generator=g).to(DT[dtype]) for n in (60, 35, 7)]
    exps = [pr.lightning(x.double(), w, "", m, 1e-5, {}) for x in xs]
    for cuts in CUTS:
        for got, exp in zip(run_states(part, ops, dtype, xs, cuts, [4, 0, 2]), exps):
            assert rel(got, exp) < (3e-5 if dtype == "float32" else 3e-2), cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_scans_carry_a_first_token_over_a_long_prompt(ops, dtype):
    """1,300 tokens, walked in parts, of which only the first is loud: states that forget slowly (steps near zero; a decay of 0.9995)
    must still show it at the end, after parts, portions and single tokens alike."""
    S = 1300
    x = torch.randn(S, 48, generator=torch.Generator().manual_seed(5)) * 0.2
    x[0] *= 60.0
    x = x.to(DT[dtype])
    gone = x.clone(); gone[0] = 0

    def slow(w):
        if "dt.b" in w:
            w["dt.b"], w["A_log"], w["D"] = torch.full_like(w["dt.b"], -5.0), w["A_log"] - 3.0, w["D"] * 0.1

    for kind, m, fn in (("mamba1", mamba(40, 6, 4, 3), pr.mamba1), ("lightning", lightning(2, 16, 16, [0.9995, 0.99]), pr.lightning)):
        part, w = part_with_weights(_mixer({"type": kind, "mixer": m}, "a", 48, 1e-5), dtype, ops, 4, scale=0.25, edit=slow)
        exp = fn(x.double(), w, "", m, 1e-5, {})
        assert (exp[-1] - fn(gone.double(), w, "", m, 1e-5, {})[-1]).abs().max() > 0.05 * exp[-1].abs().max()
        for cuts in ([[S]], [[1250] + [1] * 50], [[500, 2, 300, 498]]):
            got = run_states(part, ops, dtype, [x], cuts, [1])[0]
            tail = (got[200:].double() - exp[200:]).abs().max() / exp[200:].abs().max()
            # (bfloat16: q . k_0 cancels at some tokens; rounding the projections in the plain implementation moves those by 6 % as well)
            assert tail < (5e-5 if dtype == "float32" else 0.1), (kind, [c[:3] for c in cuts])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,width", [(1, 50), (7, 192), (96, 1024), (200, 2048), (33, 4100), (3, 8192), (2, 9000)])
def test_two_norm_step(ops, dtype, rows, width):
    """x += rms(delta) * w_b, then rms(x) * w, from a delta in the compute dtype, in 32-bit and as partial sums; gathered rows."""
    g = torch.Generator().manual_seed(rows + width)
    resid = torch.randn(rows, width, generator=g)
    delta = (torch.randn(rows, width, generator=g) * 3).to(DT[dtype])
    wb, w = 1 + 0.3 * torch.randn(width, generator=g), 1 + 0.3 * torch.randn(width, generator=g)
    parts = torch.randn(3, rows, width, generator=g)
    for d in (delta, parts, parts[0]):
        dd = d.double().sum(0) if d.dim() == 3 else d.double()
        x = resid.double() + pr.rms_norm(dd, 1e-3, wb.double())
        y = pr.rms_norm(x, 1e-5, w.double())
        r, out = resid.clone().to(DEV), torch.empty(rows, width, dtype=DT[dtype], device=DEV)
        ops.sandwich_norm(r, d.to(DEV), wb.to(DEV), 1e-3, w.to(DEV), 1e-5, out)
        assert rel(r, x) < 2e-6 and rel(out, y) < (2e-6 if dtype == "float32" else 5e-3)
        pick = torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
        r, out = resid.clone().to(DEV), torch.empty(2, width, dtype=DT[dtype], device=DEV)
        ops.sandwich_norm(r, d.to(DEV), wb.to(DEV), 1e-3, w.to(DEV), 1e-5, out, rows=pick, num_rows=2)
        assert torch.equal(r.cpu(), resid) and rel(out, y[[rows - 1, 0]]) < (2e-6 if dtype == "float32" else 5e-3)


def test_blocks_share_a_stream(ops):
    """A block that leaves its output unnormed in the stream may be followed by one that norms inputs only."""
    from tiny_transformer_inference_engine_b200.parts.norm import RMSNorm
    g = torch.Generator().manual_seed(1)
    out_norm, next_norm = RMSNorm("a", 64, 1e-5, "w", scalar=True), RMSNorm("b", 64, 1e-5, "w")
    for n, wt in ((out_norm, torch.tensor(1.7)), (next_norm, torch.randn(64, generator=g))):
        n.bind(ops, torch.float32, torch.device(DEV))
        n.load({"w": wt.to(DEV)})
    resid, delta = torch.randn(5, 64, generator=g), torch.randn(5, 64, generator=g)
    stream = ResidualStream(resid.clone().to(DEV), delta.to(DEV))
    stream.delta_norm = out_norm
    got = next_norm.add_norm(stream.resid, stream.delta, stream.delta_norm)
    x = resid.double() + pr.rms_norm(delta.double(), 1e-5, 1.7)
    assert rel(got, pr.rms_norm(x, 1e-5, next_norm.weight.double().cpu())) < 2e-6


@pytest.mark.parametrize("softcap", [None, 3.0])
def test_head_scales_and_caps(ops, softcap):
    head = build_part("head", PartSpec("linear", "", {"dim": 32, "vocab_size": 50, "name": "head", "softcap": softcap, "scale": 2.5}))
    head.bind(ops, torch.float32, torch.device(DEV))
    g = torch.Generator().manual_seed(1)
    W, x = torch.randn(50, 32, generator=g), torch.randn(4, 32, generator=g)
    head.load({"head": W.to(DEV)})
    exp = x.double() @ W.double().T * 2.5
    if softcap:
        exp = softcap * torch.tanh(exp / softcap)
    assert rel(head.forward(x.to(DEV)), exp) < 2e-6
