"""The Fokurax design in the engine against the plain implementation (plain_fokurax.py): each mechanism alone, whole prompts,
decoding through the cache, portions down to two tokens, mixed batches with pages and slots used again, keys at the edges of
chunks and pages, the first tokens and keys far back, other sizes, and greedy generation through the scheduler."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import plain_fokurax as pf
import trace_util as tu

from tiny_transformer_inference_engine_b200 import Engine, ModelConfig, EngineConfig, CacheConfig, SchedulerConfig, SamplingParams
from tiny_transformer_inference_engine_b200.parts.base import PartSpec, PagedKVView, ResidualStream, StepContext
from tiny_transformer_inference_engine_b200.parts.embedding import TOKEN_SIDE
from tiny_transformer_inference_engine_b200.registry import build_part
from tiny_transformer_inference_engine_b200.weights import random_tensors
from tiny_transformer_inference_engine_b200.models.fokurax import _mixer, _ffn                   # config.json's layer entry -> the part

from fokurax_configs import ALL as CONFIGS, FOK_A, FOK_B, FOK_C, FOK_D, attn, dense, layer, model, moe, yarn

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def ops():
    from tiny_transformer_inference_engine_b200.ops import get_ops
    return get_ops(DEV)


def weights_for(cfg, seed, store="float32"):
    """Random weights at which every mechanism shows: norm weights away from zero, biases and gates of about one, embeddings and
    side values of about one."""
    w = random_tensors(ModelConfig.from_dict(cfg), seed, std=0.15, store_dtype=store)
    g = torch.Generator().manual_seed(seed + 1)
    for k in sorted(w):
        if k.endswith(("norm1", "final.norm")):
            w[k] = (torch.randn(w[k].shape, generator=g) * 0.3).to(w[k].dtype)
        elif k.endswith("side.norm"):
            w[k] = (1.0 + torch.randn(w[k].shape, generator=g) * 0.3).to(w[k].dtype)
        elif k in ("embed", "side.embed") or k.endswith(".b"):
            w[k] = w[k] * 5.0
    return w


def engine_for(cfg, w, dtype, page=16, pages=64, max_seqs=4, budget=64, graphs=False):
    ec = EngineConfig(dtype=dtype, device=DEV, use_cuda_graphs=graphs,
                      cache=CacheConfig(block_size=page, num_gpu_blocks=pages),
                      sched=SchedulerConfig(max_num_seqs=max_seqs, max_num_batched_tokens=budget))
    return Engine(ModelConfig.from_dict(cfg), w, ec)


def requests(cfg, lens, seed):
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lens)}


def as_stored(k, v, dtype):
    """A tensor as the engine keeps it: matrices in the run's dtype, norm weights in 32-bit, integer tables."""
    if v.is_floating_point() and dtype == "bfloat16" and not k.endswith(("norm1", "norm")):
        return v.to(torch.bfloat16).double()
    return v.double() if v.is_floating_point() else v


def expected_for(cfg, w, reqs, dtype):
    ww = {k: as_stored(k, v, dtype) for k, v in w.items()}
    return {rid: pf.forward(cfg, ww, toks) for rid, toks in reqs.items()}


def check(got, exp, dtype, tail16=0.1, typical16=3e-2, worst32=1e-4):
    """32-bit: every place within 1e-4 of the row's largest logit.  bfloat16: these models are narrow and rounding alone moves a
    typical row by one or two percent, so the run is held to the typical error and to nine rows in ten (every mechanism alone is
    held to its largest error in both dtypes below)."""
    errs = []
    for (rid, pos), row in got.items():
        ref = exp[rid][pos]
        errs.append((((row.double() - ref).abs().max() / ref.abs().max()).item(), rid, pos))
    errs.sort(reverse=True)
    n = len(errs)
    assert all(e[0] == e[0] for e in errs), "a NaN among the logits"
    if dtype == "float32":
        assert errs[0][0] < worst32, errs[:3]
    else:
        assert errs[n // 2][0] < typical16 and errs[n // 10][0] < tail16, (errs[n // 2], errs[n // 10], errs[:3])


# ------------------------------------------------------------------------------------------ the whole model, four cuts
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_schedules_against_plain_model(name, dtype):
    cfg = CONFIGS[name]
    w = weights_for(cfg, 5 + ord(name))
    reqs = requests(cfg, [1, 2, 37, 70, 101, 23], seed=3)
    exp = expected_for(cfg, w, reqs, dtype)
    page = {"A": 16, "B": 8, "C": 4, "D": 2}[name]
    for cut in (tu.whole, tu.prefill_then_decode, tu.portions, tu.mixed):
        steps = cut(reqs)
        tokens = tu.max_live_tokens(steps, rounding=page)
        eng = engine_for(cfg, w, dtype, page=page, pages=tokens // page + 2)        # no slack: pages and slots are used again
        check(tu.run_steps(eng, steps), exp, dtype)


def test_residual_stream_layer_by_layer(ops):
    """The stream behind every layer, the waiting side input added, against the plain model's."""
    cfg = FOK_A
    w = weights_for(cfg, 12)
    toks = requests(cfg, [33], 2)["r0"]
    plain = []
    pf.forward(cfg, {k: as_stored(k, v, "float32") for k, v in w.items()}, toks, after_layer=lambda i, x: plain.append(x))
    eng = engine_for(cfg, w, "float32")
    seen = []

    def after(e, stream):
        d = stream.delta.double() if stream.delta.dim() == 2 else stream.delta.double().sum(0)
        y = d / torch.sqrt((d * d).mean(-1, keepdim=True) + stream.delta_norm.eps) * stream.delta_norm.weight32.double()
        seen.append((stream.resid.double() + y).cpu())

    eng.stepper.model.after_entry = after
    tu.run_steps(eng, tu.whole({"r0": toks}))
    assert len(seen) == len(plain) == 5
    for i, (a, b) in enumerate(zip(seen, plain)):
        assert (a - b).abs().max() < 2e-5 * b.abs().max(), i


def test_long_decode_past_chunks_and_pages():
    """A short prompt, then 150 tokens one by one: the edges of three chunk sizes and many page edges pass under decoded tokens."""
    w = weights_for(FOK_A, 77)
    reqs = requests(FOK_A, [160], seed=9)
    eng = engine_for(FOK_A, w, "float32", page=8, pages=24)
    check(tu.run_steps(eng, tu.prefill_then_decode(reqs, tail=150)), expected_for(FOK_A, w, reqs, "float32"), "float32")


def test_batch_of_unequal_requests_equals_each_alone():
    w = weights_for(FOK_A, 21)
    reqs = requests(FOK_A, [3, 50, 1, 29], seed=4)
    eng = engine_for(FOK_A, w, "float32", pages=40)
    alone = tu.run_steps(eng, tu.whole(reqs))
    together = tu.run_steps(eng, [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()],
                                   "end": list(reqs)}])
    for key, row in alone.items():
        assert (row - together[key]).abs().max() <= 2e-5 * row.abs().max(), key


def test_slots_and_pages_used_again_carry_nothing_over():
    """The same request replayed after others have used (and dirtied) its slot and pages gives the same logits to the bit."""
    w = weights_for(FOK_A, 23)
    reqs = requests(FOK_A, [40, 33, 40], seed=8)
    reqs["r2"] = list(reqs["r0"])
    eng = engine_for(FOK_A, w, "float32", page=8, pages=8, max_seqs=2)
    got = tu.run_steps(eng, tu.portions(reqs))
    for pos in range(40):
        assert torch.equal(got[("r0", pos)], got[("r2", pos)]), pos
    check(got, expected_for(FOK_A, w, reqs, "float32"), "float32")


@pytest.mark.parametrize("name", ["A", "B"])
def test_first_tokens_of_a_sequence(name):
    """Requests of one to three tokens, alone and beside a longer one, whole and one token at a time."""
    cfg = CONFIGS[name]
    w = weights_for(cfg, 41)
    reqs = requests(cfg, [1, 2, 3, 30], seed=5)
    exp = expected_for(cfg, w, reqs, "float32")
    eng = engine_for(cfg, w, "float32", page=2, pages=40)
    check(tu.run_steps(eng, tu.whole(reqs)), exp, "float32")
    check(tu.run_steps(eng, tu.prefill_then_decode(reqs, tail=29)), exp, "float32")
    check(tu.run_steps(eng, [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in reqs.items()], "end": list(reqs)}]), exp, "float32")


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler(graphs):
    """Tokens sampled on the device feed the next captured step: the experts' table and the side table are looked up by them."""
    cfg = dict(FOK_A, max_seq_len=256)
    w = weights_for(cfg, 31)
    prompts = [[5, 9, 2], list(range(10, 41)), [7]]
    want = []
    for p in prompts:
        toks = list(p)
        for _ in range(14):                                           # past a chunk edge for every prompt
            toks.append(int(torch.argmax(pf.forward(cfg, w, toks)[-1])))
        want.append(toks[len(p):])
    eng = engine_for(cfg, w, "float32", pages=40, max_seqs=4, budget=16, graphs=graphs)
    assert eng.generate(prompts, SamplingParams(max_new_tokens=14, greedy=True)) == want


@pytest.mark.parametrize("graphs", [False, True])
def test_two_streams_change_nothing(ops, graphs):
    """Small steps run a layer's feed-forward beside its attention; the same steps on one stream give the same bits, eagerly and from
    captured graphs, also where steps of either kind alternate."""
    cfg = dict(FOK_C, max_seq_len=256)
    w = weights_for(cfg, 19)
    prompts = [list(range(3, 80)), [4, 4, 9], list(range(50, 57))]
    runs = {}
    saved = ops.branch_max_tokens
    try:
        for limit in (0, 20, 64):
            ops.branch_max_tokens = limit
            eng = engine_for(cfg, w, "float32", pages=60, budget=40, graphs=graphs)
            assert eng.ops is ops
            runs[limit] = (tu.run_steps(eng, tu.mixed(requests(cfg, [60, 90, 5], 6))), eng.generate(prompts, SamplingParams(max_new_tokens=20, greedy=True)))
    finally:
        ops.branch_max_tokens = saved
    for limit in (20, 64):
        assert runs[limit][1] == runs[0][1]
        assert all(torch.equal(row, runs[limit][0][key]) for key, row in runs[0][0].items())


def test_command_line_and_trace_runner_with_a_model_folder(tmp_path):
    """A folder written in the random-weights mode (bfloat16 on disk), generated from by the command line and replayed by the
    trace runner: the architecture is picked from config.json by both."""
    import numpy as np
    from safetensors.torch import load_file
    from tiny_transformer_inference_engine_b200 import write_random_model
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = dict(FOK_B, max_seq_len=96)
    folder = write_random_model(ModelConfig.from_dict(cfg), 13, str(tmp_path / "model"), std=0.15, store_dtype="bfloat16")
    w = load_file(os.path.join(folder, "model.safetensors"))
    prompt = [4, 90, 7, 7, 23]
    run = subprocess.run([sys.executable, "-m", "tiny_transformer_inference_engine_b200", "--model", folder, "--tokens", "6", "--greedy",
                          "--dtype", "float32", "--num-gpu-blocks", "16", "--prompt-ids", ",".join(map(str, prompt))],
                         cwd=root, capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    toks = list(prompt)
    for _ in range(6):
        toks.append(int(torch.argmax(pf.forward(cfg, w, toks)[-1])))
    assert json.loads(run.stdout.strip().split("\n")[-1])["generated_ids"] == toks[len(prompt):]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:7], "want": [0, 6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[7:9], "want": [1]}, {"id": "b", "tokens": toks[:3], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[3:4], "want": [0]}], "end": ["b"]}]
    out = tmp_path / "out"
    run = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", cwd=root, capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [l for l in run.stdout.split("\n") if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    exp = pf.forward(cfg, w, toks)
    for name, rows in (("0.f32", [0, 6]), ("1.f32", [8]), ("2.f32", [3])):
        got = torch.from_numpy(np.fromfile(str(out / name), dtype="<f4").reshape(len(rows), cfg["vocab"]))
        assert ((got.double() - exp[rows]).abs().max() / exp[rows].abs().max()).item() < 1e-4, name


# ------------------------------------------------------------------------------------------ each mechanism alone
def ctx_for(ops, dtype, seqs, table, token_ids=None):
    pos = [s + i for s, n in seqs for i in range(n)]
    tseq = [i for i, (_, n) in enumerate(seqs) for _ in range(n)]
    qsl = [0]
    for _, n in seqs:
        qsl.append(qsl[-1] + n)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    return StepContext(ops=ops, dtype=dtype, device=torch.device(DEV), num_tokens=len(pos), num_seqs=len(seqs),
                       max_q_len=max(n for _, n in seqs), max_kv_len=max(s + n for s, n in seqs),
                       token_ids=t([0] * len(pos) if token_ids is None else token_ids),
                       positions=t(pos), token_seq=t(tseq), query_start_loc=t(qsl), seq_lens=t([s + n for s, n in seqs]),
                       slot_ids=t(list(range(len(seqs)))), logit_rows=t([0]), num_logit_rows=0, block_tables={0: table})


def rel(a, b):
    return ((a.double().cpu() - b.double()).abs().max() / b.double().abs().max()).item()


def whole_rows(y):
    return y.float().sum(0) if y.dim() == 3 else y.float()


def part_with_weights(category, spec, dtype, ops, seed, scale=0.15, edit=None):
    """The part with random tensors (matrices as the run's dtype stores them) and the same tensors in float64 for the plain
    implementation, under the names of the model folder without the part's prefix."""
    part = build_part(category, spec)
    part.bind(ops, DT[dtype], torch.device(DEV))
    g = torch.Generator().manual_seed(seed)
    w = {}
    for k, ps in part.param_specs().items():
        if ps.storage == "table":
            w[k] = torch.rand((*ps.shape[:-1], ps.high), generator=g).argsort(-1)[..., :ps.shape[-1]].to(torch.int32)
            continue
        t = torch.randn(ps.shape, generator=g) * scale
        w[k] = t.to(DT[dtype]).float() if ps.storage == "matrix" else t
    if edit is not None:
        edit(w)
    part.load({k: (w[k].to(DT[dtype]) if ps.storage == "matrix" else w[k]).to(DEV) for k, ps in part.param_specs().items()})
    return part, {k: v.double() if v.is_floating_point() else v.long() for k, v in w.items()}


def run_attention(parts, ops, dtype, x, cuts, page, table, pool_pages):
    """One request through the parts (the first stores keys and values, the others read them) in steps of ``cuts`` tokens, from pages
    that hold noise where nothing was stored; the parts' outputs."""
    first = parts[0]
    pages = [torch.randn(pool_pages, first.num_kv_heads, page, first.padded_dim, device=DEV).to(DT[dtype]) for _ in range(2)]
    outs, start = [[] for _ in parts], 0
    for n in cuts:
        ctx = ctx_for(ops, DT[dtype], [(start, n)], table)
        for i, part in enumerate(parts):
            outs[i].append(whole_rows(part.forward(x[start:start + n].to(DEV), ctx, PagedKVView(pages[0], pages[1], table, page, writable=i == 0))))
        start += n
    return [torch.cat(o) for o in outs]


def plain_attention(x, w, m, eps, w_kv=None, m_kv=None):
    kv = pf.keys_values(x.double(), w if w_kv is None else w_kv, "", m if m_kv is None else m_kv, eps)
    return pf.attention(x.double(), w, "", m, eps, kv)


TABLE = [9, 2, 7, 1, 3, 6, 11, 4, 8, 5, 10, 12]
CUTS = ([45], [10, 2, 33], [1] * 45, [3, 1, 1, 17, 2, 21])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m", [
    attn(4, 2, 20, 28, 0.5, chunk=7, rot=6, base=50.0),                                       # part of a head, a larger value size, head sizes that are padded
    attn(3, 3, 16, 16, 0.6, chunk=1, rot=16),                                                 # a chunk of one key, whole heads
    attn(5, 1, 32, 8, 0.4, chunk=4, rot=32, base=2000.0, scaling=yarn(4.0, 16, 3.0, 0.5)),    # a chunk of one page, rescaled frequencies
    attn(2, 1, 24, 24, 0.7, chunk=16),                                                        # no rotation
    attn(8, 2, 64, 64, 0.25, chunk=30, rot=32, base=300.0, scaling=yarn(2.0, 32, 4.0, 1.0)),  # a tensor-core size
    attn(4, 1, 128, 128, 0.2, chunk=200, rot=64),                                             # a chunk longer than the prompt
    attn(2, 2, 6, 4, 1.0, rot=2),                                                             # no chunks
])
def test_attention_alone(ops, dtype, m):
    """Whole, in portions and token by token from the pages; the norm sits behind the rotation (whose rescaled magnitude it sees on
    the rotated values only)."""
    eps = 2e-2                                                         # (large, so that its place inside the root shows)
    part, w = part_with_weights("mixer", _mixer(m, "a", 72, eps), dtype, ops, 1)
    x = torch.randn(45, 72, generator=torch.Generator().manual_seed(2)).to(DT[dtype])
    exp = plain_attention(x, w, m, eps)
    table = torch.tensor([TABLE], dtype=torch.int32, device=DEV)
    for cuts in CUTS:
        assert rel(run_attention([part], ops, dtype, x, cuts, 4, table, 14)[0], exp) < (3e-5 if dtype == "float32" else 3e-2), cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_that_read_another_layers_cache(ops, dtype):
    """Queries of their own, the stored keys (normed and rotated by their own layer) and values; chunks and scales of their own, one
    reader without chunks."""
    own = attn(4, 2, 24, 16, 0.5, chunk=9, rot=12, base=50.0)
    readers = [dict(own, kv_from=0, scale=0.9), dict(own, kv_from=0, mask={"size": 14}), {k: v for k, v in dict(own, kv_from=0).items() if k != "mask"}]
    built = [part_with_weights("mixer", _mixer(m, "a", 72, 1e-5, readers if i == 0 else ()), dtype, ops, 30 + i) for i, m in enumerate([own] + readers)]
    assert set(built[1][1]) == {"q", "o"}
    x = torch.randn(45, 72, generator=torch.Generator().manual_seed(3)).to(DT[dtype])
    exps = [plain_attention(x, b[1], m, 1e-5, built[0][1], own) for b, m in zip(built, [own] + readers)]
    table = torch.tensor([TABLE], dtype=torch.int32, device=DEV)
    for cuts in CUTS:
        for i, (got, exp) in enumerate(zip(run_attention([b[0] for b in built], ops, dtype, x, cuts, 4, table, 14), exps)):
            assert rel(got, exp) < (3e-5 if dtype == "float32" else 3e-2), (cuts, i)


@pytest.mark.parametrize("reader", [False, True])
def test_chunk_edge_shows(ops, reader):
    """One token brings a value far larger than the others'; every later query of its chunk must carry it and the first query of the
    next chunk must not: a chunk one position longer or shorter, or chunks counted from the cut, move the edge."""
    chunk, S, key_at = 9, 40, 20                                       # chunk 2 holds 18..26
    own = attn(2, 1, 8, 8, 0.5, chunk=chunk if not reader else 40, rot=4, base=30.0)
    m = dict(own, kv_from=0, mask={"size": chunk}) if reader else own
    parts = [part_with_weights("mixer", _mixer(own, "a", 72, 2e-5, [m] if reader else ()), "float32", ops, 5)]
    if reader:
        parts.append(part_with_weights("mixer", _mixer(m, "a", 72, 2e-5), "float32", ops, 6))
    x = torch.randn(S, 72, generator=torch.Generator().manual_seed(6)) * 0.3
    x[key_at] *= 40.0

    def plain(xx, size=chunk):
        return plain_attention(xx, parts[-1][1], dict(m, mask={"size": size}), 2e-5, parts[0][1], own)

    exp = plain(x)
    for other in (chunk - 1, chunk + 1):                               # the oracle itself tells the sizes apart at the edge
        assert (exp[24:29] - plain(x, other)[24:29]).abs().max() > 1e-2 * exp.abs().max()
    gone = x.clone(); gone[key_at] = 0
    moved = (plain(gone) - exp).abs().max(dim=-1).values
    assert moved[key_at:27].min() > 0.05 * exp.abs().max() and moved[27:].max() == 0      # 26 still sees the loud value, 27 opens a chunk
    table = torch.tensor([[3, 1, 2, 5, 4, 6, 7, 8, 9, 10]], dtype=torch.int32, device=DEV)
    for cuts in ([S], [26, 1, 1, 12], [27, 13], [21, 2, 2, 2, 2, 11], [19, 1] + [1] * 20):
        got = run_attention([p[0] for p in parts], ops, "float32", x, cuts, 4, table, 12)[-1].cpu().double()
        assert (got - exp).abs().max() < 3e-5 * exp.abs().max(), cuts


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [32, 64, 128])
def test_far_key_among_hundreds(ops, dtype, dim):
    """A chunk of 650 keys over many pages.  Values, queries and keys read three parts of the input; a few tokens carry, where queries
    read, what one early token carries where keys do, through the same matrix: this one of hundreds of scores stands out and
    their outputs are that token's value.  The same query in the next chunk must not find it."""
    S, key_at, page, eps = 700, 2, 16, 1e-5
    asks = (40, 300, 640, 649, 655, 699)
    m = attn(2, 1, dim, 32, 12.0 / dim, chunk=650)

    def apart(w):
        both = w["q"][:dim, 8:40].clone()
        w["q"].zero_(); w["k"].zero_(); w["v"][:, 8:] = 0
        w["q"][:dim, 8:40] = w["q"][dim:, 8:40] = w["k"][:, 40:] = both

    part, w = part_with_weights("mixer", _mixer(m, "a", 72, eps), dtype, ops, 7, edit=apart)
    x = torch.randn(S, 72, generator=torch.Generator().manual_seed(8)).to(DT[dtype])
    for t in asks:
        x[t, 8:40] = x[key_at, 40:]
    exp = plain_attention(x, w, m, eps)
    other = x.clone(); other[key_at, :8] = x[1, :8]                    # with another value there the askers of its chunk answer otherwise
    change = (plain_attention(other, w, m, eps) - exp).abs().max(dim=-1).values / exp.abs().max(dim=-1).values
    assert all(change[t] > 0.5 for t in asks[:4]) and change[655] == 0 and change[699] == 0
    perm = torch.randperm(S // page + 1, generator=torch.Generator().manual_seed(9)) + 1
    table = perm.to(torch.int32).to(DEV)[None]
    for cuts in ([S], [630] + [1] * 70, [300, 2, 398]):
        got = run_attention([part], ops, dtype, x, cuts, page, table, S // page + 3)[0].cpu().double()
        err = (got - exp).abs().max(dim=-1).values / exp.abs().max(dim=-1).values
        assert err.max() < (5e-5 if dtype == "float32" else 5e-2), (cuts[:3], int(err.argmax()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,Dv,rot", [(128, 128, 64), (64, 32, 64), (96, 96, 16), (20, 28, 6), (256, 256, 32), (16, 8, 0)])
def test_norm_behind_the_rotation(ops, dtype, D, Dv, rot):
    """The store kernel alone, both its forms (eight values per thread; one head per block): q and the pages' k rows have a root
    mean square of one behind a rotation that magnifies, v rows are as projected, the padding is zero."""
    T, H, G, page = 5, 4, 2, 2
    Dp = -(-max(D, Dv) // 16) * 16
    g = torch.Generator().manual_seed(D + rot)
    proj = torch.randn(T, (H + G) * D + G * Dv, generator=g).to(DT[dtype])
    f, mag = pf.frequencies({"dims": rot, "base": 70.0, "scaling": yarn(6.0, 16, 2.0, 0.5)}) if rot else ([], 1.0)
    pos = torch.tensor([3, 4, 5, 6, 7], dtype=torch.int32, device=DEV)
    cs = ops.rope_table(pos, torch.tensor(f, dtype=torch.float32, device=DEV), mag) if rot else None
    ctx = ctx_for(ops, DT[dtype], [(3, 5)], None)
    kp, vp = (torch.full((6, G, page, Dp), 7.0, device=DEV, dtype=DT[dtype]) for _ in range(2))
    table = torch.tensor([[5, 2, 4, 1]], dtype=torch.int32, device=DEV)
    q = ops.qkv_conv_rope_store(proj.to(DEV), H, G, D, Dv, Dp, 1, None, None, pos, ctx.token_seq, ctx.query_start_loc, ctx.slot_ids, cs, rot, 1,
                                kp, vp, table, page, True, norm_after=0.01)
    rows = proj.double()

    def turned(x):
        if not rot:
            return x
        out = x.clone()
        for i in range(rot // 2):
            a = torch.arange(3, 8).double() * f[i]
            c, s = (torch.cos(a) * mag)[:, None], (torch.sin(a) * mag)[:, None]
            out[..., i] = x[..., i] * c - x[..., i + rot // 2] * s
            out[..., i + rot // 2] = x[..., i + rot // 2] * c + x[..., i] * s
        return out

    tol = 2e-6 if dtype == "float32" else 6e-3
    q = q.view(T, H, Dp)
    assert rel(q[..., :D], pf.rms(turned(rows[:, :H * D].view(T, H, D)), 0.01)) < tol and (q[..., D:] == 0).all()
    for t in range(T):
        p, s = int(table[0, (3 + t) // page]), (3 + t) % page
        assert rel(kp[p, :, s, :D], pf.rms(turned(rows[:, H * D:(H + G) * D].view(T, G, D)), 0.01)[t]) < tol and (kp[p, :, s, D:] == 0).all()
        assert rel(vp[p, :, s, :Dv], rows[t, (H + G) * D:].view(G, Dv)) < tol and (vp[p, :, s, Dv:] == 0).all()
    only_q = ops.qkv_conv_rope_store(proj[:, :H * D].to(DEV), H, 0, D, Dv, Dp, 1, None, None, pos, ctx.token_seq, ctx.query_start_loc, ctx.slot_ids,
                                     cs, rot, 1, kp, vp, table, page, False, norm_after=0.01)
    assert torch.equal(only_q.view(T, H, Dp), q)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [1, 7, 20, 130, 1100])
@pytest.mark.parametrize("width,ff", [(48, 40), (50, 18), (128, 256)])
def test_gelu_unit_with_biases_alone(ops, dtype, T, width, ff):
    f = dense(ff)
    spec = _ffn(f, "f", width, 9)

    def loud(w):
        for k in w:
            w[k] = w[k] * (6.0 if k.endswith(".b") else 2.0)
    for deferred in (True, False):
        part, w = part_with_weights("ffn", PartSpec(spec.kind, spec.prefix, dict(spec.args, defer_bias=deferred)), dtype, ops, 9, edit=loud)
        x = torch.randn(T, width, generator=torch.Generator().manual_seed(T)).to(DT[dtype])
        y = whole_rows(part.forward(x.to(DEV), None))
        assert (part.out_bias is not None) == deferred
        if deferred:
            y = y + part.out_bias
        exp = pf.dense(x.double(), w, "", f, None)
        assert rel(y, exp) < (2e-5 if dtype == "float32" else 2e-2)
    assert (x.double() @ w["gate"].T + w["gate.b"]).min() < -2           # where gelu and relu, and gelu's two forms of a gate, differ


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [1, 5, 40, 300])
@pytest.mark.parametrize("experts,top", [(5, 2), (1, 1), (4, 4), (40, 7)])
def test_table_experts_alone(ops, dtype, T, experts, top):
    """Experts by the token's id, also where some get no token; the weighted sum in the part and left to the block."""
    f, vocab = moe(24, experts, top), 37
    spec = _ffn(f, "f", 48, vocab)
    toks = torch.randint(0, vocab, (T,), generator=torch.Generator().manual_seed(T)).tolist()
    ctx = ctx_for(ops, DT[dtype], [(0, T)], None, token_ids=toks)
    x = torch.randn(T, 48, generator=torch.Generator().manual_seed(T + 1)).to(DT[dtype])
    for deferred in (True, False):
        part, w = part_with_weights("ffn", PartSpec(spec.kind, spec.prefix, dict(spec.args, defer_combine=deferred)), dtype, ops, 9, scale=0.4)
        y = part.forward(x.to(DEV), ctx)
        if deferred:
            out = torch.zeros(T, 48, device=DEV)
            assert ops.residual_sum(out, None, experts=(y.rows, y.plan, y.top, y.weight)) is None
            y = out
        assert rel(y, pf.table_experts(x.double(), w, "", f, toks)) < (2e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("few", [0, 1, 2])
@pytest.mark.parametrize("T,experts,top,width,ff", [(1, 3, 1, 8, 8), (9, 4, 2, 56, 24), (40, 3, 3, 200, 72), (33, 2, 1, 1032, 136), (70, 20, 5, 128, 40)])
def test_grouped_products_in_every_form(ops, monkeypatch, few, T, experts, top, width, ff):
    """The library's, and weights streamed once for eight or sixteen rows at a time: gated and plain, either output, tiles of a single row
    and of more than sixteen, widths that leave warps without a share of the sum, an activation behind a row's weight."""
    monkeypatch.setattr(ops, "_grouped_few", lambda x, plan: few)
    g = torch.Generator().manual_seed(T)
    r = lambda *s: (torch.randn(s, generator=g) / s[-1] ** 0.5).to(torch.bfloat16)
    w_gu, w_down, x = r(experts, 2 * ff, width), r(experts, width, ff), torch.randn(T, width, generator=g).to(torch.bfloat16)
    table = torch.rand(1, 30, experts, generator=g).argsort(-1)[..., :top].to(torch.int32).contiguous()
    ids = torch.randint(0, 30, (T,), generator=g).to(torch.int32)
    plan = ops.moe_plan_table(table.to(DEV), ids.to(DEV), experts)[0]
    pair = plan["pair_of_pos"].cpu().long()
    tok, ex = pair // top, table[0][ids.long()].reshape(-1)[pair].long()
    gu = torch.einsum("pd,pfd->pf", x.double()[tok], w_gu.double()[ex])
    act = ops.grouped_glu(x.to(DEV), w_gu.to(DEV), plan, top, ff)
    assert rel(act, pf.silu(gu[:, :ff]) * gu[:, ff:]) < 2e-2
    y = torch.einsum("pf,pdf->pd", act.double().cpu(), w_down.double()[ex])
    for out_dtype in (torch.float32, torch.bfloat16):
        assert rel(ops.grouped_linear(act, w_down.to(DEV), plan, out_dtype=out_dtype), y) < 1e-2
    scale = torch.rand(T, top, generator=g)
    up = ops.grouped_act(x.to(DEV), w_gu.to(DEV), plan, top, "relu2", row_scale=scale.to(DEV))
    assert rel(up, torch.relu(gu * scale.reshape(-1)[pair][:, None].double()) ** 2) < 2e-2


@pytest.mark.parametrize("T", [1, 63, 700])
def test_plans_from_tables(ops, T):
    """Three layers' plans in one launch: every pair stands once among its expert's rows; the row tiles cover each expert's rows once."""
    vocab, top, E = 50, 3, 11
    g = torch.Generator().manual_seed(T)
    tables = torch.rand(3, vocab, E, generator=g).argsort(-1)[..., :top].to(torch.int32)
    ids = torch.randint(0, vocab, (T,), generator=g).to(torch.int32)
    for table, plan in zip(tables, ops.moe_plan_table(tables.to(DEV), ids.to(DEV), E)):
        want = table[ids.long()].reshape(-1)
        offs, pos, pair = plan["offsets"].cpu(), plan["pos_of_pair"].cpu(), plan["pair_of_pos"].cpu()
        assert offs.tolist() == [0] + torch.bincount(want, minlength=E).cumsum(0).tolist()
        assert torch.equal(pair[pos.long()], torch.arange(T * top, dtype=torch.int32))
        assert all(offs[e] <= pos[i] < offs[e + 1] for i, e in enumerate(want.tolist()))
        covered = torch.zeros(T * top, dtype=torch.int64)
        for e, first, rows, _ in plan["tiles"].view(-1, 4)[:int(plan["meta"][0])].tolist():
            assert offs[e] <= first and first + rows <= offs[e + 1] and 0 < rows
            covered[first:first + rows] += 1
        assert (covered == 1).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,d", [(9, 64), (9, 50), (9, 1032), (1030, 1032), (600, 1748)])
@pytest.mark.parametrize("kind", ["rows", "parts", "experts", "alone"])
def test_residual_sum(ops, dtype, T, d, kind):
    """x + mult * (a + f + bias) with f as rows, as partial sums, as sorted expert rows (either dtype), or absent."""
    top = 3
    g = torch.Generator().manual_seed(d)
    r = lambda *s: torch.randn(s, generator=g)
    resid, bias = r(T, d), r(d)
    a = r(4, T, d) if kind in ("parts", "alone") else r(T, d).to(DT[dtype])
    for y_dtype in ([DT[dtype], torch.float32] if kind == "experts" else [None]):
        f, experts, extra = None, None, 0.0
        if kind == "rows":
            f = r(T, d).to(DT[dtype]); extra = f.double()
        elif kind == "parts":
            f = r(6, T, d); extra = f.double().sum(0)
        elif kind == "experts":
            pos = torch.randperm(T * top, generator=g).to(torch.int32)
            y = r(T * top, d).to(y_dtype)
            extra = 0.25 * y.double()[pos.long()].view(T, top, d).sum(1)
            experts = (y.to(DEV), {"pos_of_pair": pos.to(DEV)}, top, 0.25)
        want = resid.double() + 0.7 * ((a.double().sum(0) if a.dim() == 3 else a.double()) + extra + bias.double())
        for out_dtype in (None, DT[dtype]):
            x = resid.to(DEV)
            out = ops.residual_sum(x, a.to(DEV), None if f is None else f.to(DEV), experts=experts, bias=bias.to(DEV), mult=0.7, out_dtype=out_dtype)
            assert rel(x, want) < 1e-6
            assert out is None if out_dtype is None else torch.equal(out, x.to(out_dtype))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T", [1, 6, 33, 200])
@pytest.mark.parametrize("width,dim,layer_index", [(72, 1, 0), (72, 10, 2), (50, 13, 1), (512, 64, 1), (48, 8, 2)])
def test_side_input_alone(ops, dtype, T, width, dim, layer_index):
    """The layer's own columns of the token's row; the matrices' padding adds nothing."""
    vocab, layers = 29, 3
    part, w = part_with_weights("ffn", PartSpec("token_gated", "s", {"d_model": width, "dim": dim, "column": layer_index * dim}), dtype, ops, 4, scale=0.3)
    g = torch.Generator().manual_seed(T)
    table = torch.randn(vocab, layers * dim, generator=g).to(DT[dtype])
    toks = torch.randint(0, vocab, (T,), generator=g).tolist()
    x = torch.randn(T, width, generator=g).to(DT[dtype])
    ctx = ctx_for(ops, DT[dtype], [(0, T)], None, token_ids=toks)
    ctx.step_cache[TOKEN_SIDE] = table.to(DEV)
    y = whole_rows(part.forward(x.to(DEV), ctx))
    e = table.double()[toks][:, layer_index * dim:(layer_index + 1) * dim]
    exp = (pf.gelu_tanh(x.double() @ w["gate"].T) * e) @ w["proj"].T
    assert rel(y, exp) < (2e-5 if dtype == "float32" else 2e-2)
    norm = build_part("norm", PartSpec("rmsnorm", "s", {"dim": width, "eps": 1e-3, "name": "norm", "gain": 0.6}))
    after = build_part("norm", PartSpec("rmsnorm", "n", {"dim": width, "eps": 1e-5, "name": "w", "zero_centered": True}))
    wn, wa = torch.rand(width, generator=g) + 0.5, torch.randn(width, generator=g) * 0.3
    for n, k, v in ((norm, "norm", wn), (after, "w", wa)):
        n.bind(ops, DT[dtype], torch.device(DEV))
        n.load({k: v.to(DEV)})
    resid = torch.randn(T, width, generator=g)
    r = resid.to(DEV)
    h = after.add_norm(r, y.to(DT[dtype]), norm)
    want = resid.double() + 0.6 * pf.rms(y.to(DT[dtype]).double().cpu(), 1e-3) * wn.double()
    assert rel(r, want) < 1e-5 and rel(h, pf.norm(want, wa.double(), 1e-5)) < (1e-5 if dtype == "float32" else 1e-2)


def test_pages_are_planned_for_the_longest_reader():
    """A cache whose own layer has short chunks and whose reader has long ones, decoded far: no page the reader needs goes back."""
    cfg = model(90, 48, 1e-5, 3.0, 0.7, 15.0, 6, [
        layer(attn(2, 1, 16, 16, 0.8, chunk=6, rot=8), dense(24)), layer(attn(2, 1, 16, 16, 0.8, chunk=50, rot=8, kv_from=0), moe(12, 5, 2))])
    w = weights_for(cfg, 3)
    reqs = requests(cfg, [130], 1)
    eng = engine_for(cfg, w, "float32", page=4, pages=40)
    check(tu.run_steps(eng, tu.prefill_then_decode(reqs, tail=120)), expected_for(cfg, w, reqs, "float32"), "float32")
    check(tu.run_steps(eng, tu.portions(reqs)), expected_for(cfg, w, reqs, "float32"), "float32")
