"""Small Renanex configurations for the tests: other sizes, orders, windows and constants than any model folder that is served."""


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def lightning(heads, dim, vdim, decay):
    assert len(decay) == heads
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def mamba(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def attn(heads, kv_heads, dim, vdim, scale, window=None, keep=None, rot=None, scaling=None, base=1e4, v_mix=False):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if window is not None:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling is not None:
            m["rot"]["scaling"] = scaling
    return m


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, eps, logit_scale, softcap, layers):
    cfg = {"architecture": "Renanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}
    if softcap is not None:
        cfg["logit_softcap"] = softcap
    return cfg


# every mixer; grouped heads; a window that is a multiple of nothing and keeps three tokens; part of a head rotated; value sizes above
# and below the key size; rescaled frequencies whose ramp lies inside the pairs; a layer without a feed-forward; values mixed in
# two layers and left alone in one between them
REN_A = model(131, 64, 1e-5, 1.5, 12.0, [
    layer("attention", attn(4, 2, 16, 24, 0.3, window=13, keep=3, rot=8, base=100.0, v_mix=True), 80),
    layer("mamba1", mamba(72, 10, 5, 4), 48),
    layer("lightning", lightning(3, 12, 20, [0.3, 0.9, 0.99])),
    layer("attention", attn(3, 1, 24, 12, 0.25, window=29, keep=6, rot=24, base=50.0, scaling=yarn(4.0, 64, 8.0, 1.0)), 40),
    layer("attention", attn(6, 3, 12, 16, 0.35, window=8, keep=1, rot=12, v_mix=True), 96)])

# sizes that are multiples of nothing; one kv head per head; a window of one key; no kept tokens; one tap (no state of its own); one
# state per channel; a single head; a decay of zero and one of one; no soft cap
REN_B = model(97, 50, 3e-4, 0.7, None, [
    layer("lightning", lightning(1, 10, 14, [0.0]), 30),
    layer("attention", attn(3, 3, 10, 10, 0.4, window=1, rot=10, base=30.0, v_mix=True), 18),
    layer("mamba1", mamba(54, 1, 3, 1), 30),
    layer("attention", attn(5, 1, 14, 6, 0.3, window=5, keep=0, rot=2, base=1e6)),
    layer("mamba1", mamba(30, 7, 11, 2)),
    layer("attention", attn(1, 1, 6, 30, 0.5, window=7, keep=9, v_mix=True), 22),
    layer("lightning", lightning(2, 6, 6, [1.0, 0.5]), 30)])

# sizes the tensor-core attention kernels take (joint rows of 64, 128 and 256 values), windows of several pages, many states
REN_C = model(120, 128, 1e-6, 1.0, 20.0, [
    layer("mamba1", mamba(256, 40, 16, 3), 128),
    layer("attention", attn(8, 2, 64, 64, 0.125, window=48, keep=5, rot=16, base=1000.0, v_mix=True), 64),
    layer("lightning", lightning(4, 64, 32, [0.5, 0.9, 0.98, 0.998])),
    layer("attention", attn(4, 4, 64, 32, 0.12, window=70, keep=20, rot=64, base=1e5, scaling=yarn(2.0, 128, 16.0, 2.0), v_mix=True), 64),
    layer("attention", attn(4, 1, 64, 64, 0.12, window=33, keep=4, rot=32), 64)])

# an attention layer without a mask and without a rotation; a joint row of more than 256 values; kept tokens that outreach the window;
# keys and values of one size named once
REN_D = model(80, 40, 1e-5, 2.5, 8.0, [
    layer("attention", {"heads": 8, "dim": 40, "scale": 0.16, "v_mix": True}, 44),
    layer("attention", attn(4, 2, 20, 160, 0.2, window=4, keep=17, rot=4, base=250.0, v_mix=True), 16),
    layer("lightning", lightning(2, 24, 8, [0.8, 0.95]), 16),
    layer("mamba1", mamba(20, 3, 1, 6))])

# no attention at all, and the recurrences in another order
REN_E = model(64, 48, 1e-5, 1.0, 5.0, [
    layer("lightning", lightning(4, 8, 16, [0.2, 0.7, 0.9, 0.97]), 24),
    layer("mamba1", mamba(96, 16, 8, 4), 24),
    layer("lightning", lightning(2, 16, 8, [0.99, 0.5]))])

ALL = {"A": REN_A, "B": REN_B, "C": REN_C, "D": REN_D, "E": REN_E}
