"""Small Fokurax configurations for the tests: other sizes, orders, chunks and constants than any model folder that is served."""


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attn(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None, base=1e4, scaling=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling is not None:
            m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(mixer, mlp=None):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, embed_scale, mult, softcap, side, layers):
    return {"architecture": "Fokurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "residual_mult": mult, "logit_softcap": softcap, "token_side": None if side is None else {"dim": side}, "layers": layers}


# both feed-forwards and a layer without one; caches of two layers read by three, one of them beyond another layer's cache and one with
# chunks of its own; value sizes above and below the key size; rescaled frequencies whose ramp lies inside the pairs; different
# scales on one cache
FOK_A = model(131, 64, 1e-5, 4.0, 0.6, 12.0, 10, [
    layer(attn(4, 2, 16, 24, 0.9, chunk=13, rot=8, base=100.0), dense(80)),
    layer(attn(3, 1, 24, 12, 0.7, chunk=29, rot=24, base=50.0, scaling=yarn(4.0, 64, 8.0, 1.0)), moe(20, 5, 2)),
    layer(attn(4, 2, 16, 24, 0.4, chunk=21, rot=8, base=100.0, kv_from=0), moe(36, 7, 3)),
    layer(attn(4, 2, 16, 24, 0.9, chunk=13, rot=8, base=100.0, kv_from=0)),
    layer(attn(3, 1, 24, 12, 1.1, chunk=29, rot=24, base=50.0, scaling=yarn(4.0, 64, 8.0, 1.0), kv_from=1), dense(24))])

# sizes that are multiples of nothing; a kv head per head, one head, a chunk of one key; one expert per token, every expert chosen, a
# single expert; no soft cap; a multiplier of one; one side value
FOK_B = model(97, 50, 3e-4, 1.0, 1.0, None, 1, [
    layer(attn(1, 1, 10, 6, 1.3, chunk=1, rot=2, base=30.0), moe(18, 3, 1)),
    layer(attn(5, 5, 14, 14, 0.5, chunk=5, rot=14, base=1e6), dense(30)),
    layer(attn(3, 3, 6, 30, 0.8, chunk=7, rot=4), moe(14, 4, 4)),
    layer(attn(5, 5, 14, 14, 0.3, chunk=2, rot=14, base=1e6, kv_from=1), moe(10, 1, 1))])

# sizes that the tensor-core attention kernels take, chunks of several pages, five query heads per kv head, many experts
FOK_C = model(120, 128, 1e-6, 8.0, 0.45, 20.0, 40, [
    layer(attn(8, 2, 64, 64, 0.5, chunk=48, rot=64, base=1e5, scaling=yarn(2.0, 128, 16.0, 2.0)), moe(64, 24, 5)),
    layer(attn(8, 2, 64, 64, 0.5, chunk=48, rot=64, base=1e5, scaling=yarn(2.0, 128, 16.0, 2.0), kv_from=0), dense(96)),
    layer(attn(5, 1, 128, 128, 0.3, chunk=70, rot=32, base=1000.0, scaling=yarn(8.0, 32, 4.0, 0.5)), moe(32, 9, 2)),
    layer(attn(2, 2, 32, 48, 0.6, chunk=33, rot=16), moe(48, 4, 3))])

# a layer without a mask, read by one with chunks, and a chunked one read without a mask; no rotation; no input from the token's id;
# sizes named once
FOK_D = model(80, 40, 1e-5, 2.5, 0.8, 8.0, None, [
    layer({"heads": 4, "dim": 20, "scale": 0.9}, dense(44)),
    layer({"heads": 4, "dim": 20, "scale": 0.5, "kv_from": 0, "mask": {"size": 9}}, moe(12, 6, 2)),
    layer(attn(2, 1, 8, 8, 1.0, chunk=6), dense(16)),
    layer(attn(2, 1, 8, 8, 1.0, kv_from=2), moe(12, 6, 2))])

ALL = {"A": FOK_A, "B": FOK_B, "C": FOK_C, "D": FOK_D}
