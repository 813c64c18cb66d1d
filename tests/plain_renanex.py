"""A plain, slow implementation of the Renanex design in float64: whole sequences, no cache, no state carried between calls,
one function per mechanism.  It shares no code with the engine; the tests compare the engine with it.

Notation: ``x`` [S, width] is a sequence's residual stream, ``h`` a sub-layer's input, ``W[name]`` a tensor of the model
folder (matrices are stored [out, in] and applied as ``h @ W.T``), ``m`` a layer's ``mixer`` object of config.json and ``f``
its ``mlp`` object.
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, eps, gain=1.0):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ------------------------------------------------------------------------------------------ linear attention, fixed decays
def lightning(h, W, p, m, eps, shared):
    S = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[p + "q"].T).view(S, H, D)
    k = silu(h @ W[p + "k"].T).view(S, H, D)
    v = silu(h @ W[p + "v"].T).view(S, H, Dv)
    out = torch.zeros(S, H, Dv, dtype=F64)
    for n in range(H):
        state = torch.zeros(D, Dv, dtype=F64)                     # [key channel, value channel]
        for t in range(S):
            state = m["decay"][n] * state + k[t, n][:, None] * v[t, n][None, :]
            out[t, n] = state.T @ q[t, n]
    o = rms_norm(out.reshape(S, H * Dv), eps, W[p + "norm"]) * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ selective scan
def time_conv(u, w, b):
    """u [S, C], w [C, taps], b [C]: out_t = b + sum_j w[:, j] * u_(t - taps + 1 + j), zeros before the first token."""
    S, taps = u.shape[0], w.shape[1]
    out = b.expand(S, -1).clone()
    for t in range(S):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += w[:, j] * u[src]
    return out


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-torch.abs(z)))


def mamba1(h, W, p, m, eps, shared):
    S, I, N, R = h.shape[0], m["inner"], m["state"], m["dt_rank"]
    xz = h @ W[p + "in"].T
    u, z = silu(time_conv(xz[:, :I], W[p + "conv"], W[p + "conv.b"])), xz[:, I:]
    low = u @ W[p + "x"].T
    step = softplus(low[:, :R] @ W[p + "dt"].T + W[p + "dt.b"])
    Bm, Cm = low[:, R:R + N], low[:, R + N:]
    A = -torch.exp(W[p + "A_log"])
    state = torch.zeros(I, N, dtype=F64)
    y = torch.zeros(S, I, dtype=F64)
    for t in range(S):
        state = torch.exp(step[t][:, None] * A) * state + (step[t] * u[t])[:, None] * Bm[t][None, :]
        y[t] = state @ Cm[t] + W[p + "D"] * u[t]
    return (y * silu(z)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ attention
def frequencies(rot):
    """The angle per position of every rotated pair, and what cosine and sine are multiplied by."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def turn(t):
        return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turn(sc["fast"])), 0)
    hi = min(math.ceil(turn(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [S, heads, D]: value i of a head turns with value i + dims/2 by ``position * frequency``, for the first rot.dims values."""
    if not rot or not rot["dims"]:
        return x
    S, half = x.shape[0], rot["dims"] // 2
    f, mag = frequencies(rot)
    out = x.clone()
    for i in range(half):
        angle = torch.arange(S, dtype=F64) * f[i]
        c, s = (torch.cos(angle) * mag)[:, None], (torch.sin(angle) * mag)[:, None]
        out[:, :, i] = x[:, :, i] * c - x[:, :, i + half] * s
        out[:, :, i + half] = x[:, :, i + half] * c + x[:, :, i] * s
    return out


def visible(S, mask):
    """[S, S] bool: row i sees column j <= i if it is one of the last ``size`` or one of the sequence's first ``keep_first``."""
    i = torch.arange(S)[:, None]
    j = torch.arange(S)[None, :]
    ok = j <= i
    if mask is not None:
        ok &= (i - j < mask["size"]) | (j < mask.get("keep_first", 0))
    return ok


def mixed_scores(q, k, talk, scale):
    """q [S, H, D], k [S, G, D] -> [H, S, S]: every query head's products with its kv head's keys, then each head's scores
    replaced by a sum over all heads' with the row's weights of ``talk`` [H, H]."""
    H, G = q.shape[1], k.shape[1]
    raw = torch.stack([q[:, n] @ k[:, n // (H // G)].T * scale for n in range(H)])
    return torch.einsum("hg,gij->hij", talk, raw)


def attention(h, W, p, m, eps, shared):
    S = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, Dv = m.get("kv_heads", H), m.get("vdim", D)
    q = rms_norm(h @ W[p + "q"].T, eps, W[p + "q.norm"])
    k = rms_norm(h @ W[p + "k"].T, eps, W[p + "k.norm"])
    v = h @ W[p + "v"].T
    if m.get("v_mix"):
        if "v_first" not in shared:
            shared["v_first"] = v
        else:
            lam = W[p + "vmix"]
            v = (1.0 - lam) * v + lam * shared["v_first"]
    q, k, v = rotate(q.view(S, H, D), m.get("rot")), rotate(k.view(S, G, D), m.get("rot")), v.view(S, G, Dv)
    s = mixed_scores(q, k, W[p + "talk"], m["scale"])
    s = s.masked_fill(~visible(S, m.get("mask")), float("-inf"))
    w = torch.softmax(s, dim=-1)
    o = torch.cat([w[n] @ v[:, n // (H // G)] for n in range(H)], dim=-1)
    return o @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forward
def dense(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ------------------------------------------------------------------------------------------ the model
MIXERS = {"lightning": lightning, "mamba1": mamba1, "attention": attention}


def forward(config, weights, tokens, after_layer=None):
    """Logits [S, vocab] (float64) of one whole sequence.  ``after_layer(i, x)`` sees the stream behind every layer."""
    W = {k: v.to(F64) for k, v in weights.items() if v.is_floating_point()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    shared = {}
    for i, L in enumerate(config["layers"]):
        p = f"l{i}."
        a = MIXERS[L["type"]](rms_norm(x, eps, W[p + "norm1"]), W, p + "mix.", L["mixer"], eps, shared)
        x = x + rms_norm(a, eps, W[p + "norm1b"])
        if L.get("mlp") is not None:
            x = x + rms_norm(dense(rms_norm(x, eps, W[p + "norm2"]), W, p + "mlp."), eps, W[p + "norm2b"])
        if after_layer is not None:
            after_layer(i, x)
    logits = rms_norm(x, eps, W["final.norm"]) @ W["head"].T * config["logit_scale"]
    cap = config.get("logit_softcap")
    return logits if not cap else cap * torch.tanh(logits / cap)
