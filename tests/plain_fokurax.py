"""A plain, slow implementation of the Fokurax design in float64: whole sequences, no cache, one function per mechanism.  It shares
no code with the engine; the tests compare the engine with it.

Notation: ``x`` [S, width] is a sequence's residual stream, ``h`` its normed rows (what both sub-layers of a layer read),
``W[name]`` a tensor of the model folder (matrices are stored [out, in] and applied as ``h @ W.T``), ``m`` a layer's ``mixer`` object
of config.json and ``f`` its ``mlp`` object.
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x over its root mean square (last dimension)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """The model's norm: the weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


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
    """[S, S] bool: row i sees column j <= i of its own chunk of ``size`` positions (no mask: every j <= i)."""
    i = torch.arange(S)[:, None]
    j = torch.arange(S)[None, :]
    ok = j <= i
    if mask is not None:
        ok &= (i // mask["size"]) == (j // mask["size"])
    return ok


def keys_values(h, W, p, m, eps):
    """The layer's own keys (rotated, then normed without a weight) and values, [S, kv heads, size]."""
    S, G, D = h.shape[0], m.get("kv_heads", m["heads"]), m["dim"]
    k = rms(rotate((h @ W[p + "k"].T).view(S, G, D), m.get("rot")), eps)
    return k, (h @ W[p + "v"].T).view(S, G, m.get("vdim", D))


def attention(h, W, p, m, eps, kv):
    S, H, D = h.shape[0], m["heads"], m["dim"]
    k, v = kv
    G = k.shape[1]
    q = rms(rotate((h @ W[p + "q"].T).view(S, H, D), m.get("rot")), eps)
    heads = []
    for n in range(H):
        s = q[:, n] @ k[:, n // (H // G)].T * m["scale"]
        s = s.masked_fill(~visible(S, m.get("mask")), float("-inf"))
        heads.append(torch.softmax(s, dim=-1) @ v[:, n // (H // G)])
    return torch.cat(heads, dim=-1) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forwards
def dense(h, W, p, f, tokens):
    g = gelu_tanh(h @ W[p + "gate"].T + W[p + "gate.b"])
    return (g * (h @ W[p + "up"].T + W[p + "up.b"])) @ W[p + "down"].T + W[p + "down.b"]


def table_experts(h, W, p, f, tokens):
    """Each token's experts stand in the table's row of its id; their outputs are averaged."""
    out = torch.zeros_like(h)
    top = f["router"]["top"]
    for t, tok in enumerate(tokens):
        for e in W[p + "table"][tok].tolist():
            q = f"{p}e{e}."
            y = (silu(h[t] @ W[q + "gate"].T) * (h[t] @ W[q + "up"].T)) @ W[q + "down"].T
            out[t] += y / top
    return out


FEED_FORWARDS = {"dense": dense, "moe": table_experts}


# ------------------------------------------------------------------------------------------ what a token adds to every layer
def side_input(x, W, p, i, dim, tokens, eps):
    e = W["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return rms(y, eps) * W[p + "side.norm"]


# ------------------------------------------------------------------------------------------ the model
def forward(config, weights, tokens, after_layer=None):
    """Logits [S, vocab] (float64) of one whole sequence.  ``after_layer(i, x)`` sees the stream behind every layer."""
    W = {k: (v.to(F64) if v.is_floating_point() else v.long()) for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = W["embed"][tokens] * config["embedding"]["scale"]
    stored = {}                                                    # layer -> its keys and values
    for i, L in enumerate(config["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        h = norm(x, W[p + "norm1"], eps)
        source = m.get("kv_from")
        if source is None:
            source = i
            stored[i] = keys_values(h, W, p + "mix.", m, eps)
        y = attention(h, W, p + "mix.", m, eps, stored[source])
        if f is not None:
            y = y + FEED_FORWARDS[f["kind"]](h, W, p + "mlp.", f, tokens)
        x = x + mult * y
        if config.get("token_side"):
            x = x + mult * side_input(x, W, p, i, config["token_side"]["dim"], tokens, eps)
        if after_layer is not None:
            after_layer(i, x)
    logits = norm(x, W["final.norm"], eps) @ W["head"].T
    cap = config.get("logit_softcap")
    return logits if not cap else cap * torch.tanh(logits / cap)
