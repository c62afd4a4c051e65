"""Oracle: the Pekasun decoder in plain float64 torch on the CPU, one function per mechanism.

TEST INFRASTRUCTURE ONLY: nothing under compactor-vllm_b200/ imports this module and it imports nothing from
there.  Every function works on one whole sequence (no cache, no batching): attention with a dense score matrix and a
mask built from the positions, latent attention with per-head keys and values built from the latent.

The model is given as it is stored: `cfg`, the dict of a config.json, and `tensors`, name -> tensor with the
checkpoint's names (`embed`, `embed.norm`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`).  Linear
weights are [out, in]; the gain of every norm of the stream is ONE number.

    x = norm(embed[token]);   per layer:  h = norm(x),  x += mixer(h) + ff(h);   logits = head(norm(x))
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def _d(x):
    return x.to(F64)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def linear(x, w):
    return _d(x) @ _d(w).T


def rms_unit(x, eps):
    """x over its root mean square along the last dimension."""
    x = _d(x)
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    """RMS norm whose gain is one number for all coordinates."""
    return rms_unit(x, eps) * _d(gain).reshape(())


# ---- masks -------------------------------------------------------------------------------------------------------
def visible(T, mask):
    """[T, T] bool: query i (row) sees key j.  `mask`: `size` positions back from the query (itself included; 0 or
    absent: all) and, whatever their distance, the sequence's first `keep_first` positions."""
    mask = mask or {}
    size, keep = int(mask.get("size", 0) or 0), int(mask.get("keep_first", 0) or 0)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size:
        seen = seen & ((i - j < size) | (j < keep))
    return seen


def attend(q, k, v, scale, seen, sink=None):
    """q, k [T, D], v [T, Dv] of one head -> [T, Dv].  A sink is one more term exp(sink) of the denominator."""
    s = (q @ k.T) * scale
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    mx = s.max(dim=1, keepdim=True).values
    if sink is not None:
        mx = torch.maximum(mx, sink)
    e = torch.exp(s - mx)
    den = e.sum(dim=1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - mx)
    return (e / den) @ v


# ---- rotation ----------------------------------------------------------------------------------------------------
def frequencies(dims, base, scaling=None):
    """dims / 2 angular frequencies.  `scaling`: pairs that turn fast over `original` positions keep their frequency,
    slow ones are divided by `factor`, with a linear ramp over the pair index between the two."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            def index_of(turns):
                return dims * math.log(scaling["original"] / (turns * 2 * math.pi)) / (2 * math.log(base))

            lo = max(math.floor(index_of(scaling["fast"])), 0)
            hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / scaling["factor"] * ramp + f * (1.0 - ramp)
        out.append(f)
    return torch.tensor(out, dtype=F64)


def amplitude(scaling):
    return 0.1 * math.log(scaling["factor"]) + 1.0 if scaling else 1.0


def rotate(x, rot):
    """x [T, ..., dims]: neighbours (2i, 2i + 1) turn by position * f_i; the result times the amplitude."""
    T, dims = x.shape[0], x.shape[-1]
    sc = rot.get("scaling")
    a = torch.arange(T, dtype=F64)[:, None] * frequencies(dims, float(rot["base"]), sc)[None, :]
    c, s = torch.cos(a) * amplitude(sc), torch.sin(a) * amplitude(sc)
    shape = [T] + [1] * (x.dim() - 2) + [dims // 2]
    c, s = c.view(shape), s.view(shape)
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


# ---- mixers ------------------------------------------------------------------------------------------------------
def attention(h, m, t, p, eps):
    """Grouped heads, q and k normed with a weight, values normed without one, window plus kept first tokens."""
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = rms_unit(linear(h, t[p + "q"]).view(T, H, D), eps) * _d(t[p + "q.norm"])
    k = rms_unit(linear(h, t[p + "k"]).view(T, G, D), eps) * _d(t[p + "k.norm"])
    v = rms_unit(linear(h, t[p + "v"]).view(T, G, Dv), eps)
    seen = visible(T, m.get("mask"))
    out = torch.stack([attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], seen) for i in range(H)], 1)
    return linear(out.reshape(T, H * Dv), t[p + "o"])


def latent_attention(h, m, t, p, eps):
    """Keys and values of every head from one latent row per token plus a rotated key part shared by the heads."""
    H, D, R, Dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = linear(h, t[p + "q"]).view(T, H, D + R)
    ckr = linear(h, t[p + "dkv"])
    c = rms_unit(ckr[:, :r], eps) * _d(t[p + "dkv.norm"])
    kr = rotate(ckr[:, r:], m["rot"])
    qr = rotate(q[..., D:], m["rot"])
    k = linear(c, t[p + "uk"]).view(T, H, D)
    v = linear(c, t[p + "uv"]).view(T, H, Dv)
    seen = visible(T, m.get("mask"))
    sink = _d(t[p + "sink"])
    heads = []
    for i in range(H):
        qi = torch.cat([q[:, i, :D], qr[:, i]], dim=-1)
        ki = torch.cat([k[:, i], kr], dim=-1)
        heads.append(attend(qi, ki, v[:, i], m["scale"], seen, sink[i]))
    out = torch.stack(heads, 1).reshape(T, H * Dv) * sigmoid(linear(h, t[p + "g"]))
    return linear(out, t[p + "o"])


def feed_forward(h, t, p):
    return linear(silu(linear(h, t[p + "gate"])) * linear(h, t[p + "up"]), t[p + "down"])


MIXERS = {"attention": attention, "latent_attention": latent_attention}


def forward(cfg, tensors, tokens, collect=None):
    """Logits [T, vocab] of one whole sequence; `collect` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = scalar_norm(_d(tensors["embed"])[torch.tensor(list(tokens), dtype=torch.long)], tensors["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        owner = i
        while cfg["layers"][owner].get("weights_of") is not None:
            owner = cfg["layers"][owner]["weights_of"]
        p = f"l{owner}."
        h = scalar_norm(x, tensors[p + "norm1"], eps)
        y = MIXERS[layer["type"]](h, layer["mixer"], tensors, p + "mix.", eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, tensors, p + "mlp.")
        x = x + y
        if collect is not None:
            collect.append(x.clone())
    return linear(scalar_norm(x, tensors["final.norm"], eps), tensors["head"])
