"""Oracle: the Fikudra decoder in plain float64 torch on the CPU, one function per mechanism.

TEST INFRASTRUCTURE ONLY: nothing under compactor-vllm_b200/ imports this module and it imports nothing from
there.  Every function works on one whole sequence (no cache, no state slots, no batching): attention with a dense
score matrix, the recurrence token by token, the experts one token at a time.

The model is given as it is stored: `cfg`, the dict of a config.json, and `tensors`, name -> tensor with the
checkpoint's names (`embed`, `bigram`, `l<i>.norm1|norm2`, `l<i>.hc1|hc2.in|mix|out`, `l<i>.mix.*`, `l<i>.mlp.*`,
`final.norm`, `head`).  Linear weights are [out, in].

    x_1 = .. = x_s = embed[token] * scale + bigram[hash(previous token, token)]         (s parallel streams)
    per layer, for the mixer and then (if the layer has one) the feed-forward:
        u = sum_s in[s] x_s;   y = sublayer(rms_norm(u) * (1 + w))
        x_t <- sum_s mix[s, t] x_s + out[t] y           (all t at once, from the old streams)
    logits = head(rms_norm(sum_s x_s) * (1 + w))
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


def rms_unit(x, eps):
    x = _d(x)
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    return rms_unit(x, eps) * (1.0 + _d(w))


def linear(x, w, b=None):
    y = _d(x) @ _d(w).T
    return y if b is None else y + _d(b)


# ---- embedding ---------------------------------------------------------------------------------------------------
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * mul_prev + int(cur) * mul_cur) % buckets)
    return rows


def embedding(cfg, tensors, tokens):
    e = cfg["embedding"]
    bg = e["bigram"]
    tok = torch.tensor(list(tokens), dtype=torch.long)
    rows = torch.tensor(bigram_rows(list(tokens), bg["buckets"], bg["mul_prev"], bg["mul_cur"]))
    return _d(tensors["embed"])[tok] * e["scale"] + _d(tensors["bigram"])[rows]


# ---- streams -----------------------------------------------------------------------------------------------------
def streams_read(xs, w_in):
    """xs: list of s tensors [T, W] -> sum_s w_in[s] x_s."""
    return sum(_d(w_in)[s] * x for s, x in enumerate(xs))


def streams_write(xs, mix, w_out, y):
    """x_t <- sum_s mix[s, t] x_s + w_out[t] y."""
    mix, w_out = _d(mix), _d(w_out)
    return [sum(mix[s, t] * x for s, x in enumerate(xs)) + w_out[t] * y for t in range(len(xs))]


# ---- mixers ------------------------------------------------------------------------------------------------------
def gla_recurrence(q, k, v, alpha):
    """q, k, alpha [T, H, D], v [T, H, Dv]:  S <- diag(alpha) S + k v^T;  o = S^T q, from a zero state."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    o = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        S = alpha[i].unsqueeze(-1) * S + k[i].unsqueeze(-1) * v[i].unsqueeze(1)
        o[i] = torch.einsum("hkv,hk->hv", S, q[i])
    return o


def gla(h, m, t, p, eps):
    """Gated linear attention: one decay per key channel, alpha = sigmoid(z)^(1 / tau)."""
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = linear(h, t[p + "q"]).view(T, H, D) * D ** -0.5
    k = linear(h, t[p + "k"]).view(T, H, D)
    v = linear(h, t[p + "v"]).view(T, H, Dv)
    z = linear(linear(h, t[p + "a1"]), t[p + "a2"], t[p + "a2.b"]).view(T, H, D)
    alpha = sigmoid(z) ** (1.0 / m["tau"])
    o = rms_unit(gla_recurrence(q, k, v, alpha), eps) * _d(t[p + "norm"])
    return linear(o.reshape(T, H * Dv) * silu(linear(h, t[p + "g"])), t[p + "o"])


def rotate(x, rot):
    """x [T, heads, D]: numbers 2i and 2i + 1 of the first rot.dims turn by position * f_i."""
    if not rot or not rot.get("dims"):
        return x
    dims, x = rot["dims"], x.clone()
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=F64)
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, w = x[:, :, 0:dims:2].clone(), x[:, :, 1:dims:2].clone()
    x[:, :, 0:dims:2] = u * c - w * s
    x[:, :, 1:dims:2] = w * c + u * s
    return x


def sink_softmax(s):
    """Rows of scores (-inf = unseen) -> exp(s) / (1 + sum exp(s))."""
    mx = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - mx)
    return e / (torch.exp(-mx) + e.sum(dim=-1, keepdim=True))


def attention_keys(h, m, t, p, eps):
    """(keys [T, G, D] after norm and rotation, values [T, G, Dv]) of a layer with projections of its own."""
    G, D, Dv = m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    k = rms_unit(linear(h, t[p + "k"]), eps) * _d(t[p + "k.norm"])      # over all heads' rows at once
    return rotate(k.view(T, G, D), m.get("rot")), linear(h, t[p + "v"]).view(T, G, Dv)


def attention(h, m, t, p, eps, kv=None):
    """kv: the (keys, values) of another layer, or None.  Returns (output, the keys and values used)."""
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    T = h.shape[0]
    q = rms_unit(linear(h, t[p + "q"]), eps) * _d(t[p + "q.norm"])
    q = rotate(q.view(T, H, D), m.get("rot"))
    k, v = attention_keys(h, m, t, p, eps) if kv is None else kv
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    seen = torch.ones(T, T, dtype=torch.bool).tril()
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        out[:, hh] = sink_softmax(torch.where(seen, s, torch.full_like(s, -math.inf))) @ v[:, g]
    out = out * sigmoid(linear(h, t[p + "g"])).unsqueeze(-1)            # one gate per head
    return linear(out.reshape(T, -1), t[p + "o"]), (k, v)


# ---- feed-forward ------------------------------------------------------------------------------------------------
def gated_expert(h, t, p):
    return linear(silu(linear(h, t[p + "gate"])) * linear(h, t[p + "up"]), t[p + "down"])


def route_token(s, router):
    """Scores of one token (plain list) -> {expert: weight}."""
    E, top = router["experts"], router["top"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = E // groups["count"]
    rank = [sum(sorted(s[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda g: -rank[g])[:groups["keep"]]
    allowed = [e for e in range(E) if e // size in kept]
    chosen = sorted(allowed, key=lambda e: -s[e])[:top]
    total = sum(s[e] for e in chosen) + 1e-20
    return {e: s[e] / total * router.get("scale", 1.0) for e in chosen}


def moe_ff(h, f, t, p):
    s = sigmoid(linear(h, t[p + "router"]))
    assert s.shape[1] == f["router"]["experts"]
    rows = []
    for i in range(h.shape[0]):
        rows.append(sum(w * gated_expert(h[i:i + 1], t, p + f"e{e}.")[0]
                        for e, w in route_token(s[i].tolist(), f["router"]).items()))
    out = torch.stack(rows)
    if f.get("shared"):
        out = out + gated_expert(h, t, p + "shared.") * sigmoid(linear(h, t[p + "shared.sg"]))
    return out


# ---- the model ---------------------------------------------------------------------------------------------------
def forward(cfg, tensors, tokens, collect=None):
    """Logits [T, vocab] of one whole sequence; `collect` (a list) receives the sum of the streams after every layer."""
    eps = cfg["norm"]["eps"]
    x0 = embedding(cfg, tensors, tokens)
    xs = [x0 for _ in range(cfg["streams"])]
    kept = {}       # layer -> the keys and values it made
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]

        def mixer(h):
            if layer["type"] == "gla":
                return gla(h, m, tensors, p + "mix.", eps)
            src = m.get("kv_from")
            y, kv = attention(h, m, tensors, p + "mix.", eps, None if src is None else kept[src])
            if src is None:
                kept[i] = kv
            return y

        subs = [("1", mixer)]
        if layer.get("mlp") is not None:
            subs.append(("2", lambda h: moe_ff(h, layer["mlp"], tensors, p + "mlp.")))
        for tag, fn in subs:
            hc = p + "hc" + tag + "."
            y = fn(zero_centred_norm(streams_read(xs, tensors[hc + "in"]), tensors[p + "norm" + tag], eps))
            xs = streams_write(xs, tensors[hc + "mix"], tensors[hc + "out"], y)
        if collect is not None:
            collect.append(sum(xs))
    return linear(zero_centred_norm(sum(xs), tensors["final.norm"], eps), tensors["head"])
