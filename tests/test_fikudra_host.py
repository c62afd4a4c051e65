"""Host-side tests of the Fikudra design (no GPU): the configuration reader and its refusals, weight loading on the CPU,
and the oracle against second formulations of its own mechanisms."""
import json
import math

import pytest
import torch

from fikudra_common import attn, clean, config_a, config_b, gla, model_cfg, moe, random_checkpoint, tokens


def test_config_reader():
    from compactor_vllm.config.model_config import FikudraConfig

    c = FikudraConfig.from_json(clean(config_a()))
    assert [l.mixer_type for l in c.layers] == ["attention", "gla", "attention", "gla", "attention", "attention", "attention"]
    assert (c.vocab_size, c.hidden_size, c.streams, c.embedding_scale) == (83, 48, 3, 5.0)
    assert (c.buckets, c.mul_prev, c.mul_cur, c.rms_norm_eps) == (61, 29, 7, 1e-5)
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.rot_dims, a.rot_base, a.rot_factor, a.kv_from) == \
        (4, 2, 12, 10, 8, 500.0, 4.0, None)
    assert c.layers[4].mixer.rot_factor == 1.0 and c.layers[2].mixer.kv_from == 0 and c.layers[2].mixer.scale == 0.5
    m = c.layers[3].mixer
    assert (m.heads, m.dim, m.vdim, m.tau) == (2, 22, 7, 3.0)
    assert c.layers[2].mlp is None
    f = c.layers[0].mlp
    assert (f.ff, f.experts, f.top, f.groups, f.keep, f.route_scale, f.shared_ff) == (12, 6, 2, 3, 2, 1.7, 20)
    assert (c.layers[1].mlp.groups, c.layers[1].mlp.keep, c.layers[1].mlp.shared_ff) == (1, 1, 0)
    assert (c.num_key_value_heads, c.num_attention_heads, c.head_dim) == (3, 4, 14)
    assert FikudraConfig.from_json(clean(model_cfg([(gla(), None)]))).num_key_value_heads == 1


def test_config_refusals():
    from compactor_vllm.config.model_config import FikudraConfig

    for layers in ([({"type": "conv", "mixer": {}}, None)], [(attn(4, 3), None)], [(attn(rot=5), None)],
                   [(attn(rot=14), None)], [(gla(tau=0.0), None)], [(gla(), {"kind": "dense", "ff": 8})],
                   [(gla(), moe(6, 2, groups=4))], [(gla(), moe(6, 3, groups=3, keep=1))], [(gla(), moe(4, 5, groups=0))],
                   [(attn(kv_from=0), None)], [(attn(), None), (attn(kv_from=2), None)],
                   [(gla(), None), (attn(kv_from=0), None)], [(attn(), None), (attn(kv_from=0), None), (attn(kv_from=1), None)],
                   [(attn(), None), (attn(base=7.0, kv_from=0), None)], [(attn(), None), (attn(vdim=8, kv_from=0), None)]):
        with pytest.raises(ValueError):
            FikudraConfig.from_json(clean(model_cfg(layers)))
    bad = clean(model_cfg([(gla(), None)]))
    del bad["embedding"]["bigram"]
    with pytest.raises(ValueError):
        FikudraConfig.from_json(bad)


def test_config_is_found_by_its_architecture_name(tmp_path):
    from compactor_vllm.config.model_config import FikudraConfig, load_model_config
    from compactor_vllm.models import MODEL_REGISTRY, registry_key

    (tmp_path / "config.json").write_text(json.dumps(clean(config_a())))
    c = load_model_config(str(tmp_path))
    assert isinstance(c, FikudraConfig) and registry_key(c) == "fikudra"
    assert MODEL_REGISTRY["fikudra"].mixed_steps


def test_weights_land_in_the_joined_products():
    """in_proj rows = everything that reads the mixer's input, then zero rows up to a multiple of 8; a layer that reads
    another layer's cache has queries and gates alone; every other tensor under its own name."""
    from compactor_vllm.config.model_config import FikudraConfig
    from compactor_vllm.models import FikudraForCausalLM

    c = config_a()
    t = random_checkpoint(c, 2)
    m = FikudraForCausalLM(FikudraConfig.from_json(clean(c)))
    m.load_weights(t)
    for i, names in ((0, "qkvg"), (2, "qg"), (1, ["q", "k", "v", "g", "a1"])):
        want = torch.cat([t[f"l{i}.mix.{n}"] for n in names]).float()
        w = m.layers[i].in_proj.weight.float()
        assert w.shape[0] % 8 == 0 and torch.equal(w[:want.shape[0]], want) and not w[want.shape[0]:].any()
    assert m.layers[1].mixer.a2.weight.shape == (36, 5) and m.layers[3].mixer.a2.weight.shape == (44, 3)
    assert torch.equal(m.layers[0].hc2.mix.float(), t["l0.hc2.mix"].float())
    assert torch.equal(m.layers[0].mlp.router[:6].float(), t["l0.mlp.router"].float())
    assert torch.equal(m.layers[0].mlp.router[6:].float(), t["l0.mlp.shared.sg"].float())
    assert m.layers[2].mixer.attn.source is m.layers[0].mixer.attn and m.layers[2].mixer.attn.k_norm_weight is None
    assert [s[1:] for s in m.cache_specs()] == [(2, 12, 10), (3, 14, 6)]
    assert len(m.state_layers()) == 3
    used = sum(p.numel() for p in m.parameters())
    assert sum(v.numel() for v in t.values()) <= used            # nothing of the checkpoint is left out (pads come on top)
    t.pop("l2.hc1.mix")
    with pytest.raises(KeyError):
        m.load_weights(t)
    t["l2.hc1.mix"] = torch.zeros(2, 2)
    with pytest.raises(ValueError):
        m.load_weights(t)


# ------------------------------------------------------------------------------ the oracle's mechanisms a second time
def test_gla_recurrence_as_a_sum_over_earlier_tokens():
    """o_t = sum_(s <= t) (q_t . (prod of the decays after s) k_s) v_s."""
    from oracle import fikudra as O

    g = torch.Generator().manual_seed(1)
    T, H, D, Dv = 9, 2, 5, 4
    q, k = torch.randn(T, H, D, generator=g).double(), torch.randn(T, H, D, generator=g).double()
    v, al = torch.randn(T, H, Dv, generator=g).double(), torch.rand(T, H, D, generator=g).double()
    got = O.gla_recurrence(q, k, v, al)
    want = torch.zeros(T, H, Dv).double()
    for t in range(T):
        for s in range(t + 1):
            decay = al[s + 1:t + 1].prod(dim=0)
            want[t] += (q[t] * decay * k[s]).sum(-1, keepdim=True) * v[s]
    assert torch.allclose(got, want, rtol=1e-10, atol=1e-12)


def test_sink_as_one_more_column_of_score_zero():
    from oracle import fikudra as O

    s = 3 * torch.randn(6, 6, dtype=torch.float64, generator=torch.Generator().manual_seed(2))
    s = s.masked_fill(~torch.ones(6, 6, dtype=torch.bool).tril(), -math.inf)
    want = torch.softmax(torch.cat([s, torch.zeros(6, 1, dtype=torch.float64)], 1), 1)[:, :-1]
    assert torch.allclose(O.sink_softmax(s), want, rtol=1e-12, atol=1e-14)


def test_rotation_is_relative_and_slowed():
    from oracle import fikudra as O

    rot = {"base": 100.0, "dims": 6, "scaling": {"factor": 4.0}}
    g = torch.Generator().manual_seed(3)
    a, b = torch.randn(8, generator=g).double(), torch.randn(8, generator=g).double()
    x, y = O.rotate(a.expand(40, 1, 8), rot)[:, 0], O.rotate(b.expand(40, 1, 8), rot)[:, 0]
    assert torch.equal(x[:, 6:], a[6:].expand(40, 2))
    for d in (0, 3, 11):                                    # a score depends on the distance alone
        diag = torch.diagonal(x @ y.T, offset=-d)
        assert torch.allclose(diag, diag[:1].expand_as(diag), rtol=1e-10, atol=1e-10)
    plain = O.rotate(a.expand(40, 1, 8), {"base": 100.0, "dims": 6})[:, 0]
    assert torch.allclose(x[::4], plain[:10], rtol=1e-12, atol=1e-12)       # position 4 p turns as far as p did
    from compactor_vllm.layers.attention import pair_rotation_frequencies
    f = pair_rotation_frequencies(6, 100.0, linear_factor=4.0)
    assert torch.allclose(f, torch.tensor([100.0 ** (-i / 3) / 4 for i in range(3)], dtype=torch.float64), rtol=1e-14)


def test_routing_by_enumeration():
    """Every pair of groups and every choice inside them: the best sum of the groups' two largest scores, then the best
    `top` scores."""
    from itertools import combinations

    from oracle import fikudra as O

    g = torch.Generator().manual_seed(4)
    router = {"experts": 12, "top": 3, "scale": 2.5, "groups": {"count": 4, "keep": 2}}
    differs = 0
    for _ in range(50):
        s = torch.rand(12, generator=g).tolist()
        rank = [sum(sorted(s[3 * i:3 * i + 3])[-2:]) for i in range(4)]
        pair = max(combinations(range(4), 2), key=lambda c: rank[c[0]] + rank[c[1]])
        allowed = [e for e in range(12) if e // 3 in pair]
        best = max(combinations(allowed, 3), key=lambda c: sum(s[e] for e in c))
        w = O.route_token(s, router)
        assert sorted(w) == sorted(best) and abs(sum(w.values()) - 2.5) < 1e-9
        assert all(abs(w[e] - 2.5 * s[e] / sum(s[i] for i in best)) < 1e-9 for e in best)
        differs += sorted(w) != sorted(sorted(range(12), key=lambda e: -s[e])[:3])
    assert differs > 5


def test_equal_streams_reduce_to_a_plain_residual():
    """Streams that keep to themselves (identity mix), read as their mean and all written alike stay equal, and each is
    the plain residual sum."""
    from oracle import fikudra as O

    g = torch.Generator().manual_seed(5)
    x = torch.randn(4, 7, generator=g).double()
    y = torch.randn(4, 7, generator=g).double()
    xs = O.streams_write([x, x, x], torch.eye(3), torch.ones(3), y)
    assert all(torch.allclose(s, x + y) for s in xs)
    assert torch.allclose(O.streams_read(xs, torch.full((3,), 1 / 3)), x + y, rtol=1e-6)
    mix = torch.tensor([[0.0, 1.0], [0.0, 0.0]])        # from stream 0 to stream 1
    out = O.streams_write([x, y], mix, torch.zeros(2), y)
    assert torch.equal(out[0], torch.zeros_like(x)) and torch.equal(out[1], x)


def test_one_layer_rebuilt_from_its_parts():
    from oracle import fikudra as O

    cfg = model_cfg([(attn(4, 2, 12, 10, rot=8), moe(6, 2, 12, 20, 3, 2))])
    t = random_checkpoint(cfg, 5)
    toks, got = tokens(9, 83, 1), []
    logits = O.forward(clean(cfg), t, toks, got)
    rows = [61] + [(a * 29 + b * 7) % 61 for a, b in zip(toks[:-1], toks[1:])]
    x0 = t["embed"].double()[torch.tensor(toks)] * 5.0 + t["bigram"].double()[torch.tensor(rows)]
    X = x0.unsqueeze(1).repeat(1, 3, 1)                                                  # [T, S, W]

    def normed(u, w):
        return u / (u.pow(2).mean(-1, keepdim=True) + 1e-5).sqrt() * (1 + w.double())

    for tag in ("1", "2"):
        hc = {n: t[f"l0.hc{tag}.{n}"].double() for n in ("in", "mix", "out")}
        h = normed(torch.einsum("s,tsw->tw", hc["in"], X), t[f"l0.norm{tag}"])
        if tag == "1":
            y, _ = O.attention(h, cfg["layers"][0]["mixer"], t, "l0.mix.", 1e-5)
        else:
            y = O.moe_ff(h, cfg["layers"][0]["mlp"], t, "l0.mlp.")
        X = torch.einsum("su,tsw->tuw", hc["mix"], X) + hc["out"][None, :, None] * y[:, None]
    assert torch.allclose(got[0], X.sum(1), rtol=1e-10, atol=1e-10)
    assert torch.allclose(logits, normed(X.sum(1), t["final.norm"]) @ t["head"].double().T, rtol=1e-10, atol=1e-10)
