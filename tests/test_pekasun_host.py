"""Host-side tests of the Pekasun design (no GPU): the configuration reader and its refusals, weight loading on the CPU,
and the oracle against second formulations of its own mechanisms."""
import json
import math

import pytest
import torch

from pekasun_common import attn, config_a, config_b, dense, latent, model_cfg, random_checkpoint, tokens


def test_config_reader():
    from compactor_vllm.config.model_config import PekasunConfig

    c = PekasunConfig.from_json(config_a())
    assert [l.mixer_type for l in c.layers] == ["latent_attention", "attention", "latent_attention", "attention",
                                                "attention", "latent_attention", "latent_attention"]
    assert [l.owner for l in c.layers] == [0, 1, 0, 3, 1, 5, 0]
    assert c.num_hidden_layers == 7 and c.layers[3].mlp is None and c.layers[0].mlp.ff == 40
    a = c.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first) == (4, 2, 12, 10, 7, 3)
    m = c.layers[5].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window) == (2, 5, 2, 3, 7, 23)
    assert (m.rot_base, m.rot_scaling) == (50.0, (1.5, 100.0, 20.0, 2.0))
    assert (c.num_key_value_heads, c.num_attention_heads, c.head_dim, c.rms_norm_eps) == (3, 4, 26, 1e-5)
    only = PekasunConfig.from_json(model_cfg([(latent(), None)]))
    assert only.num_key_value_heads == 1


def test_config_refusals():
    from compactor_vllm.config.model_config import PekasunConfig

    for layers in ([({"type": "conv", "mixer": {}}, None)], [(attn(4, 3), None)], [(attn(window=-1), None)],
                   [(latent(rot=5), None)], [(attn(), {"kind": "moe", "ff": 8})]):
        with pytest.raises(ValueError):
            PekasunConfig.from_json(model_cfg(layers))
    bad = model_cfg([(latent(rot=6), None)])
    bad["layers"][0]["mixer"]["rot"]["dims"] = 4                 # only part of the rotated part
    with pytest.raises(ValueError):
        PekasunConfig.from_json(bad)
    for target in (1, 5, -1):                                    # itself, beyond the end, before the start
        bad = model_cfg([(attn(), None), 0])
        bad["layers"][1]["weights_of"] = target
        with pytest.raises(ValueError):
            PekasunConfig.from_json(bad)
    bad = model_cfg([(attn(), None), 0])
    bad["layers"][1]["mixer"]["mask"] = {"size": 99, "keep_first": 3}     # the rest of the entry must equal the owner's
    with pytest.raises(ValueError):
        PekasunConfig.from_json(bad)


def test_config_is_found_by_its_architecture_name(tmp_path):
    from compactor_vllm.config.model_config import PekasunConfig, load_model_config
    from compactor_vllm.models import MODEL_REGISTRY, registry_key

    (tmp_path / "config.json").write_text(json.dumps(config_a()))
    c = load_model_config(str(tmp_path))
    assert isinstance(c, PekasunConfig) and registry_key(c) == "pekasun"
    assert MODEL_REGISTRY["pekasun"].mixed_steps


def test_weights_land_in_the_joined_products():
    """in_proj rows = the mixer's columns, then gate | up; out_proj columns = W_o, then W_down; shared layers own nothing."""
    from compactor_vllm.config.model_config import PekasunConfig
    from compactor_vllm.models import PekasunForCausalLM

    c = config_b()
    t = random_checkpoint(c, 2)
    m = PekasunForCausalLM(PekasunConfig.from_json(c))
    m.load_weights(t)
    assert sorted(m.layers) == ["0", "1", "2", "4"] and [o for o, _ in m.runs] == ["0", "1", "2", "1", "4"]
    lat = m.layers["1"]
    want = torch.cat([t[f"l1.mix.{n}"] for n in ("q", "dkv", "g")] + [t["l1.mlp.gate"], t["l1.mlp.up"]]).float()
    assert torch.equal(lat.in_proj.weight.float(), want)
    assert torch.equal(lat.out_proj.weight.float(), torch.cat([t["l1.mix.o"], t["l1.mlp.down"]], 1).float())
    assert m.runs[3][1] is not m.runs[1][1] and m.runs[3][1].sink_logits is m.runs[1][1].sink_logits
    specs = m.cache_specs()
    assert [s[1:] for s in specs] == [(2, 32, 32), (1, 64, 0), (1, 64, 64), (1, 64, 0), (1, 96, 0)]


# ------------------------------------------------------------------------------ the oracle's mechanisms a second time
def test_masks_by_enumeration():
    from oracle import pekasun as O

    for size, keep in ((0, 0), (1, 0), (3, 2), (5, 7), (4, 1)):
        seen = O.visible(12, {"size": size, "keep_first": keep})
        for i in range(12):
            for j in range(12):
                want = j <= i and (size == 0 or i - j < size or j < keep)
                assert bool(seen[i, j]) == want


def test_latent_attention_in_the_latent_space():
    """Scores and outputs through q W_uk and the cached latents equal per-head keys and values."""
    from oracle import pekasun as O

    layer = latent(3, 10, 6, 14, 20, 9)
    m = layer["mixer"]
    t = random_checkpoint(model_cfg([(layer, None)]), 4)
    p, eps = "l0.mix.", 1e-5
    h = torch.randn(15, 48, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    want = O.latent_attention(h, m, t, p, eps)
    H, D, R, Dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = O.linear(h, t[p + "q"]).view(15, H, D + R)
    ckr = O.linear(h, t[p + "dkv"])
    c = O.rms_unit(ckr[:, :r], eps) * t[p + "dkv.norm"].double()
    rows = torch.cat([c, O.rotate(ckr[:, r:], m["rot"])], 1)
    uk, uv = t[p + "uk"].double().view(H, D, r), t[p + "uv"].double().view(H, Dv, r)
    heads = []
    for i in range(H):
        qi = torch.cat([q[:, i, :D] @ uk[i], O.rotate(q[:, i, D:], m["rot"])], 1)
        s = (qi @ rows.T * m["scale"]).masked_fill(~O.visible(15, m["mask"]), -math.inf)
        s = torch.cat([s, t[p + "sink"].double()[i].expand(15, 1)], 1)           # the sink as one more column
        heads.append((torch.softmax(s, 1)[:, :-1] @ c) @ uv[i].T)
    o = torch.cat(heads, 1) * torch.sigmoid(O.linear(h, t[p + "g"]))
    assert torch.allclose(O.linear(o, t[p + "o"]), want, rtol=1e-10, atol=1e-12)


def test_rotation_is_relative_and_stretched():
    from oracle import pekasun as O

    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    g = torch.Generator().manual_seed(2)
    a, b = torch.randn(8, generator=g).double(), torch.randn(8, generator=g).double()
    x, y = O.rotate(a.expand(30, 8), rot), O.rotate(b.expand(30, 8), rot)
    dots = x @ y.T
    for d in (0, 3, 11):                                    # a score depends on the distance alone
        diag = torch.diagonal(dots, offset=-d)
        assert torch.allclose(diag, diag[:1].expand_as(diag), rtol=1e-10, atol=1e-10)
    assert torch.allclose(x.norm(dim=1), a.norm() * (0.1 * math.log(4.0) + 1.0) * torch.ones(30).double())
    f, plain = O.frequencies(8, 100.0, rot["scaling"]), O.frequencies(8, 100.0)
    turns = 64 * plain / (2 * math.pi)
    assert torch.equal(f[turns >= 8], plain[turns >= 8]) and f[-1] < plain[-1]
    assert torch.allclose(f[turns < 0.2], plain[turns < 0.2] / 4)
    assert (f <= plain + 1e-15).all() and (f >= plain / 4 - 1e-15).all()


def test_one_layer_rebuilt_from_its_parts():
    from oracle import pekasun as O

    cfg = model_cfg([(attn(4, 2, 12, 10, 7, 3), dense(20)), 0])
    t = random_checkpoint(cfg, 5)
    toks = tokens(9, 83, 1)
    got = []
    logits = O.forward(cfg, t, toks, got)
    e = t["embed"].double()[torch.tensor(toks)]
    x = e / (e.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * t["embed.norm"].double()
    for i in range(2):
        h = x / (x.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * t["l0.norm1"].double()
        gate, up, down = (t[f"l0.mlp.{n}"].double() for n in ("gate", "up", "down"))
        ff = (torch.nn.functional.silu(h @ gate.T) * (h @ up.T)) @ down.T
        x = x + O.attention(h, cfg["layers"][0]["mixer"], t, "l0.mix.", 1e-5) + ff
        assert torch.allclose(got[i], x, rtol=1e-10, atol=1e-10)
    h = x / (x.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * t["final.norm"].double()
    assert torch.allclose(logits, h @ t["head"].double().T, rtol=1e-10, atol=1e-10)
