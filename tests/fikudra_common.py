"""Helpers of the Fikudra tests: small configurations, checkpoints with random tensors under the design's names, a
runner that holds them."""
import json
from pathlib import Path

import torch

from nununex_common import TOL, close, feed, new_seq, rel_err, row_errs, run_in_portions, tokens  # noqa: F401


def gla(heads=3, dim=12, vdim=10, tau=8.0, rank=5):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "_rank": rank}}


def attn(heads=4, kv_heads=2, dim=12, vdim=10, rot=8, base=500.0, factor=4.0, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if factor:
            m["rot"]["scaling"] = {"factor": factor}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def moe(experts=6, top=2, ff=12, shared=20, groups=3, keep=2, scale=1.7):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        m["router"]["groups"] = {"count": groups, "keep": keep}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def model_cfg(layers, vocab=83, width=48, eps=1e-5, streams=3, scale=5.0, buckets=61, mul_prev=29, mul_cur=7):
    """`_rank` (the inner size of a decay projection) is not a key of the design's config.json: the checkpoint's tensors
    carry it; `random_checkpoint` reads it from here."""
    return {"architecture": "Fikudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": [dict(mixer_layer, mlp=mlp) for mixer_layer, mlp in layers]}


def config_a():
    """Both mixers, two layers that read an earlier layer's keys with scales of their own, a layer without a feed-forward;
    odd sizes (the kernels' scalar paths)."""
    return model_cfg([
        (attn(4, 2, 12, 10, rot=8, base=500.0, factor=4.0), moe(6, 2, 12, 20, 3, 2, 1.7)),
        (gla(3, 12, 10, 8.0, 5), moe(5, 3, 10, 0, 0)),
        (attn(4, 2, 12, 10, rot=8, base=500.0, factor=4.0, scale=0.5, kv_from=0), None),
        (gla(2, 22, 7, 3.0, 3), moe(8, 3, 8, 12, 2, 1, 0.6)),
        (attn(3, 3, 14, 6, rot=14, base=30.0, factor=0, scale=0.3), moe(4, 1, 16, 0, 4, 3, 2.0)),
        (attn(3, 3, 14, 6, rot=14, base=30.0, factor=0, scale=0.2, kv_from=4), moe(4, 4, 8, 16, 1, 1, 1.0)),
        (attn(2, 2, 12, 10, rot=8, base=500.0, factor=4.0, scale=0.4, kv_from=0), moe(6, 2, 12, 20, 3, 2, 1.7)),
    ])


def config_b():
    """Sizes in multiples of 16: the vector and tensor-core paths."""
    return model_cfg([
        (gla(2, 32, 32, 16.0, 16), moe(8, 2, 16, 32, 4, 2, 2.5)),
        (attn(4, 2, 32, 16, rot=16, base=10000.0, factor=2.0), moe(8, 2, 16, 32, 4, 2, 2.5)),
        (gla(4, 16, 64, 16.0, 8), moe(8, 3, 24, 16, 2, 1, 1.5)),
        (attn(2, 1, 64, 64, rot=64, base=10000.0, factor=8.0), None),
        (attn(4, 2, 32, 16, rot=16, base=10000.0, factor=2.0, scale=0.25, kv_from=1), moe(8, 2, 16, 32, 4, 2, 2.5)),
    ], vocab=96, width=64, eps=1e-6, streams=4, scale=8.0, buckets=127, mul_prev=1000003, mul_cur=31)


def random_checkpoint(cfg: dict, seed: int = 0) -> dict:
    """Every tensor name of the design with random bfloat16 values, for the given config.json dict."""
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    g = torch.Generator().manual_seed(seed)
    t = {}

    def mat(name, *shape, scale=None):
        t[name] = (torch.randn(*shape, generator=g) * (scale if scale is not None else shape[-1] ** -0.5)).to(torch.bfloat16)

    def vec(name, *shape, mean=0.0, spread=0.1):
        t[name] = (mean + spread * torch.randn(*shape, generator=g)).to(torch.bfloat16)

    mat("embed", V, W, scale=1.0 / cfg["embedding"]["scale"])
    mat("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, W, scale=0.5)
    mat("head", V, W, scale=2.0 * W ** -0.5)
    vec("final.norm", W, spread=0.2)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        for s in ("1", "2") if mlp is not None else ("1",):
            vec(p + "norm" + s, W, spread=0.2)
            vec(p + f"hc{s}.in", S, mean=1.0 / S, spread=0.4)
            vec(p + f"hc{s}.out", S, mean=0.7, spread=0.4)
            t[p + f"hc{s}.mix"] = (0.7 * torch.eye(S) + 0.3 / S * torch.randn(S, S, generator=g) + 0.2 / S).to(torch.bfloat16)
        q = p + "mix."
        if layer["type"] == "gla":
            H, D, Dv, R = m["heads"], m["dim"], m["vdim"], m.get("_rank", 5)
            mat(q + "q", H * D, W); mat(q + "k", H * D, W)
            mat(q + "v", H * Dv, W); mat(q + "g", H * Dv, W)
            mat(q + "a1", R, W)
            mat(q + "a2", H * D, R, scale=1.0)
            vec(q + "a2.b", H * D, mean=1.0, spread=1.0)
            vec(q + "norm", Dv, mean=1.0)
            mat(q + "o", W, H * Dv)
        else:
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mat(q + "q", H * D, W)
            vec(q + "q.norm", H * D, mean=1.0, spread=0.3)
            if m.get("kv_from") is None:
                mat(q + "k", G * D, W); mat(q + "v", G * Dv, W)
                vec(q + "k.norm", G * D, mean=1.0, spread=0.3)
            mat(q + "g", H, W)
            mat(q + "o", W, H * Dv)
        if mlp is None:
            continue
        f, ff = p + "mlp.", mlp["expert"]["ff"]
        mat(f + "router", mlp["router"]["experts"], W, scale=2.0 * W ** -0.5)
        for e in range(mlp["router"]["experts"]):
            mat(f + f"e{e}.gate", ff, W); mat(f + f"e{e}.up", ff, W); mat(f + f"e{e}.down", W, ff)
        if mlp.get("shared"):
            sf = mlp["shared"]["ff"]
            mat(f + "shared.gate", sf, W); mat(f + "shared.up", sf, W); mat(f + "shared.down", W, sf)
            mat(f + "shared.sg", 1, W)
    return t


def clean(cfg: dict) -> dict:
    """The config.json as a checkpoint folder holds it: without the helpers' private keys."""
    c = json.loads(json.dumps(cfg))
    for layer in c["layers"]:
        layer["mixer"].pop("_rank", None)
    return c


def make_runner(cfg_json, tensors=None, dtype="float32", pages=24, page_size=16, max_seqs=4, seed=0,
                max_batched_tokens=None, device_allocator=False, eager=True):
    """A runner for the configuration; `tensors` (checkpoint names) are loaded over the synthetic weights."""
    from compactor_vllm.config.engine_config import LLMConfig
    from compactor_vllm.config.model_config import FikudraConfig
    from compactor_vllm.core.model_runner import ModelRunner

    hf = FikudraConfig.from_json(clean(cfg_json))
    cfg = LLMConfig(model="synthetic", hf_config=hf, dtype=dtype, max_num_seqs=max_seqs, kvcache_page_size=page_size,
                    max_model_len=pages * page_size, enforce_eager=eager)
    r = ModelRunner(cfg, num_pages=pages, seed=seed, device_allocator=device_allocator,
                    max_batched_tokens=max_batched_tokens)
    if tensors is not None:
        r.model.load_weights(tensors)
    return r


def build(cfg_json, dtype="float32", seed=0, **kw):
    """(runner, clean config, tensors) of a random model."""
    tensors = random_checkpoint(cfg_json, seed)
    return make_runner(cfg_json, tensors, dtype, **kw), clean(cfg_json), tensors


def write_checkpoint(folder: Path, cfg: dict, tensors: dict) -> None:
    import nununex_common

    nununex_common.write_checkpoint(folder, clean(cfg), tensors)


def routed_close(got, want, dtype):
    """`close` for models with routed experts.  In bfloat16 a token whose routing is a close call may take another expert
    than in exact arithmetic, which changes its whole row: a few such rows are allowed (random routers have close calls;
    float32 has none)."""
    if dtype == "float32":
        return close(got, want, dtype)
    e = row_errs(got, want).flatten()
    return bool(e.median() < 0.03 and (e > 0.15).sum() <= max(2, 0.08 * e.numel()))
