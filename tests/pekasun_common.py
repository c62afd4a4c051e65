"""Helpers of the Pekasun tests: small configurations, checkpoints with random tensors under the design's names, a
runner that holds them."""
import copy

import torch

from nununex_common import close, feed, new_seq, rel_err, row_errs, run_in_portions, tokens  # noqa: F401


def attn(heads=4, kv_heads=2, dim=12, vdim=10, window=7, keep=3, scale=None):
    mask = {"size": window, "keep_first": keep}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": mask,
                                           "scale": scale or 1.3 * dim ** -0.5}}


def latent(heads=3, dim=10, rot=6, vdim=14, rank=20, window=9, base=300.0, factor=3.0, original=40, fast=4.0, slow=0.5,
           scale=None):
    r = {"base": base, "dims": rot, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": r,
                      "mask": {"size": window}, "scale": scale or 1.2 * (dim + rot) ** -0.5}}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def model_cfg(layers, vocab=83, width=48, eps=1e-5):
    """`layers`: (mixer, feed-forward) pairs, or the index of the layer whose weights this one uses."""
    out = []
    for entry in layers:
        if isinstance(entry, int):
            owner = {k: v for k, v in out[entry].items() if k != "weights_of"}
            out.append(dict(copy.deepcopy(owner), weights_of=entry))
        else:
            out.append(dict(entry[0], mlp=entry[1]))
    return {"architecture": "Pekasun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": copy.deepcopy(out)}


def config_a():
    """Both mixers, layers with and without a feed-forward, two that use another layer's weights (one of them twice
    removed), odd sizes (the kernels' scalar paths)."""
    return model_cfg([
        (latent(3, 10, 6, 14, 20, window=9), dense(40)),
        (attn(4, 2, 12, 10, window=7, keep=3), dense(27)),
        0,
        (attn(3, 3, 7, 5, window=19, keep=1), None),
        1,
        (latent(2, 5, 2, 3, 7, window=23, base=50.0, factor=1.5, original=100, fast=20.0, slow=2.0), None),
        2,
    ])


def config_b():
    """Sizes in multiples of 16: the vector and tensor-core paths of the attention kernels."""
    return model_cfg([
        (attn(4, 2, 32, 32, window=21, keep=5), dense(64)),
        (latent(4, 16, 16, 32, 48, window=33), dense(48)),
        (attn(6, 1, 64, 64, window=40, keep=2), None),
        1,
        (latent(2, 32, 32, 16, 64, window=18), dense(32)),
    ], vocab=96, width=64, eps=1e-6)


def random_checkpoint(cfg: dict, seed: int = 0) -> dict:
    """Every tensor name of the design with random bfloat16 values, for the given config.json dict."""
    W, V = cfg["width"], cfg["vocab"]
    g = torch.Generator().manual_seed(seed)
    t = {}

    def mat(name, *shape, scale=None):
        t[name] = (torch.randn(*shape, generator=g) * (scale if scale is not None else shape[-1] ** -0.5)).to(torch.bfloat16)

    def vec(name, *shape, mean=0.0, spread=0.1):
        t[name] = (mean + spread * torch.randn(shape, generator=g)).to(torch.bfloat16)

    mat("embed", V, W, scale=1.0)
    mat("head", V, W, scale=2.0 * W ** -0.5)
    vec("embed.norm", mean=1.3)
    vec("final.norm", mean=0.8)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        vec(p + "norm1", mean=1.1, spread=0.3)
        q, H = p + "mix.", m["heads"]
        if layer["type"] == "attention":
            G, D, Dv = m["kv_heads"], m["dim"], m["vdim"]
            mat(q + "q", H * D, W); mat(q + "k", G * D, W); mat(q + "v", G * Dv, W)
            vec(q + "q.norm", D, mean=1.2, spread=0.4); vec(q + "k.norm", D, mean=0.9, spread=0.4)
        else:
            D, R, Dv, r = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            mat(q + "q", H * (D + R), W); mat(q + "dkv", r + R, W)
            vec(q + "dkv.norm", r, mean=1.1, spread=0.3)
            mat(q + "uk", H * D, r); mat(q + "uv", H * Dv, r)
            vec(q + "sink", H, spread=1.0)
            mat(q + "g", H * Dv, W)
        mat(q + "o", W, H * m["vdim"])
        if layer.get("mlp"):
            ff, f = layer["mlp"]["ff"], p + "mlp."
            mat(f + "gate", ff, W); mat(f + "up", ff, W); mat(f + "down", W, ff)
    return t


def make_runner(cfg_json, tensors=None, dtype="float32", pages=24, page_size=16, max_seqs=4, seed=0,
                max_batched_tokens=None, device_allocator=False, eager=True):
    """A runner for the configuration; `tensors` (checkpoint names) are loaded over the synthetic weights."""
    from compactor_vllm.config.engine_config import LLMConfig
    from compactor_vllm.config.model_config import PekasunConfig
    from compactor_vllm.core.model_runner import ModelRunner

    cfg = LLMConfig(model="synthetic", hf_config=PekasunConfig.from_json(cfg_json), dtype=dtype, max_num_seqs=max_seqs,
                    kvcache_page_size=page_size, max_model_len=pages * page_size, enforce_eager=eager)
    r = ModelRunner(cfg, num_pages=pages, seed=seed, device_allocator=device_allocator,
                    max_batched_tokens=max_batched_tokens)
    if tensors is not None:
        r.model.load_weights(tensors)
    return r


def build(cfg_json, dtype="float32", seed=0, **kw):
    """(runner, tensors) of a random model."""
    tensors = random_checkpoint(cfg_json, seed)
    return make_runner(cfg_json, tensors, dtype, **kw), tensors
