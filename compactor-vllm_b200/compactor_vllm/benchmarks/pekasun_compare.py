"""Prefill and decode throughput of a Pekasun model beside a Fafelix and a Batasun model of equal size (random weights),
all through the engine's runner, plus the design's kernels timed alone against the measured peaks.

Used by `bench.py --arch pekasun`; the default workload of bench.py does not touch this module.  Fafelix is the closest
existing model of the attention layers (parallel layers, one input product, a dense feed-forward, the same paged
kernels), Batasun that of the latent-attention layers (the same cached rows; its feed-forward is routed).
Timing as in arch_compare: CUDA events on the launching stream after warm-up, a buffer larger than L2 written between
timed kernel iterations; engine-level numbers include the runner's host work.
"""
from __future__ import annotations

import json
from typing import List

import torch

from compactor_vllm.benchmarks.arch_compare import (DECODE_BATCH, DECODE_CONTEXT, DECODE_STEPS, HEAD_DIM, PREFILL_TOKENS,
                                                    SIZES, _events_ms, engine_throughput)
from compactor_vllm.benchmarks.batasun_compare import LATENT, batasun_config
from compactor_vllm.benchmarks.fafelix_compare import fafelix_config

WINDOW, KEEP = 1024, 4
ROT = {"base": 10000.0, "dims": LATENT["rot_dim"],
       "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
WIDE_RANK = 512        # the latent of the large published latent-attention models, beside the 64 of the comparison


def pekasun_config(s: dict, pattern: str, kv_rank: int = LATENT["kv_rank"], window: int = WINDOW) -> dict:
    """`pattern`: one letter per layer, cycled over the size's layer count: A attention, L latent attention, and = for a
    layer that uses the weights of the layer before it."""
    dense = {"kind": "dense", "ff": s["ff"]}
    layers = []
    for i in range(s["layers"]):
        kind = pattern[i % len(pattern)]
        if kind == "=":
            owner = layers[-1].get("weights_of", i - 1)
            layers.append(dict(layers[-1], weights_of=owner))
        elif kind == "A":
            mixer = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": HEAD_DIM, "vdim": HEAD_DIM,
                     "scale": HEAD_DIM ** -0.5, "mask": {"size": window, "keep_first": KEEP}}
            layers.append({"type": "attention", "mixer": mixer, "mlp": dense})
        else:
            mixer = dict(LATENT, heads=s["heads"], kv_rank=kv_rank, rot=ROT, mask={"size": window},
                         scale=(LATENT["dim"] + LATENT["rot_dim"]) ** -0.5)
            layers.append({"type": "latent_attention", "mixer": mixer, "mlp": dense})
    return {"architecture": "Pekasun", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "layers": layers}


def kernel_rooflines(peaks: dict, reps: int) -> List[dict]:
    """The design's kernels alone at width 4096, bfloat16: achieved rate and its fraction of the measured copy
    bandwidth / cuBLAS bf16 rate."""
    from compactor_vllm import _native as N
    from compactor_vllm.config.constants import RESERVED_BATCH
    from compactor_vllm.kv_cache.page_table import KVAllocationStatus, PagedKVCache
    from compactor_vllm.layers.attention import BiasedChunkAttention, yarn_amplitude, yarn_rotation_frequencies
    from compactor_vllm.layers.latent_attention import DirectLatentAttention, sigmoid_gate
    from compactor_vllm.layers.layernorm import NORM_RMS_ONE_GAIN, embed_norm, residual_norm
    from compactor_vllm.utils.context import reset_context, set_context

    dev = torch.device("cuda", torch.cuda.current_device())
    bf = torch.bfloat16
    flush_buf = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
    hbm = float(peaks["hbm"]) * 1e9
    tflops = float(peaks["tensor_burst"]) * 1e12
    rows: List[dict] = []
    lib, code, st = N.lib(), N.CVLLM_BF16, N.stream(dev)

    def timed(fn):
        def run():
            flush_buf.zero_()
            fn()
        return max(_events_ms(run, reps) - _events_ms(lambda: flush_buf.zero_(), reps), 1e-4)

    def add(name, ms, *, nbytes=None, flops=None, like=None):
        r = {"kernel": name, "ms": round(ms, 4), "like": like}
        if nbytes is not None:
            r["GBs"] = round(nbytes / ms / 1e6, 1)
            r["frac_hbm_of_measured"] = round(nbytes / (ms * 1e-3) / hbm, 3)
        if flops is not None:
            r["TFLOPs"] = round(flops / ms / 1e9, 2)
            r["frac_bf16_of_measured"] = round(flops / (ms * 1e-3) / tflops, 4)
        rows.append(r)

    def i32(v):
        return torch.tensor(v, dtype=torch.int32, device=dev)

    T, W, PS, L, B = 8192, 4096, 128, 4096, 8
    # --- the residual update of a parallel layer: one branch (2 B), the residual read and written (8 B), the normed row
    x = torch.randn(T, W, device=dev)
    y = torch.randn(T, W, device=dev).to(bf)
    one = torch.ones(1, device=dev)
    add("residual_norm (one branch, rms norm with one gain)",
        timed(lambda: residual_norm(x, add=(y,), weight=one, kind=NORM_RMS_ONE_GAIN, out_dtype=bf)), nbytes=12 * T * W,
        like="residual_norm (two branches, layer norm)")
    del x, y
    table = torch.randn(32000, W, device=dev).to(bf)
    ids = torch.randint(0, 32000, (L,), device=dev)
    add("embed_norm (4096 tokens, with the first layer's norm)",
        timed(lambda: embed_norm(ids, table, one, next_weight=one, out_dtype=bf)), nbytes=L * W * (2 + 4 + 2),
        like="pair_hash_embed")
    del table

    def paged(attn, heads, dim, vdim):
        cache = PagedKVCache(1, L // PS + 1, (L // PS + 1) * (B + 1) * heads, PS, heads, dim, B + 1, bf, device=dev,
                             v_head_dim=vdim)
        attn.k_cache, attn.v_cache, attn.page_table, attn.bh_seq_lens = cache.layer_slices(0)
        attn.page_size = PS
        slots = []
        for _ in range(B):
            s = cache.new_batch()
            assert cache.reserve_tokens(s, L + 1) == KVAllocationStatus.SUCCESS
            slots.append(s)
        attn.k_cache.normal_()
        if vdim:
            attn.v_cache.normal_()
        return slots

    pos_all = torch.arange(L, dtype=torch.int32, device=dev)
    seen = sum(min(i + 1, WINDOW) + min(max(i + 1 - WINDOW, 0), KEEP) for i in range(L))   # (query, key) pairs

    def portion(slots):
        set_context(is_prefill=True, cu_seqlens_q=i32([0, L]), max_seqlen_q=L, max_seqlen_k=L, batch_mapping=i32(slots[:1]),
                    positions_i32=pos_all, token_slot=torch.full((L,), slots[0], dtype=torch.int32, device=dev),
                    seq_start=i32([0]))

    def decode(slots):
        set_context(is_prefill=False, batch_mapping=i32(slots), positions_i32=i32([L - 1] * B), token_slot=i32(slots),
                    max_seqlen_q=1, max_seqlen_k=L)

    # --- attention: norms and store, then the windowed portion and decode kernels; 32 / 8 heads of 128
    H, G, D = 32, 8, HEAD_DIM
    prev = torch.get_default_dtype()
    torch.set_default_dtype(bf)
    try:
        with torch.device(dev):
            attn = BiasedChunkAttention(H, G, D, D, D ** -0.5, qk_norm=True, window=WINDOW, keep_first=KEEP,
                                        value_norm=True)
            lat = {r: DirectLatentAttention(
                H, LATENT["dim"], LATENT["rot_dim"], LATENT["vdim"], r, 0.07, 1e-6,
                inv_freq=yarn_rotation_frequencies(ROT["dims"], ROT["base"], 4.0, 4096, 32.0, 1.0).to(dev),
                amplitude=yarn_amplitude(4.0), neighbours=True, window=WINDOW, learned_sink=True, dtype=bf)
                for r in (LATENT["kv_rank"], WIDE_RANK)}
    finally:
        torch.set_default_dtype(prev)
    slots = paged(attn, G, D, D)
    portion(slots)
    qkv = torch.randn(L, attn.qkv_width, device=dev).to(bf)
    q = torch.randn(L, H, D, device=dev).to(bf)
    pt = attn.page_table
    tok = torch.full((L,), slots[0], dtype=torch.int32, device=dev)

    def store():
        N.check(lib.cvllm_rope_qknorm_store(N.ptr(qkv), qkv.stride(0), None, 0, 3, N.ptr(attn.q_norm_weight),
                                            N.ptr(attn.k_norm_weight), 1e-6, N.ptr(pos_all), N.ptr(tok), N.ptr(q),
                                            N.ptr(attn.k_cache), N.ptr(attn.v_cache), N.ptr(pt), pt.stride(0), pt.stride(1),
                                            PS, N.ptr(attn.bh_seq_lens), L, H, G, D, D, RESERVED_BATCH, code, st), "store")

    add("q / k / v norms + store (4096 tokens)", timed(store), nbytes=2 * L * 2 * (H + 2 * G) * D,
        like="rope_qknorm_store")
    add(f"portion attention, window {WINDOW} + {KEEP} first tokens (4096 tokens, 32 / 8 heads of 128; tcgen05)",
        timed(lambda: attn.attend(q)), flops=4.0 * D * H * seen, like="prefill_attn_bias, chunk 1024")
    N.set_test_option("bias_attn_fma", 2)
    add("portion attention (the same on the mma.sync kernel)", timed(lambda: attn.attend(q)), flops=4.0 * D * H * seen,
        like="bias_attn_varlen_mma")
    N.set_test_option("bias_attn_fma", 0)
    decode(slots)
    qd = torch.randn(B, H, D, device=dev).to(bf)
    add(f"bias_attn_decode, window {WINDOW} + {KEEP} first tokens (8 sequences)", timed(lambda: attn.attend(qd)),
        nbytes=2 * 2 * B * G * (WINDOW + KEEP) * D, like="bias_attn_decode, chunk 1024")
    reset_context()
    # --- latent attention: 32 heads over rows of 64 + 64 numbers, and over rows of 512 + 64
    seen_l = sum(min(i + 1, WINDOW) for i in range(L))
    for r, la in lat.items():
        slots = paged(la.attn, 1, la.row, 0)
        with torch.no_grad():
            la.uk.normal_(0, 0.1)
            la.uv.normal_(0, 0.1)
        portion(slots)
        tok = torch.full((L,), slots[0], dtype=torch.int32, device=dev)
        cols = torch.randn(L, la.in_cols, device=dev).to(bf)
        q_full = torch.randn(L, H, la.row, device=dev).to(bf)
        lpt = la.attn.page_table

        def prepare():
            N.check(lib.cvllm_latent_prepare(
                N.ptr(cols), cols.stride(0), 0, H, la.dim, H * (la.dim + la.rot_dim), r, la.rot_dim, N.ptr(la.kv_norm), 1e-6,
                N.ptr(la.inv_freq), la.amplitude, 1, N.ptr(pos_all), N.ptr(tok), N.ptr(q_full), q_full.stride(0), la.row, r,
                N.ptr(la.attn.k_cache), N.ptr(lpt), lpt.stride(0), PS, N.ptr(la.attn.bh_seq_lens), L, RESERVED_BATCH, code,
                st), "prepare")

        add(f"latent_prepare (4096 tokens, 32 heads, latent of {r})", timed(prepare),
            nbytes=2 * L * 2 * (H * la.rot_dim + la.row), like="latent_q_rope")
        add(f"portion attention, latent rows of {r} + 64, window {WINDOW}, sinks (4096 tokens, 32 heads)",
            timed(lambda: la.attn.attend(q_full, flat=False)), flops=2.0 * (la.row + r) * H * seen_l,
            like="portion attention, values in keys")
        if r == LATENT["kv_rank"]:
            o = torch.randn(L, H * la.vdim, device=dev).to(bf)
            wide = torch.empty(L, H * la.vdim + 14336, dtype=bf, device=dev)
            add("sigmoid_gate into a wider row (4096 x 4096)",
                timed(lambda: sigmoid_gate(o, cols[:, la.in_cols - H * la.vdim:], wide[:, :H * la.vdim])),
                nbytes=6 * L * H * la.vdim, like="sigmoid_gate")
            del o, wide
        decode(slots)
        qd = torch.randn(B, H, la.row, device=dev).to(bf)
        add(f"bias_attn_decode, latent rows of {r} + 64, window {WINDOW}, sinks (8 sequences)",
            timed(lambda: la.attn.attend(qd, flat=False)), nbytes=2 * B * WINDOW * la.row,
            like="bias_attn_decode, values in keys")
        rows[-1]["G_head_keys_per_s"] = round(B * H * WINDOW / rows[-1]["ms"] / 1e6, 2)
        reset_context()
    return rows


def run(peaks: dict, sizes: List[str], reps: int) -> dict:
    from compactor_vllm.config.model_config import BatasunConfig, FafelixConfig, PekasunConfig

    result = {"arch": "pekasun", "closest": "fafelix (parallel layers, dense feed-forward) for the attention layers; "
                                            "batasun (routed experts) for the latent-attention layers",
              "dtype": "bf16", "data": "synthetic (random weights)",
              "workload": {"prefill_tokens": PREFILL_TOKENS, "decode_batch": DECODE_BATCH,
                           "decode_context": DECODE_CONTEXT, "decode_steps": DECODE_STEPS, "window": WINDOW,
                           "keep_first": KEEP}, "sizes": {}}
    for name in sizes:
        s = SIZES[name]
        row = {"shape": s}
        row["fafelix_attention_only"] = engine_throughput("fafelix", FafelixConfig.from_json(fafelix_config(s, "A")), reps)
        row["batasun_latent_only"] = engine_throughput("batasun", BatasunConfig.from_json(batasun_config(s, "A")), reps)
        for label, pattern, rank, window in (
                ("pekasun_attention_only", "A", LATENT["kv_rank"], WINDOW),
                ("pekasun_attention_only_no_window", "A", LATENT["kv_rank"], 0),
                ("pekasun_latent_only", "L", LATENT["kv_rank"], WINDOW),
                ("pekasun_mixed_shared_weights", "LA=L", LATENT["kv_rank"], WINDOW),
                ("pekasun_latent_only_rank_512", "L", WIDE_RANK, WINDOW)):
            row[label] = engine_throughput("pekasun", PekasunConfig.from_json(pekasun_config(s, pattern, rank, window)), reps)
        result["sizes"][name] = row
    result["kernels"] = kernel_rooflines(peaks, max(reps, 5))
    result["peaks"] = peaks
    return result


def main(peaks: dict, sizes: str, reps: int) -> None:
    print(json.dumps(run(peaks, [x for x in sizes.split(",") if x], reps)))
