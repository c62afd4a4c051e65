"""Prefill and decode throughput of a Fikudra model beside Movolorn, Nununex and Batasun models of equal size with routed
experts (random weights), all through the engine's runner, plus the design's kernels timed alone against the measured peaks
beside the like kernels of the Fafelix design on the same box.

Used by `bench.py --arch fikudra`; the default workload of bench.py does not touch this module.  Movolorn with routed
experts is the closest existing model for the attention layers (the same paged kernels with a sink of score 0,
group-limited routing), Nununex' general-delta layers with routed experts for the recurrent ones.
Timing as in arch_compare: CUDA events on the launching stream after warm-up, a buffer larger than L2 written between
timed kernel iterations; engine-level numbers include the runner's host work.
"""
from __future__ import annotations

import json
from typing import List

import torch

from compactor_vllm.benchmarks.arch_compare import (DECODE_BATCH, DECODE_CONTEXT, DECODE_STEPS, HEAD_DIM, PREFILL_TOKENS,
                                                    SIZES, _events_ms, engine_throughput, movolorn_config)
from compactor_vllm.benchmarks.nununex_compare import nununex_config

GLA_DIM, TAU, STREAMS, RANK = 128, 16.0, 4, 16


def fikudra_config(s: dict, pattern: str, streams: int = STREAMS) -> dict:
    """`pattern`: one letter per layer, cycled over the size's layer count: L gated linear attention, A attention, S
    attention over the keys of the last A layer."""
    W = s["width"]
    # 8 experts of a quarter of the dense size, 2 per token, plus a shared one: about the dense layer's work
    mlp = {"kind": "moe", "expert": {"ff": s["ff"] // 4}, "shared": {"ff": s["ff"] // 2},
           "router": {"experts": 8, "top": 2, "scale": 2.5, "groups": {"count": 2, "keep": 1}}}
    layers, own = [], None
    for i in range(s["layers"]):
        kind = pattern[i % len(pattern)]
        if kind == "L":
            layers.append({"type": "gla", "mlp": mlp, "mixer": {"heads": W // GLA_DIM, "dim": GLA_DIM, "vdim": GLA_DIM,
                                                                "tau": TAU, "decay_rank": RANK}})
            continue
        mixer = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": HEAD_DIM, "vdim": HEAD_DIM,
                 "scale": HEAD_DIM ** -0.5, "rot": {"base": 1e6, "dims": HEAD_DIM, "scaling": {"factor": 8.0}}}
        if kind == "S":
            mixer["kv_from"] = own
        else:
            own = i
        layers.append({"type": "attention", "mlp": mlp, "mixer": mixer})
    return {"architecture": "Fikudra", "vocab": s["vocab"], "width": W, "norm": {"eps": 1e-6}, "streams": streams,
            "embedding": {"scale": 16.0, "bigram": {"buckets": 65521, "mul_prev": 1000003, "mul_cur": 31}},
            "layers": layers}


def kernel_rooflines(peaks: dict, reps: int) -> List[dict]:
    """The design's kernels alone at width 4096, bfloat16: achieved rate and its fraction of the measured copy
    bandwidth / cuBLAS bf16 rate."""
    from compactor_vllm import _native as N
    from compactor_vllm.config.constants import RESERVED_BATCH
    from compactor_vllm.kv_cache.page_table import KVAllocationStatus, PagedKVCache
    from compactor_vllm.layers.attention import BiasedChunkAttention, pair_rotation_frequencies
    from compactor_vllm.layers.latent_attention import group_gate
    from compactor_vllm.layers.layernorm import StreamCoefficients, stream_mix_norm
    from compactor_vllm.layers.moe import ROUTE_SIGMOID_GROUPS, ROUTE_SOFTMAX_ALL, route
    from compactor_vllm.layers.recurrent import GATE_SILU
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

    def add(name, ms, *, nbytes=None, flops=None, fp32_flops=None, like=None):
        r = {"kernel": name, "ms": round(ms, 4), "like": like}
        if nbytes is not None:
            r["GBs"] = round(nbytes / ms / 1e6, 1)
            r["frac_hbm_of_measured"] = round(nbytes / (ms * 1e-3) / hbm, 3)
        if flops is not None:
            r["TFLOPs"] = round(flops / ms / 1e9, 2)
            r["frac_bf16_of_measured"] = round(flops / (ms * 1e-3) / tflops, 4)
        if fp32_flops is not None:
            r["GFLOPs_fp32"] = round(fp32_flops / ms / 1e6, 1)
        rows.append(r)

    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    W, PS, L, B = 4096, 128, 4096, 8
    # --- between two sublayers: the streams read and written (8 S B), the branch (bf16 mixer 2 B, fp32 experts 4 B), the
    #     normed row (2 B)
    w1 = torch.zeros(W, device=dev)
    for S, ydt, yb in ((STREAMS, bf, 2), (STREAMS, torch.float32, 4), (2, bf, 2)):
        x = torch.randn(L, S, W, device=dev)
        y = torch.randn(L, W, device=dev).to(ydt)
        c = StreamCoefficients(S).to(dev)
        add(f"stream_mix_norm, {S} streams, {'bf16' if yb == 2 else 'fp32'} branch (4096 tokens)",
            timed(lambda: stream_mix_norm(x, S, branch=y, coeff=c, dst=x, w_in=c.w_in, weight=w1, gain_offset=1.0, out_dtype=bf)),
            nbytes=(8 * S + yb + 2) * L * W, like="residual_norm")
    del x, y
    # --- attention: norms over the whole projections + rotation + store, portions, decoding, gates
    H, G, D = 32, 8, HEAD_DIM
    attn = BiasedChunkAttention(H, G, D, D, D ** -0.5, sink=True, qk_norm=True, row_norm=True,
                                rotation=pair_rotation_frequencies(D, 1e6, linear_factor=8.0)).to(dev)
    cache = PagedKVCache(1, L // PS + 1, (L // PS + 1) * (B + 1) * G, PS, G, D, B + 1, bf, device=dev, v_head_dim=D)
    attn.k_cache, attn.v_cache, attn.page_table, attn.bh_seq_lens = cache.layer_slices(0)
    attn.page_size = PS
    slots = []
    for _ in range(B):
        s = cache.new_batch()
        assert cache.reserve_tokens(s, L + 1) == KVAllocationStatus.SUCCESS
        slots.append(s)
    attn.k_cache.normal_()
    attn.v_cache.normal_()
    cu, st0, slots1 = i32([0, L]), i32([0]), i32(slots[:1])
    pos_all = torch.arange(L, dtype=torch.int32, device=dev)
    tok_slot = torch.full((L,), slots[0], dtype=torch.int32, device=dev)
    qkv = torch.randn(L, attn.qkv_width + H, device=dev).to(bf)
    q = torch.empty(L, H, D, dtype=bf, device=dev)
    pt = attn.page_table

    def store(T, positions, token_slot, own):
        kv = (N.ptr(attn.k_cache), N.ptr(attn.v_cache)) if own else (None, None)
        N.check(lib.cvllm_row_norm_rope_store(
            N.ptr(qkv), qkv.stride(0), N.ptr(attn.inv_freq), D, N.ptr(attn.q_norm_weight), N.ptr(attn.k_norm_weight), 1e-6,
            N.ptr(positions), N.ptr(token_slot), N.ptr(q), *kv, N.ptr(pt), pt.stride(0), pt.stride(1), PS,
            N.ptr(attn.bh_seq_lens), T, H, G, D, D, RESERVED_BATCH, code, st), "row_norm_rope_store")

    add("row_norm_rope_store (4096 tokens)", timed(lambda: store(L, pos_all, tok_slot, True)),
        nbytes=2 * L * 2 * (H + 2 * G) * D, like="rope_qknorm_store")
    add("row_norm_rope_store, queries alone (4096 tokens)", timed(lambda: store(L, pos_all, tok_slot, False)),
        nbytes=2 * L * 2 * H * D, like="rope_qknorm_store")
    set_context(is_prefill=True, cu_seqlens_q=cu, max_seqlen_q=L, max_seqlen_k=L, batch_mapping=slots1,
                positions_i32=pos_all, token_slot=tok_slot, seq_start=st0)
    q.normal_()
    add("portion attention with a sink (4096 tokens, 32 / 8 heads of 128; tcgen05 pipeline)",
        timed(lambda: attn.attend(q)), flops=4.0 * D * H * L * (L + 1) / 2, like="portion attention with learned sinks")
    posd, slotsB = i32([L - 1] * B), i32(slots)
    set_context(is_prefill=False, batch_mapping=slotsB, positions_i32=posd, token_slot=slotsB, max_seqlen_q=1,
                max_seqlen_k=L)
    qd = torch.randn(B, H, D, device=dev).to(bf)
    add("bias_attn_decode with a sink (8 x 4096 keys)", timed(lambda: attn.attend(qd)),
        nbytes=2 * 2 * B * G * L * D, like="bias_attn_decode with learned sinks")
    reset_context()
    o = torch.randn(L, H * D, device=dev).to(bf)
    add("group_gate, one gate per head, in place (4096 tokens)", timed(lambda: group_gate(o, qkv[:, -H:], out=o)),
        nbytes=2 * 2 * L * H * D, like="sigmoid_gate")
    # --- gated linear attention: decays and scan at two head shapes
    pre, dec = (N.ptr(cu), N.ptr(st0), None), (None, None, N.ptr(posd))
    bm1, bmd = i32([1]), i32(list(range(1, B + 1)))
    for heads, dim in ((W // 64, 64), (W // GLA_DIM, GLA_DIM)):
        HD = heads * dim
        cols = torch.randn(L, 4 * HD + RANK, device=dev).to(bf)
        a2, bias = torch.randn(HD, RANK, device=dev).to(bf), torch.zeros(HD, device=dev)
        alpha = torch.empty(L, HD, device=dev)
        state, nw = torch.zeros(B + 1, heads, dim, dim, device=dev), torch.ones(dim, device=dev)
        out = torch.empty(L, HD, dtype=bf, device=dev)
        a1 = cols[:, 4 * HD:]

        def decay(T):
            N.check(lib.cvllm_lowrank_decay(N.ptr(a1), cols.stride(0), N.ptr(a2), N.ptr(bias), 1.0 / TAU, N.ptr(alpha), HD,
                                            T, HD, RANK, code, st), "lowrank_decay")

        def scan(geom, bm, Bn, mx):
            N.check(lib.cvllm_gla_scan(N.ptr(cols), cols.stride(0), 0, HD, 2 * HD, N.ptr(alpha), HD, dim ** -0.5,
                                       N.ptr(state), 3 * HD, GATE_SILU, N.ptr(nw), 0, 1e-6, *geom, N.ptr(bm), Bn, mx,
                                       N.ptr(out), HD, heads, dim, dim, RESERVED_BATCH, code, st), "gla_scan")

        if dim == GLA_DIM:
            add("lowrank_decay (4096 tokens, 4096 channels, rank 16)", timed(lambda: decay(L)),
                nbytes=4 * L * HD + 2 * L * RANK, like="sigmoid_gate (elementwise)")
        decay(L)
        like = "wkv_scan" if dim == 64 else "delta_rule"
        add(f"gla_scan (one portion of 4096 tokens, {heads} heads of {dim} x {dim}, with the gated norm)",
            timed(lambda: scan(pre, bm1, 1, L)), nbytes=L * HD * 14, fp32_flops=5.0 * dim * dim * heads * L,
            like=f"{like} (the same head shape)")
        add(f"gla_scan (decode, 8 sequences, {heads} heads of {dim} x {dim}: state read + written)",
            timed(lambda: scan(dec, bmd, B, 1)), nbytes=2 * 4 * B * heads * dim * dim, like=f"{like} (decode)")
    # --- routing
    logits = torch.randn(L, 65, device=dev)
    for mode, name in ((ROUTE_SIGMOID_GROUPS, "route, sigmoid groups (4096 tokens, 64 experts, top 8 of 4 / 8 groups)"),
                       (ROUTE_SOFTMAX_ALL, "route, softmax groups (the same; Movolorn's)")):
        add(name, timed(lambda: route(logits, None, 8, 8, 4, mode, 64)), nbytes=4 * L * 65 + 8 * L * 8, like="route")
    return rows


def run(peaks: dict, sizes: List[str], reps: int) -> dict:
    from compactor_vllm.benchmarks import fafelix_compare
    from compactor_vllm.config.model_config import FikudraConfig, MovolornConfig, NununexConfig

    result = {"arch": "fikudra", "closest": "movolorn with routed experts (attention layers), nununex general delta rule with "
                                            "routed experts (recurrent layers)",
              "dtype": "bf16", "data": "synthetic (random weights)",
              "workload": {"prefill_tokens": PREFILL_TOKENS, "decode_batch": DECODE_BATCH,
                           "decode_context": DECODE_CONTEXT, "decode_steps": DECODE_STEPS}, "sizes": {}}
    for name in sizes:
        s = SIZES[name]
        row = {"shape": s}
        row["movolorn_moe"] = engine_throughput("movolorn", MovolornConfig.from_json(movolorn_config(s, 0, True)), reps)
        row["nununex_general_delta_moe"] = engine_throughput("nununex", NununexConfig.from_json(nununex_config(s, "G", True)), reps)
        for label, pattern, streams in (("fikudra_attention_only", "A", STREAMS), ("fikudra_attention_shared_keys", "AS", STREAMS),
                                        ("fikudra_gla_only", "L", STREAMS), ("fikudra_mixed", "LA" if s["layers"] < 4 else "LALS", STREAMS),
                                        ("fikudra_attention_only_one_stream", "A", 1)):
            row[label] = engine_throughput("fikudra", FikudraConfig.from_json(fikudra_config(s, pattern, streams)), reps)
        result["sizes"][name] = row
    result["kernels"] = kernel_rooflines(peaks, max(reps, 5))
    result["like_kernels"] = fafelix_compare.kernel_rooflines(peaks, max(reps, 5))
    result["peaks"] = peaks
    return result


def main(peaks: dict, sizes: str, reps: int) -> None:
    print(json.dumps(run(peaks, [x for x in sizes.split(",") if x], reps)))
