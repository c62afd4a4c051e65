"""Pekasun through the engine against the plain CPU oracle (oracle/pekasun.py).

Every test makes its own small configuration and random weights (checkpoint tensors under the design's names, loaded
by the model's `load_weights`).  The engine runs them through its runner (`ModelRunner.run_step`, the paged cache, the
native kernels); the oracle recomputes whole sequences without a cache.  float32 runs are compared sharply (they show a
key that is one position off or a missing sink), bfloat16 loosely; the attention kernels that only serve bfloat16 are
compared with a dense softmax on the same rounded rows, with keys planted so that one that is wrongly seen or wrongly
hidden decides the result."""
import math

import pytest
import torch

from pekasun_common import (attn, build, close, config_a, config_b, dense, feed, latent, make_runner, model_cfg, new_seq,
                            random_checkpoint, rel_err, run_in_portions, tokens)

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0) if torch.cuda.is_available() else None
TOL = 3e-5       # float32


# ------------------------------------------------------------------------------------------ mechanisms one by one
@pytest.mark.parametrize("width", [1, 40, 257, 1024])
def test_norms_with_one_gain(width):
    from compactor_vllm.layers.layernorm import NORM_RMS_ONE_GAIN, embed_norm, residual_norm
    from oracle import pekasun as O

    g = torch.Generator().manual_seed(1)
    w0, w1 = torch.tensor([1.7]), torch.tensor([-0.6])
    table = torch.randn(31, width, generator=g) * 2
    ids = torch.tensor([3, 30, 0, 3, 17])
    for dt in (torch.float32, torch.bfloat16):
        tab = table.to(dt)
        x, h = embed_norm(ids.to(DEV), tab.to(DEV), w0.to(DEV), next_weight=w1.to(DEV), eps=1e-3, out_dtype=torch.float32)
        want = O.scalar_norm(tab.double()[ids], w0, 1e-3)
        assert torch.allclose(x.cpu().double(), want, rtol=1e-5, atol=1e-6)
        assert torch.allclose(h.cpu().double(), O.scalar_norm(want, w1, 1e-3), rtol=1e-5, atol=1e-6)
        x2, none = embed_norm(ids.to(DEV), tab.to(DEV), w0.to(DEV), eps=1e-3)
        assert none is None and torch.equal(x2, x)
    y = torch.randn(5, width, generator=g)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        xr = x.clone()
        h = residual_norm(xr, add=(y.to(dt).to(DEV),), weight=w1.to(DEV), eps=1e-3, kind=NORM_RMS_ONE_GAIN, out_dtype=dt)
        want = x.cpu().double() + y.to(dt).double()
        assert torch.allclose(xr.cpu().double(), want, rtol=1e-6, atol=1e-6)     # the sum is 32-bit in both
        assert torch.allclose(h.cpu().double(), O.scalar_norm(want, w1, 1e-3), rtol=tol, atol=tol)


def test_embed_norm_with_a_gain_per_coordinate():
    from compactor_vllm.layers.layernorm import embed_norm
    from oracle import pekasun as O

    g = torch.Generator().manual_seed(2)
    table, w0, w1 = (torch.randn(*s, generator=g) for s in ((9, 33), (33,), (33,)))
    ids = torch.tensor([8, 0, 4])
    x, h = embed_norm(ids.to(DEV), table.to(DEV), w0.to(DEV), next_weight=w1.to(DEV), eps=1e-5, out_dtype=torch.float32)
    want = O.rms_unit(table[ids], 1e-5) * w0.double()
    assert torch.allclose(x.cpu().double(), want, rtol=1e-5, atol=1e-6)
    assert torch.allclose(h.cpu().double(), O.rms_unit(want, 1e-5) * w1.double(), rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("sizes", [(4, 2, 12, 10), (3, 1, 32, 64), (2, 2, 1, 1), (2, 1, 130, 300)])
def test_query_key_and_value_norms_in_the_store(sizes):
    """q out, k and v in the cache: k with its weight, v without one; small values, so that eps counts."""
    from compactor_vllm import _native as N
    from oracle import pekasun as O

    H, G, D, Dv = sizes
    T, eps, ps = 5, 1e-2, 4
    g = torch.Generator().manual_seed(3)
    qkv = 0.1 * torch.randn(T, (H + G) * D + G * Dv, generator=g)
    wq, wk = 1 + torch.randn(D, generator=g), 1 + torch.randn(D, generator=g)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    pos, slot = i32([2, 3, 4, 5, 0]), i32([1, 1, 1, 1, 2])
    table = torch.arange(3 * G * 2, dtype=torch.int32, device=DEV).view(3, G, 2)
    kc, vc = torch.zeros(3 * G * 2 * ps, D, device=DEV), torch.zeros(3 * G * 2 * ps, Dv, device=DEV)
    qkv_d, wq_d, wk_d = qkv.to(DEV), wq.to(DEV), wk.to(DEV)
    for norm in (0, 1, 2, 3):
        q = torch.empty(T, H, D, device=DEV)
        N.check(N.lib().cvllm_rope_qknorm_store(
            N.ptr(qkv_d), qkv.stride(0), None, 0, norm, N.ptr(wq_d), N.ptr(wk_d), eps, N.ptr(pos),
            N.ptr(slot), N.ptr(q), N.ptr(kc), N.ptr(vc), N.ptr(table), table.stride(0), table.stride(1), ps, None, T, H, G,
            D, Dv, 0, N.CVLLM_F32, N.stream(DEV)), "store")
        k_in, v_in = qkv[:, H * D:(H + G) * D].view(T, G, D), qkv[:, (H + G) * D:].view(T, G, Dv)
        want_q = O.rms_unit(qkv[:, :H * D].view(T, H, D), eps) * wq.double() if norm & 1 else qkv[:, :H * D].view(T, H, D).double()
        want_k = O.rms_unit(k_in, eps) * wk.double() if norm & 1 else k_in.double()
        want_v = O.rms_unit(v_in, eps) if norm & 2 else v_in.double()
        assert torch.allclose(q.cpu().double(), want_q, rtol=1e-5, atol=1e-6)
        for t in range(T):
            for gg in range(G):
                p = int(pos[t])
                row = int(table[int(slot[t]), gg, p // ps]) * ps + p % ps
                assert torch.allclose(kc[row].cpu().double(), want_k[t, gg], rtol=1e-5, atol=1e-6)
                assert torch.allclose(vc[row].cpu().double(), want_v[t, gg], rtol=1e-5, atol=1e-6)


@pytest.mark.parametrize("neighbours", [0, 1])
@pytest.mark.parametrize("sizes", [(3, 10, 6, 20), (2, 5, 2, 7), (4, 16, 64, 100), (1, 1, 0, 3)])
def test_latent_prepare(neighbours, sizes):
    """Norm of the latent, rotation of the shared key part (with its amplitude) and of every head's query part, at
    positions around 5000; the reserved slot stores nothing."""
    from compactor_vllm import _native as N
    from oracle import pekasun as O

    H, D, R, r = sizes
    T, ps, eps, amp, p0 = 6, 8, 1e-4, 1.25, 4997
    g = torch.Generator().manual_seed(4)
    cols = torch.randn(T, H * (D + R) + r + R + 3, generator=g)
    w = 1 + 0.5 * torch.randn(r, generator=g)
    freq = torch.rand(R // 2, generator=g).double()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    pos = i32([p0 + i for i in range(T)])
    slot = i32([1] * (T - 1) + [0])
    table = torch.zeros(2, 1, 700, dtype=torch.int32, device=DEV)
    table[1, 0] = torch.arange(700)
    cache = torch.full((700 * ps, r + R), 7.0, device=DEV)
    q_full = torch.full((T, H, r + R), 5.0, device=DEV)
    lens = torch.zeros(2, dtype=torch.int32, device=DEV)
    cols_d, w_d, freq_d = cols.to(DEV), w.to(DEV), freq.to(DEV)
    N.check(N.lib().cvllm_latent_prepare(
        N.ptr(cols_d), cols.stride(0), 0, H, D, H * (D + R), r, R, N.ptr(w_d), eps, N.ptr(freq_d), amp,
        neighbours, N.ptr(pos), N.ptr(slot), N.ptr(q_full), q_full.stride(0), r + R, r, N.ptr(cache), N.ptr(table),
        table.stride(0), ps, N.ptr(lens), T, 0, N.CVLLM_F32, N.stream(DEV)), "prepare")

    def turned(x):      # x [T, ..., R]
        a = (torch.arange(T, dtype=torch.float64) + p0)[:, None] * freq
        c, s = amp * torch.cos(a), amp * torch.sin(a)
        c, s = c.view(T, *[1] * (x.dim() - 2), R // 2), s.view(T, *[1] * (x.dim() - 2), R // 2)
        x = x.double()
        u, v = (x[..., 0::2], x[..., 1::2]) if neighbours else (x[..., :R // 2], x[..., R // 2:])
        a, b = u * c - v * s, v * c + u * s
        return torch.stack([a, b], -1).flatten(-2) if neighbours else torch.cat([a, b], -1)

    q_in = cols[:, :H * (D + R)].view(T, H, D + R)
    assert torch.allclose(q_full[:, :, r:].cpu().double(), turned(q_in[..., D:]), rtol=1e-5, atol=1e-5)
    assert (q_full[:, :, :r] == 5.0).all()
    off = H * (D + R)
    want = torch.cat([O.rms_unit(cols[:, off:off + r], eps) * w.double(), turned(cols[:, off + r:off + r + R])], -1)
    assert torch.allclose(cache[p0:p0 + T - 1].cpu().double(), want[:-1], rtol=1e-5, atol=1e-5)
    assert (cache[p0 + T - 1:] == 7.0).all() and (cache[:p0] == 7.0).all()
    assert lens.tolist() == [0, p0 + T - 1]


@pytest.mark.parametrize("width,stride", [(64, 96), (30, 37), (8, 8)])
def test_sigmoid_gate_into_a_wider_row(width, stride):
    from compactor_vllm.layers.latent_attention import sigmoid_gate
    from oracle import pekasun as O

    g = torch.Generator().manual_seed(5)
    for dt, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-2)):
        x, z = torch.randn(7, width, generator=g).to(dt), (4 * torch.randn(7, stride, generator=g)).to(dt)
        buf = torch.full((7, stride + 8), 3.0, dtype=dt, device=DEV)
        sigmoid_gate(x.to(DEV), z.to(DEV)[:, stride - width:], buf[:, :width])
        want = x.double() * O.sigmoid(z[:, stride - width:].double())
        assert torch.allclose(buf[:, :width].cpu().double(), want, rtol=tol, atol=tol)
        assert (buf[:, width:] == 3.0).all()


# --------------------------------------------------------------- the attention kernels alone, with keys planted at edges
def dense_reference(starts, seqs, window, keep, scale, sink):
    """`seqs`: (q, k, v) of whole sequences (float64, [L, heads, size]); the outputs of the portions [start, L)."""
    from oracle import pekasun as O

    outs = []
    for (qs, ks, vs), start in zip(seqs, starts):
        L, H, G = qs.shape[0], qs.shape[1], ks.shape[1]
        seen = O.visible(L, {"size": window, "keep_first": keep})
        o = torch.stack([O.attend(qs[:, h], ks[:, h // (H // G)], vs[:, h // (H // G)], scale, seen,
                                  None if sink is None else sink[h]) for h in range(H)], 1)
        outs.append(o[start:])
    return torch.cat(outs)


def paged_attention(module, dtype, seqs, starts, page_size, option, decode=False, values_in_keys=False, wide_out=False):
    """The engine's attention kernels on the given sequences: every key in a paged cache with shuffled pages, the queries
    of the portions [start, L) (or, with `decode`, of the last position alone)."""
    from compactor_vllm import _native as N
    from compactor_vllm.utils.context import reset_context, set_context

    G, D, Dv = module.num_kv_heads, module.head_dim, module.v_head_dim
    B = len(seqs)
    P = max(-(-s[0].shape[0] // page_size) for s in seqs)
    n_pages = (B + 1) * G * P
    perm = torch.randperm(n_pages, generator=torch.Generator().manual_seed(9)).to(torch.int32)
    table = perm.view(B + 1, G, P).to(DEV)
    # rows nobody wrote hold NaN: reading one shows
    kc = torch.full((n_pages * page_size, D), float("nan"), dtype=dtype, device=DEV)
    vc = None if values_in_keys else torch.full((n_pages * page_size, Dv), float("nan"), dtype=dtype, device=DEV)
    for b, (_, ks, vs) in enumerate(seqs):
        for g in range(G):
            p = torch.arange(ks.shape[0], device=DEV)
            rows = table[b + 1, g].long()[p // page_size] * page_size + p % page_size
            kc[rows] = ks[:, g].to(dtype).to(DEV)
            if vc is not None:
                vc[rows] = vs[:, g].to(dtype).to(DEV)
    module.k_cache, module.v_cache, module.page_table, module.page_size = kc, vc, table, page_size
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    lens = [s[0].shape[0] for s in seqs]
    if decode:
        starts = [n - 1 for n in lens]
    new = [n - s for n, s in zip(lens, starts)]
    q = torch.cat([s[0][st:] for s, st in zip(seqs, starts)]).to(dtype).to(DEV).contiguous()
    cu = [0]
    for n in new:
        cu.append(cu[-1] + n)
    slots = i32(list(range(1, B + 1)))
    set_context(is_prefill=not decode, cu_seqlens_q=i32(cu), max_seqlen_q=max(new), max_seqlen_k=max(lens),
                batch_mapping=slots, positions_i32=i32([p for s, n in zip(starts, lens) for p in range(s, n)]),
                token_slot=i32([b + 1 for b, n in enumerate(new) for _ in range(n)]), seq_start=i32(starts))
    N.set_test_option("bias_attn_fma", option)
    try:
        if wide_out:
            H = module.num_heads
            buf = torch.full((q.shape[0], H * Dv + 24), 9.0, dtype=dtype, device=DEV)
            module.attend(q, out=buf[:, :H * Dv])
            assert (buf[:, H * Dv:] == 9.0).all()
            out = buf[:, :H * Dv].unflatten(1, (H, Dv))
        else:
            out = module.attend(q, flat=False)
    finally:
        N.set_test_option("bias_attn_fma", 0)
        reset_context()
    return out.double().cpu()


def make_module(H, G, D, Dv, scale, **kw):
    from compactor_vllm.layers.attention import BiasedChunkAttention

    with torch.device(DEV):
        return BiasedChunkAttention(H, G, D, Dv, scale, **kw)


def planted(L, H, G, D, Dv, seed, at, strength=6.0):
    """A sequence whose queries share a direction; the keys at the positions `at` point along it, the later in the list
    the stronger, so that the strongest VISIBLE one takes nearly all the weight (the numbers are bfloat16 ones)."""
    g = torch.Generator().manual_seed(seed)
    u = torch.nn.functional.normalize(torch.randn(D, generator=g), dim=0) * math.sqrt(D)
    q = 0.3 * torch.randn(L, H, D, generator=g) + u
    k = 0.3 * torch.randn(L, G, D, generator=g)
    v = torch.randn(L, G, Dv, generator=g)
    for i, p in enumerate(at):
        if p < L:
            k[p] += u * (strength + 4.0 * i) / math.sqrt(D)
    bf = lambda x: x.to(torch.bfloat16).double()
    return bf(q), bf(k), bf(v)


# (name, option, dtype, H, G, D, Dv, page size): the kernels an attention layer can land on
KERNELS = {
    "tcgen05": (0, torch.bfloat16, 4, 2, 128, 128, 128),
    "tcgen05_pages_of_256": (0, torch.bfloat16, 2, 1, 128, 128, 256),
    "mma_128": (2, torch.bfloat16, 2, 1, 128, 128, 128),
    "mma_64": (0, torch.bfloat16, 3, 1, 48, 40, 16),
    "fma_bf16": (1, torch.bfloat16, 2, 2, 48, 40, 16),
    "fma_f32": (0, torch.float32, 3, 3, 17, 23, 16),
    "fma_wide_rows": (0, torch.float32, 1, 1, 576, 512, 64),
}


@pytest.mark.parametrize("name", sorted(KERNELS))
@pytest.mark.parametrize("window,keep", [(0, 0), (150, 0), (150, 5), (300, 140), (129, 1), (7, 3), (1, 2)])
def test_window_and_kept_tokens_in_portions(name, window, keep):
    """Three sequences in a batch, each with ONE planted key that takes nearly all the weight wherever it is seen: the
    last kept token, the first one that is not kept, and one a little later.  One token too many or too few at either
    edge changes whole rows (the case asks the dense softmax with edges moved by one first).  Portions at the start, in
    the middle and across tile borders; cache rows that were never written hold NaN."""
    option, dtype, H, G, D, Dv, ps = KERNELS[name]
    L = 500
    if name == "fma_wide_rows":
        L, window, keep = 180, -(-window // 3), keep // 3
    seqs = [planted(L, H, G, D, Dv, 1, [keep]), planted(L - 11, H, G, D, Dv, 2, [keep - 1 if keep else 1]),
            planted(L - 23, H, G, D, Dv, 3, [keep + 10])]
    scale = D ** -0.5
    whole = dense_reference([0, 0, 0], seqs, window, keep, scale, None)
    if window > 1:
        others = [(window - 1, keep), (window + 1, keep), (window, keep + 1)] + ([(window, keep - 1)] if keep else [])
        for w2, k2 in others:
            assert (dense_reference([0, 0, 0], seqs, w2, k2, scale, None) - whole).abs().max() > 1.0, (w2, k2)
    m = make_module(H, G, D, Dv, scale, window=window, keep_first=keep)
    for starts in ([0, 0, 0], [L - 131, 64, 1], [128, L - 13, keep + window // 2]):
        want = dense_reference(starts, seqs, window, keep, scale, None)
        got = paged_attention(m, dtype, seqs, starts, ps, option, wide_out=starts[0] == 0)
        tol = 3e-2 if dtype == torch.bfloat16 else 2e-4
        assert (got - want).abs().max() < tol, (starts, (got - want).abs().max())


DECODE_KERNELS = {"split_bf16": (torch.bfloat16, 6, 1, 64, 64, 64), "split_f32": (torch.float32, 4, 2, 40, 24, 16),
                  "split_128": (torch.bfloat16, 8, 2, 128, 128, 128), "plain_odd": (torch.float32, 3, 1, 17, 23, 16),
                  "plain_wide_rows": (torch.bfloat16, 2, 1, 576, 512, 64)}


@pytest.mark.parametrize("name", sorted(DECODE_KERNELS))
@pytest.mark.parametrize("splits", [1, 3, None])
@pytest.mark.parametrize("window,keep", [(0, 0), (37, 0), (37, 5), (64, 70), (1, 2), (200, 1)])
def test_window_and_kept_tokens_in_decoding(name, splits, window, keep):
    """Sequences whose lengths put the planted keys just inside and just outside the window of the last token."""
    dtype, H, G, D, Dv, ps = DECODE_KERNELS[name]
    scale = D ** -0.5
    lens = [1, 2, 40, window + 1, window + 2, window + keep + 1, window + keep + 30, 333]
    seqs = []
    for i, n in enumerate(lens):
        last = n - 1
        edge_in, edge_out = max(last - window + 1, 0), max(last - window, 0)
        at = [p for p in (edge_in, keep - 1, keep, edge_out) if 0 <= p < n] if i % 2 else [p for p in (keep, edge_out, edge_in, keep - 1) if 0 <= p < n]
        seqs.append(planted(n, H, G, D, Dv, 20 + i, at))
    m = make_module(H, G, D, Dv, scale, window=window, keep_first=keep)
    if splits is not None:
        m.decode_splits = lambda *_: splits
    want = dense_reference([n - 1 for n in lens], seqs, window, keep, scale, None)
    for wide in (False, True):
        got = paged_attention(m, dtype, seqs, None, ps, 0, decode=True, wide_out=wide)
        assert (got - want).abs().max() < (3e-2 if dtype == torch.bfloat16 else 2e-4)


@pytest.mark.parametrize("case", ["tcgen05_whole_row", "mma", "fma_f32", "fma_wide"])
@pytest.mark.parametrize("window", [0, 33, 150])
def test_latent_rows_with_a_window_and_sinks(case, window):
    """Values that are columns of the key rows, learned sinks of very different size; portions and decoding.  Rows of
    128 numbers in pages of 128 take the tcgen05 kernel with the whole row as the value."""
    dtype, H, D, Dv, ps = {"tcgen05_whole_row": (torch.bfloat16, 4, 128, 96, 128), "mma": (torch.bfloat16, 3, 80, 64, 16),
                           "fma_f32": (torch.float32, 3, 25, 19, 16), "fma_wide": (torch.float32, 2, 576, 512, 64)}[case]
    scale = D ** -0.5
    L = 400 if case != "fma_wide" else 170
    seqs = []
    for i, n in enumerate((L, L // 2 + 5)):
        q, k, _ = planted(n, H, 1, D, Dv, 30 + i, [20, 60, 61, n // 2])
        seqs.append((q, k, k[..., :Dv]))
    m = make_module(H, 1, D, Dv, scale, window=window, values_in_keys=True, sink=True, learned_sink=True)
    for sink in (torch.tensor([-40.0, 2.5, 14.0, 0.0])[:H], torch.tensor([3.0, -1.0, 6.0, 9.0])[:H]):
        with torch.no_grad():
            m.sink_logits.copy_(sink)
        for starts in ([0, 0], [L - 140, 70], [L - 2, L // 2]):
            want = dense_reference(starts, seqs, window, 0, scale, sink.double())
            got = paged_attention(m, dtype, seqs, starts, ps, 0, values_in_keys=True)
            assert (got - want).abs().max() < (3e-2 if dtype == torch.bfloat16 else 2e-4), starts
        want = dense_reference([L - 1, L // 2 + 4], seqs, window, 0, scale, sink.double())
        got = paged_attention(m, dtype, seqs, None, ps, 0, decode=True, values_in_keys=True)
        assert (got - want).abs().max() < (3e-2 if dtype == torch.bfloat16 else 2e-4)


# (heads, D, Dv, page size, option): decoding with fewer than 8 heads takes the kernel only when it is asked for
WIDE = {"576": (5, 576, 512, 64, 3), "576_heads_of_48": (48, 576, 512, 128, 0), "partial_chunks": (3, 200, 136, 64, 3),
        "130_heads": (130, 144, 80, 64, 0), "two_slices_of_320": (16, 384, 320, 192, 0), "whole_row": (2, 136, 136, 64, 3),
        "narrow": (7, 80, 64, 64, 3), "one_chunk": (33, 64, 64, 128, 3)}


@pytest.mark.parametrize("name", sorted(WIDE))
@pytest.mark.parametrize("window,keep", [(0, 0), (33, 0), (150, 0), (64, 70), (1, 2)])
@pytest.mark.parametrize("threshold", [-1.0, 0.0])
def test_wide_latent_rows_on_tensor_cores(name, window, keep, threshold):
    """csrc/latent_attn_umma.cu: one planted key per sequence at the edges of window and kept tokens, sinks of very
    different size, portions and decoding with one and several key splits; threshold 0 rescales at every growing maximum."""
    import ctypes

    from compactor_vllm import _native as N

    H, D, Dv, ps, option = WIDE[name]
    scale = D ** -0.5
    L = 250 if D > 300 else 400
    seqs = []
    for i, (n, at) in enumerate(((L, [keep]), (L - 11, [keep - 1 if keep else 1, 60]), (L // 3, [20]))):
        q, k, _ = planted(n, H, 1, D, Dv, 40 + i, at)
        seqs.append((q, k, k[..., :Dv]))
    m = make_module(H, 1, D, Dv, scale, window=window, keep_first=keep, values_in_keys=True, sink=True, learned_sink=True)
    g = torch.Generator().manual_seed(3)
    sink = 4 * torch.randn(H, generator=g)
    with torch.no_grad():
        m.sink_logits.copy_(sink)
    N.set_test_option("prefill_threshold", threshold)
    try:
        for starts in ([0, 1, 2], [L - 70, L - 13, L // 3 - 1]):
            want = dense_reference(starts, seqs, window, keep, scale, sink.double())
            got = paged_attention(m, torch.bfloat16, seqs, starts, ps, option, values_in_keys=True, wide_out=starts[0] == 0)
            assert (got - want).abs().max() < 3e-2, (starts, (got - want).abs().max())
        want = dense_reference([len(s[0]) - 1 for s in seqs], seqs, window, keep, scale, sink.double())
        for splits in (1, 2, 5):
            m.decode_splits = lambda *_: splits
            got = paged_attention(m, torch.bfloat16, seqs, None, ps, option, decode=True, values_in_keys=True,
                                  wide_out=splits == 2)
            assert (got - want).abs().max() < 3e-2, splits
    finally:
        N.set_test_option("prefill_threshold", -1.0)
    count = ctypes.c_int(-1)
    N.check(N.lib().cvllm_latent_attn_aborts(ctypes.byref(count)), "aborts")
    assert count.value == 0


# ------------------------------------------------------------------------------------------------------ single layers
MIXER_CASES = {
    "attention": (attn(4, 2, 12, 10, 7, 3), None),
    "attention_with_ff": (attn(2, 1, 16, 16, 9, 2), dense(24)),
    "attention_no_kept_tokens": (attn(2, 2, 8, 12, 5, 0), None),
    "attention_window_of_one": (attn(3, 1, 10, 6, 1, 4), dense(9)),
    "attention_keeps_more_than_its_window": (attn(3, 3, 9, 9, 4, 20), None),
    "attention_no_window": (attn(2, 1, 16, 8, 0, 0), dense(16)),
    "latent": (latent(3, 10, 6, 14, 20, 9), None),
    "latent_with_ff": (latent(2, 16, 8, 8, 24, 17), dense(31)),
    "latent_window_of_one": (latent(2, 6, 4, 5, 9, 1), None),
    "latent_no_window": (latent(4, 8, 16, 8, 16, 0), dense(12)),
    "latent_factor_one": (latent(2, 8, 8, 8, 16, 12, factor=1.0), None),
}


@pytest.mark.parametrize("name", sorted(MIXER_CASES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mixer_alone(name, dtype):
    """One layer: whole prompt, portions down to two and one tokens, token-by-token decoding."""
    from oracle import pekasun as O

    cfg = model_cfg([MIXER_CASES[name]])
    r, t = build(cfg, dtype, pages=12, page_size=16)
    toks = tokens(45, 83, 5)
    want = O.forward(cfg, t, toks)
    for sizes in ([45], [2], [1], [7, 1, 16, 3]):
        assert close(run_in_portions(r, toks, sizes), want, dtype), sizes


@pytest.mark.parametrize("kw", [dict(base=50.0, factor=8.0, original=64, fast=8.0, slow=1.0),
                                dict(base=10000.0, factor=2.0, original=4096, fast=32.0, slow=1.0),
                                dict(base=7.0, factor=40.0, original=500, fast=3.0, slow=2.9),
                                dict(base=1e6, factor=1.5, original=20, fast=1.0, slow=0.01)])
@pytest.mark.parametrize("rot", [2, 8, 20])
def test_rotation_frequencies(kw, rot):
    """The frequencies are the oracle's; in a model the rotated part alone decides the scores (dim 1), so a wrong pairing,
    ramp or amplitude shows at once."""
    from compactor_vllm.layers.attention import yarn_amplitude, yarn_rotation_frequencies
    from oracle import pekasun as O

    f = yarn_rotation_frequencies(rot, kw["base"], kw["factor"], kw["original"], kw["fast"], kw["slow"])
    assert torch.allclose(f, O.frequencies(rot, kw["base"], kw), rtol=1e-12)
    assert abs(yarn_amplitude(kw["factor"]) - O.amplitude(kw)) < 1e-12
    cfg = model_cfg([(latent(3, 1, rot, 8, 12, 60, scale=1.0, **kw), None)])
    r, t = build(cfg, "float32", pages=12)
    t["l0.mix.q"] = t["l0.mix.q"] * 2
    r.model.load_weights(t)
    toks = tokens(90, 83, 6)
    want = O.forward(cfg, t, toks)
    for sizes in ([90], [33, 1, 2]):
        assert rel_err(run_in_portions(r, toks, sizes), want) < TOL, sizes


def test_a_large_sink_takes_the_weight():
    from oracle import pekasun as O

    cfg = model_cfg([(latent(2, 8, 8, 8, 16, 9), None)])
    r, t = build(cfg, "float32", pages=8)
    toks = tokens(40, 83, 6)
    outs = []
    for value in (-30.0, 0.0, 9.0):
        t["l0.mix.sink"] = torch.tensor([value, value / 2]).to(torch.bfloat16)
        r.model.load_weights(t)
        want = O.forward(cfg, t, toks)
        outs.append(want)
        for sizes in ([40], [33, 1], [5]):
            assert rel_err(run_in_portions(r, toks, sizes), want) < TOL, (value, sizes)
    assert (outs[0] - outs[1]).abs().max() > 1e-3 and (outs[1] - outs[2]).abs().max() > 1e-3


@pytest.mark.parametrize("kind", ["attention", "latent"])
@pytest.mark.parametrize("window", [2, 5, 16, 17, 33])
def test_window_edges_in_portions_and_decoding(kind, window):
    """Sharp scores through the whole model: windows shorter than, equal to and longer than a page of 16, cuts before,
    at and behind the edge; the oracle is asked with a window one shorter and one longer first."""
    from oracle import pekasun as O

    layer = (lambda w: attn(2, 1, 16, 16, w, 3, scale=1.5)) if kind == "attention" else (lambda w: latent(2, 12, 8, 16, 16, w, scale=1.5))
    cfg = model_cfg([(layer(window), None)])
    r, t = build(cfg, "float32", pages=12, page_size=16)
    toks = tokens(80, 83, 7)
    want = O.forward(cfg, t, toks)
    for other in (window - 1, window + 1):
        assert rel_err(O.forward(model_cfg([(layer(other), None)]), t, toks), want) > 1e-2
    for sizes in ([80], [window, 1], [window - 1, 2], [16], [3, 64]):
        assert rel_err(run_in_portions(r, toks, sizes), want) < TOL, sizes
    seq = new_seq()
    out = [feed(r, seq, toks[:3])] + [feed(r, seq, [x]) for x in toks[3:]]
    r.release([seq])
    assert rel_err(torch.cat(out), want) < TOL


@pytest.mark.parametrize("keep", [1, 15, 16, 17, 40])
def test_kept_tokens_in_portions_and_decoding(keep):
    """Kept tokens that end before, at and behind a page's border, and more of them than the window; the first ones are
    seen 190 tokens later."""
    from oracle import pekasun as O

    cfg = model_cfg([(attn(2, 1, 16, 16, 11, keep, scale=1.5), None)])
    r, t = build(cfg, "float32", pages=16, page_size=16)
    toks = tokens(200, 83, 8)
    want = O.forward(cfg, t, toks)
    for other in (keep - 1, keep + 1):
        assert rel_err(O.forward(model_cfg([(attn(2, 1, 16, 16, 11, other, scale=1.5), None)]), t, toks), want) > 1e-2
    alt = [(toks[0] + 1) % 83] + toks[1:]
    assert (O.forward(cfg, t, alt)[-1] - want[-1]).abs().max().item() > 2e-4
    for sizes in ([200], [keep, 2], [max(keep - 1, 1), 64, 1], [16], [150, 1, 1, 7]):
        assert rel_err(run_in_portions(r, toks, sizes), want) < TOL, sizes


def test_layers_that_share_weights_have_caches_of_their_own():
    """The same attention weights three times in a row: the second and third see their own inputs' keys, so a cache that
    was shared as well would give other logits (the oracle with one layer differs from it with three)."""
    from oracle import pekasun as O

    cfg = model_cfg([(attn(2, 1, 16, 16, 9, 2), dense(20)), 0, (latent(2, 8, 4, 8, 12, 7), None), 1, 2])
    r, t = build(cfg, "float32", pages=10)
    assert len(r.model.layers) == 2 and len(r.model.runs) == 5
    caches = [a.k_cache.data_ptr() for _, a in r.model.runs]
    assert len(set(caches)) == 5
    toks = tokens(50, 83, 12)
    want = O.forward(cfg, t, toks)
    assert rel_err(O.forward(model_cfg([cfg_layer for cfg_layer in [(attn(2, 1, 16, 16, 9, 2), dense(20))]]), t, toks), want) > 1e-2
    for sizes in ([50], [2], [1], [17, 3]):
        assert rel_err(run_in_portions(r, toks, sizes), want) < TOL, sizes


# ------------------------------------------------------------------- whole prompts, portions, decoding, first tokens
@pytest.mark.parametrize("dtype,cfg", [("float32", config_a), ("float32", config_b), ("bfloat16", config_b),
                                       ("bfloat16", config_a)])
def test_prefill_portions_and_decoding_agree_with_the_oracle(dtype, cfg):
    from oracle import pekasun as O

    c = cfg()
    r, t = build(c, dtype, pages=16, page_size=16)
    toks = tokens(70, c["vocab"], 7)
    want = O.forward(c, t, toks)
    for sizes in ([70], [2], [16], [17, 1, 1, 30], [3, 64]):
        assert close(run_in_portions(r, toks, sizes), want, dtype), sizes
    seq = new_seq()
    out = [feed(r, seq, toks[:1])] + [feed(r, seq, [x]) for x in toks[1:]]
    r.release([seq])
    assert close(torch.cat(out), want, dtype)


def test_large_heads_in_pages_of_128():
    """bfloat16 heads of 128 and latent rows of 128: the portion kernel on the tensor cores' TMEM pipeline inside a model,
    portions that start and end inside its tiles, then decoding."""
    from oracle import pekasun as O

    c = model_cfg([(attn(4, 2, 128, 128, 200, 4), dense(64)), (latent(2, 32, 32, 32, 96, 150), None), 0], width=64)
    r, t = build(c, "bfloat16", pages=8, page_size=128)
    toks = tokens(600, 83, 3)
    want = O.forward(c, t, toks)
    for sizes in ([600], [130, 1, 250], [64]):
        assert close(run_in_portions(r, toks, sizes), want, "bfloat16"), sizes


def test_residual_stream_after_every_layer():
    from oracle import pekasun as O

    c = config_a()
    r, t = build(c, "float32", pages=8)
    toks = tokens(20, 83, 8)
    want = []
    O.forward(c, t, toks, want)
    r.model.debug_residuals = got = []
    seq = new_seq()
    feed(r, seq, toks)
    r.model.debug_residuals = None
    r.release([seq])
    assert len(got) == len(want) == 7
    for i, (g, w) in enumerate(zip(got, want)):
        assert torch.allclose(g.cpu().double(), w, rtol=1e-4, atol=1e-4), i


@pytest.mark.parametrize("eager", [True, False])
def test_first_tokens_of_a_sequence(eager):
    """One-token requests, and the first steps of a request one token at a time (the graph's first replay included)."""
    from oracle import pekasun as O

    c = config_a()
    r, t = build(c, "float32", pages=8, eager=eager)
    for seed in (1, 2):
        toks = tokens(6, 83, seed)
        want = O.forward(c, t, toks)
        seq = new_seq()
        out = [feed(r, seq, [x]) for x in toks]
        r.release([seq])
        assert rel_err(torch.cat(out), want) < TOL
        assert rel_err(run_in_portions(r, toks[:1], [1]), want[:1]) < TOL


@pytest.mark.parametrize("eager", [True, False])
def test_long_decoding_over_pages(eager):
    """A short prompt, then 150 single-token steps over ten pages and several windows (eager kernels, graph replays)."""
    from oracle import pekasun as O

    c = config_a()
    r, t = build(c, "float32", pages=12, eager=eager)
    toks = tokens(160, 83, 11)
    want = O.forward(c, t, toks)
    seq = new_seq()
    out = [feed(r, seq, toks[:10])] + [feed(r, seq, [x]) for x in toks[10:]]
    r.release([seq])
    if not eager:
        assert r.stats["graph_replays"] == 150
    assert rel_err(torch.cat(out), want) < TOL


def test_graph_decode_batches_with_padding_rows():
    """Three decoding requests (padded to four rows in the graph) of unequal lengths, one of which ends early."""
    from oracle import pekasun as O

    c = config_a()
    r, t = build(c, "float32", pages=20, eager=False)
    reqs = [tokens(n, 83, 40 + i) for i, n in enumerate((30, 12, 21))]
    want = [O.forward(c, t, q) for q in reqs]
    seqs = [new_seq() for _ in reqs]
    got = [[feed(r, s, q[:4])] for s, q in zip(seqs, reqs)]
    for k in range(4, 30):
        live = [i for i, q in enumerate(reqs) if k < len(q)]
        for i in live:
            seqs[i].prompt_token_ids.append(reqs[i][k])
        logits = r.run_step([(seqs[i], [reqs[i][k]]) for i in live])
        for j, i in enumerate(live):
            got[i].append(logits[j:j + 1])
        r.release([seqs[i] for i in live if k == len(reqs[i]) - 1])
    for i in range(3):
        assert rel_err(torch.cat(got[i]), want[i]) < TOL


# ---------------------------------------------------------------------------------- batches, pages and slots reused
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_each_request_alone(dtype):
    """Four requests of unequal lengths in one step after another: portions of some beside single tokens of others."""
    from oracle import pekasun as O

    c = config_a() if dtype == "float32" else config_b()
    r, t = build(c, dtype, pages=30)
    reqs = [tokens(n, c["vocab"], 70 + i) for i, n in enumerate((61, 9, 33, 2))]
    plan = [[5, 1, 1, 1, 20, 1, 1, 30, 1], [9], [1, 1, 16, 2, 13], [1, 1]]      # portion sizes per request, step by step
    seqs, at, outs = [new_seq() for _ in reqs], [0] * 4, [[] for _ in reqs]
    step = 0
    while any(at[i] < len(reqs[i]) for i in range(4)):
        entries, spans, base = [], [], 0
        for i in range(4):
            if step < len(plan[i]) and at[i] < len(reqs[i]):
                n = min(plan[i][step], len(reqs[i]) - at[i])
                part = reqs[i][at[i]:at[i] + n]
                seqs[i].prompt_token_ids.extend(part)
                entries.append((seqs[i], part))
                spans.append((i, base, n))
                at[i] += n
                base += n
        logits = r.run_step(entries, rows=list(range(base)))
        for i, b, n in spans:
            outs[i].append(logits[b:b + n])
        step += 1
    for i in range(4):
        assert close(torch.cat(outs[i]), O.forward(c, t, reqs[i]), dtype), i


@pytest.mark.parametrize("device_allocator", [False, True])
def test_pages_and_slots_are_reused(device_allocator):
    """A pool of 8 pages and 2 slots serves 6 requests, two at a time: every page and slot is used again by a later
    request - also by a shorter one, whose first tokens must not see what the pages held before."""
    from oracle import pekasun as O

    c = config_a()
    r, t = build(c, "float32", pages=8, max_seqs=2, device_allocator=device_allocator)
    lens = (50, 60, 64, 3, 1, 49)
    for k in range(0, len(lens), 2):
        pair = [tokens(lens[k], 83, 20 + k), tokens(lens[k + 1], 83, 21 + k)]
        seqs, outs, at = [new_seq(), new_seq()], [[], []], [0, 0]
        while any(at[i] < len(pair[i]) for i in range(2)):
            entries, spans, base = [], [], 0
            for i in range(2):
                n = min(11 + 6 * i, len(pair[i]) - at[i])
                if n:
                    part = pair[i][at[i]:at[i] + n]
                    seqs[i].prompt_token_ids.extend(part)
                    entries.append((seqs[i], part))
                    spans.append((i, base, n))
                    at[i] += n
                    base += n
            logits = r.run_step(entries, rows=list(range(base)))
            for i, b, n in spans:
                outs[i].append(logits[b:b + n])
        r.release(seqs)
        for i in range(2):
            assert rel_err(torch.cat(outs[i]), O.forward(c, t, pair[i])) < TOL, (k, i)
    assert r.kv.num_free_batches == 2


def test_a_request_left_out_of_steps_goes_on_later():
    from oracle import pekasun as O

    c = config_a()
    r, t = build(c, "float32", pages=12)
    a, b = tokens(40, 83, 31), tokens(30, 83, 32)
    sa, sb = new_seq(), new_seq()
    out_a = [feed(r, sa, a[:13])]
    out_b = [feed(r, sb, b[:20]), feed(r, sb, b[20:21]), feed(r, sb, b[21:])]     # a waits meanwhile
    out_a += [feed(r, sa, a[13:14]), feed(r, sa, a[14:])]
    r.release([sa, sb])
    assert rel_err(torch.cat(out_a), O.forward(c, t, a)) < TOL
    assert rel_err(torch.cat(out_b), O.forward(c, t, b)) < TOL


# ------------------------------------------------------------------------------------------------------ other sizes
OTHER_SIZES = {
    "everything_one": [(attn(1, 1, 1, 1, 1, 1, scale=1.0), dense(1)),
                       (latent(1, 1, 2, 1, 1, 1, factor=1.0, original=10), dense(1)), 0, 1],
    "one_head_per_group": [(attn(5, 5, 8, 8, 6, 2), None), (latent(1, 8, 8, 8, 8, 5), dense(16))],
    "all_heads_share_one": [(attn(6, 1, 16, 8, 12, 4), dense(32)), (latent(6, 4, 2, 30, 5, 12), None)],
    "wide_heads": [(attn(2, 1, 128, 128, 30, 2), None), (latent(2, 64, 64, 128, 192, 26), dense(32))],
    "key_of_72_value_of_136": [(attn(2, 2, 72, 136, 25, 9), None), (latent(3, 40, 24, 8, 136, 25), None)],
    "rows_of_576": [(latent(2, 128, 64, 128, 512, 21), dense(8))],
    "wide_latent_pages": [(latent(6, 32, 32, 24, 160, 21), dense(8)), (attn(2, 1, 64, 64, 9, 2), None), 0],
    "attention_alone_no_mlp": [(attn(2, 1, 8, 8, 5, 1), None), 0, 0],
}


@pytest.mark.parametrize("name", sorted(OTHER_SIZES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(name, dtype):
    from oracle import pekasun as O

    width = {"everything_one": 6, "wide_heads": 128}.get(name, 40)
    c = model_cfg(OTHER_SIZES[name], vocab=37, width=width, eps=3e-6)
    r, t = build(c, dtype, pages=4 if "wide_latent" in name else 10, page_size=64 if "wide_latent" in name else 16)
    toks = tokens(50, 37, 9)
    want = O.forward(c, t, toks)
    for sizes in ([50], [9, 2, 1]):
        assert close(run_in_portions(r, toks, sizes), want, dtype), sizes
    seq = new_seq()
    out = [feed(r, seq, toks[:31])] + [feed(r, seq, [x]) for x in toks[31:]]
    r.release([seq])
    assert close(torch.cat(out), want, dtype)


def _random_config(seed):
    g = torch.Generator().manual_seed(1000 + seed)
    ri = lambda lo, hi: int(torch.randint(lo, hi + 1, (1,), generator=g))
    layers = []
    for i in range(ri(2, 6)):
        kind = ri(0, 4)
        mlp = dense(ri(4, 50)) if ri(0, 2) else None
        if kind == 0 and i:
            layers.append(ri(0, i - 1))
        elif kind <= 2:
            G = ri(1, 3)
            layers.append((attn(G * ri(1, 3), G, ri(2, 24), ri(2, 24), ri(1, 40), ri(0, 12), scale=0.1 + 0.05 * ri(0, 8)), mlp))
        else:
            layers.append((latent(ri(1, 5), ri(1, 20), 2 * ri(1, 10), ri(1, 20), ri(2, 40), ri(1, 40), base=float(ri(5, 20000)),
                                  factor=1.0 + ri(0, 30) / 4, original=ri(10, 3000), fast=float(ri(2, 40)),
                                  slow=ri(1, 10) / 5, scale=0.1 + 0.05 * ri(0, 8)), mlp))
    return model_cfg(layers, vocab=ri(20, 120), width=ri(8, 70), eps=10.0 ** -ri(4, 7))


@pytest.mark.parametrize("seed", range(12))
def test_models_drawn_at_random(seed):
    """Layer order, shared weights, every size and every constant drawn at random; whole, in portions, decoding, two in a
    batch."""
    from oracle import pekasun as O

    c = _random_config(seed)
    r, t = build(c, "float32", seed=seed, pages=16, max_seqs=2)
    a, b = tokens(57, c["vocab"], seed), tokens(23, c["vocab"], seed + 50)
    wa, wb = O.forward(c, t, a), O.forward(c, t, b)
    for sizes in ([57], [5, 1, 2, 30]):
        assert rel_err(run_in_portions(r, a, sizes), wa) < TOL, sizes
    sa, sb = new_seq(), new_seq()
    oa, ob = [feed(r, sa, a[:40])], []
    for k in range(17):
        sa.prompt_token_ids.append(a[40 + k])
        part = b[:7] if k == 0 else b[6 + k:7 + k]
        sb.prompt_token_ids.extend(part)
        logits = r.run_step([(sa, [a[40 + k]]), (sb, part)], rows=list(range(1 + len(part))))
        oa.append(logits[:1])
        ob.append(logits[1:])
    r.release([sa, sb])
    assert rel_err(torch.cat(oa), wa) < TOL
    assert rel_err(torch.cat(ob), wb) < TOL


# ----------------------------------------------------------------------------------------- the engine's entry point
@pytest.mark.parametrize("eager", [True, False])
def test_greedy_generation_through_llm_generate(eager):
    """`LLM.generate` with the step scheduler: prompts in portions of at most 16 tokens beside decoding requests, five
    requests on three slots, single-token steps from the decode graph.  Teacher forcing against the oracle: every
    generated token must be the oracle's argmax unless the oracle's two best logits are closer than rounding."""
    from compactor_vllm import LLM
    from compactor_vllm.api_types import SamplingParams
    from compactor_vllm.config.engine_config import LLMConfig
    from compactor_vllm.config.model_config import PekasunConfig
    from oracle import pekasun as O

    c = config_a()
    t = random_checkpoint(c, 3)
    cfg = LLMConfig(model="synthetic", hf_config=PekasunConfig.from_json(c), dtype="float32", max_num_seqs=3,
                    kvcache_page_size=16, max_model_len=160, enforce_eager=eager)
    llm = LLM(cfg, num_pages=14, device_allocator=False, max_batched_tokens=16)
    llm.model_runner.model.load_weights(t)
    prompts = [tokens(n, 83, 30 + i) for i, n in enumerate((40, 3, 25, 1, 18))]
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=12))
    assert llm.model_runner.kv.num_free_batches == 3
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        logits = O.forward(c, t, p + o[:-1])[len(p) - 1:]
        for k, tok in enumerate(o):
            best = torch.topk(logits[k], 2)
            assert tok == int(best.indices[0]) or float(best.values[0] - best.values[1]) < 1e-3, (k, tok)


def test_checkpoints_that_do_not_fit_are_refused():
    c = config_b()
    t = random_checkpoint(c, 1)
    r = make_runner(c, t, pages=4)
    missing = dict(t)
    del missing["l1.mix.sink"]
    with pytest.raises(KeyError):
        r.model.load_weights(missing)
    with pytest.raises(ValueError):
        r.model.load_weights(dict(t, **{"l0.mix.k": t["l0.mix.k"][:-1]}))
