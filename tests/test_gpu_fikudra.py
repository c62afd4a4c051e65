"""Fikudra through the engine against the plain CPU oracle (oracle/fikudra.py).

Every test makes its own small configuration and random weights (checkpoint tensors under the design's names, loaded
by the model's `load_weights`).  The engine runs them through its runner (`ModelRunner.run_step`, the paged cache, the
state pool, the native kernels); the oracle recomputes whole sequences without a cache or a carried state.  float32
runs are compared sharply (they show a key that is one position off, a lost state or a missing sink), bfloat16 loosely."""
import pytest
import torch

from fikudra_common import (TOL, attn, build, clean, close, config_a, config_b, feed, gla, model_cfg, moe, new_seq,
                            random_checkpoint, rel_err, routed_close, row_errs, run_in_portions, tokens)

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0) if torch.cuda.is_available() else None


# ------------------------------------------------------------------------------------------ mechanisms one by one
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8, 11, 16])
@pytest.mark.parametrize("width", [37, 64, 1032])
def test_streams_mix_read_and_norm(streams, width):
    """Both directions of the mix matrix differ, so [from, to] shows; from one tensor (equal streams), from separate
    streams into another tensor, and in place; the sum of the streams through a norm without writing them."""
    from compactor_vllm.layers.layernorm import StreamCoefficients, stream_mix_norm
    from oracle import fikudra as O

    g = torch.Generator().manual_seed(streams)
    T, S, eps = 5, streams, 1e-3
    c = StreamCoefficients(S)
    c.mix.data, c.w_out.data, c.w_in.data = (torch.randn(S, S, generator=g), torch.randn(S, generator=g),
                                             torch.randn(S, generator=g))
    w = 0.3 * torch.randn(width, generator=g)
    X = torch.randn(T, S, width, generator=g)
    cd = StreamCoefficients(S).to(DEV)
    cd.load_state_dict(c.state_dict())

    def read(xs, w_in):
        return O.zero_centred_norm(O.streams_read(xs, w_in), w, eps)

    for ydt in (torch.float32, torch.bfloat16):
        y = torch.randn(T, width, generator=g).to(ydt)
        for src in (X, X[:, 0]):
            xs = [X[:, s].double() for s in range(S)] if src.dim() == 3 else [X[:, 0].double()] * S
            new = O.streams_write(xs, c.mix.detach(), c.w_out.detach(), y.double())
            tol = dict(rtol=1e-5, atol=2e-5)
            dst = torch.full((T, S, width), float("nan"), device=DEV)
            h = stream_mix_norm(src.to(DEV), S, branch=y.to(DEV), coeff=cd, dst=dst, w_in=cd.w_in, weight=w.to(DEV),
                                gain_offset=1.0, eps=eps, out_dtype=torch.float32)
            assert torch.allclose(dst.cpu().double(), torch.stack(new, 1), **tol)
            assert torch.allclose(h.cpu().double(), read(new, c.w_in.detach()), rtol=2e-4, atol=2e-4)
            if src.dim() == 3:
                x = src.to(DEV)
                assert stream_mix_norm(x, S, branch=y.to(DEV), coeff=cd, dst=x) is None      # in place, the update alone
                assert torch.allclose(x.cpu().double(), torch.stack(new, 1), **tol)
            h = stream_mix_norm(src.to(DEV), S, branch=y.to(DEV), coeff=cd, weight=w.to(DEV), gain_offset=1.0, eps=eps,
                                out_dtype=torch.bfloat16)                                    # the sum, nothing written
            assert torch.allclose(h.float().cpu().double(), read(new, torch.ones(S)), rtol=1e-2, atol=1e-2)
            h = stream_mix_norm(src.to(DEV), S, w_in=cd.w_in, weight=w.to(DEV), gain_offset=1.0, eps=eps)
            assert torch.allclose(h.cpu().double(), read(xs, c.w_in.detach()), rtol=2e-4, atol=2e-4)


@pytest.mark.parametrize("E,top,groups,keep", [(10, 3, 2, 1), (12, 3, 4, 2), (8, 4, 4, 2), (6, 1, 6, 3), (5, 5, 1, 1),
                                               (64, 8, 8, 3), (96, 40, 4, 2), (1, 1, 1, 1)])
def test_group_limited_sigmoid_routing(E, top, groups, keep):
    """A group's rank is the sum of its two largest scores (of its one score when it has one), the weights are
    renormalized and scaled; a correction (not part of this design) shifts the choice alone."""
    from compactor_vllm.layers.moe import ROUTE_SIGMOID_GROUPS, route
    from oracle import fikudra as O

    g = torch.Generator().manual_seed(E + top)
    z = 2 * torch.randn(40, E + 1, generator=g)        # one more column that is no router output
    idx, w = route(z.to(DEV), None, top, groups, keep, ROUTE_SIGMOID_GROUPS, E, 1.9)
    s = torch.sigmoid(z.double())
    for t in range(40):
        want = O.route_token(s[t, :E].tolist(), {"experts": E, "top": top, "scale": 1.9, "groups": {"count": groups, "keep": keep}})
        got = dict(zip(idx[t].tolist(), w[t].tolist()))
        assert sorted(got) == sorted(want) and len(got) == top
        assert all(abs(got[e] - want[e]) < 1e-5 for e in got)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("groups,dim", [(4, 16), (3, 7), (1, 1), (6, 24)])
def test_one_gate_per_head(dtype, groups, dim):
    from compactor_vllm.layers.latent_attention import group_gate

    g = torch.Generator().manual_seed(1)
    x = torch.randn(9, groups * dim, generator=g).to(dtype).to(DEV)
    cols = (3 * torch.randn(9, groups + 5, generator=g)).to(dtype).to(DEV)
    want = x.double().view(9, groups, dim) * torch.sigmoid(cols[:, 2:2 + groups].double()).unsqueeze(-1)
    tol = dict(rtol=1e-5, atol=1e-6) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    assert torch.allclose(group_gate(x, cols[:, 2:2 + groups]).double(), want.flatten(1), **tol)
    assert group_gate(x, cols[:, 2:2 + groups], out=x) is x                       # in place
    assert torch.allclose(x.double(), want.flatten(1), **tol)


@pytest.mark.parametrize("rank", [1, 5, 16, 40])
@pytest.mark.parametrize("tau", [1.0, 16.0])
def test_decays_from_a_low_rank_product(rank, tau):
    """sigmoid(z)^(1 / tau) with z from far below to far above zero, to fp32 accuracy also close to one."""
    from compactor_vllm import _native as N

    g = torch.Generator().manual_seed(rank)
    for dt in (torch.float32, torch.bfloat16):
        cols = torch.randn(50, rank + 3, generator=g).to(dt).to(DEV)
        w = (4 * torch.randn(300, rank, generator=g)).to(dt).to(DEV)
        b = (20 * torch.randn(300, generator=g)).to(DEV)
        out = torch.empty(50, 300, device=DEV)
        a = cols[:, 2:]
        N.check(N.lib().cvllm_lowrank_decay(N.ptr(a), cols.stride(0), N.ptr(w), N.ptr(b), 1.0 / tau, N.ptr(out), 300, 50, 300,
                                            rank, N.block_dtype_code(dt), N.stream(DEV)), "lowrank_decay")
        z = a[:, :rank].double() @ w.double().T + b.double()
        want = torch.sigmoid(z) ** (1.0 / tau)
        assert torch.allclose(out.double(), want, rtol=1e-4, atol=1e-30)
        near = want > 0.99
        assert near.any() and (out.double() - want)[near].abs().max() < 2e-7


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv,rot", [(4, 2, 16, 8, 16), (3, 1, 12, 10, 6), (2, 2, 7, 5, 4), (6, 3, 128, 64, 128), (1, 1, 1, 1, 0)])
def test_whole_projection_norm_rotation_and_store(dtype, H, G, D, Dv, rot):
    """Heads of very unequal sizes (a norm per head would level them), an eps that counts, positions far out; keys and
    values land in their cache rows and nowhere else, rows of the reserved slot store nothing."""
    from compactor_vllm.layers.attention import BiasedChunkAttention, pair_rotation_frequencies
    from compactor_vllm.config.constants import RESERVED_BATCH
    from compactor_vllm import _native as N
    from oracle import fikudra as O

    g = torch.Generator().manual_seed(H * D)
    eps, PS, T = 0.05, 16, 5
    freq = pair_rotation_frequencies(rot, 300.0, linear_factor=2.0) if rot else None
    a = BiasedChunkAttention(H, G, D, Dv, 1.0, sink=True, rotation=freq, qk_norm=True, row_norm=True, eps=eps).to(DEV)
    a.q_norm_weight.data = (1 + 0.3 * torch.randn(H * D, generator=g)).to(DEV)
    a.k_norm_weight.data = (1 + 0.3 * torch.randn(G * D, generator=g)).to(DEV)
    qkv = torch.randn(T, a.qkv_width + 3, generator=g)
    qkv[:, :D] *= 5.0
    qkv = qkv.to(dtype)
    pos = [0, 37, 38, 39, 9]
    slots = [1, 2, 2, 2, RESERVED_BATCH]
    pages = torch.randperm(3 * G * 3, generator=g).to(torch.int32).view(3, G, 3)
    pos_d, slots_d = (torch.tensor(v, dtype=torch.int32, device=DEV) for v in (pos, slots))
    x, table = qkv.to(DEV), pages.to(DEV)
    for has_kv in (True, False):
        kc, vc = (torch.full((27 * G, PS, n), 7.0, dtype=dtype, device=DEV).view(-1, n) for n in (D, Dv))
        lens = torch.zeros(3, G, dtype=torch.int32, device=DEV)
        q = torch.empty(T, H, D, dtype=dtype, device=DEV)
        N.check(N.lib().cvllm_row_norm_rope_store(
            N.ptr(x), x.stride(0), N.ptr(a.inv_freq), rot, N.ptr(a.q_norm_weight), N.ptr(a.k_norm_weight), eps,
            N.ptr(pos_d), N.ptr(slots_d), N.ptr(q), N.ptr(kc) if has_kv else None, N.ptr(vc), N.ptr(table),
            table.stride(0), table.stride(1), PS, N.ptr(lens), T, H, G, D, Dv, RESERVED_BATCH, N.block_dtype_code(dtype),
            N.stream(DEV)), "row_norm_rope_store")
        rotd = {"base": 300.0, "dims": rot, "scaling": {"factor": 2.0}} if rot else None
        tol = dict(rtol=2e-4, atol=2e-5) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)

        def turned(v, heads, p):
            full = torch.zeros(p + 1, heads, D, dtype=torch.float64)
            full[p] = v.view(heads, D)
            return O.rotate(full, rotd)[p]

        want_k, want_v = kc.new_full(kc.shape, 7.0).double().cpu(), vc.new_full(vc.shape, 7.0).double().cpu()
        for t in range(T):
            qd = O.rms_unit(qkv[t, :H * D], eps) * a.q_norm_weight.double().cpu()
            assert torch.allclose(q[t].cpu().double(), turned(qd, H, pos[t]), **tol), t
            if has_kv and slots[t] != RESERVED_BATCH:
                kd = turned(O.rms_unit(qkv[t, H * D:(H + G) * D], eps) * a.k_norm_weight.double().cpu(), G, pos[t])
                for gg in range(G):
                    r = int(pages[slots[t], gg, pos[t] // PS]) * PS + pos[t] % PS
                    want_k[r] = kd[gg]
                    at = (H + G) * D + gg * Dv
                    want_v[r] = qkv[t, at:at + Dv].double()
        assert torch.allclose(kc.cpu().double(), want_k, **tol) and torch.equal(vc.cpu().double(), want_v)
        assert lens.cpu().tolist() == ([[0] * G, [1] * G, [40] * G] if has_kv else [[0] * G] * 3)


@pytest.mark.parametrize("portions", [True, False])
@pytest.mark.parametrize("mlp", [moe(6, 2, 12, 20, 3, 2, 1.7), moe(5, 3, 12, 0, 0, scale=0.5), moe(8, 4, 8, 8, 4, 2, 1.0)])
def test_routed_experts(portions, mlp):
    from compactor_vllm.config.model_config import GroupedMoEConfig
    from compactor_vllm.models.fikudra import make_experts
    from compactor_vllm.utils.context import reset_context, set_context
    from oracle import fikudra as O

    W, T = 24, 11 if portions else 3
    g = torch.Generator().manual_seed(3)
    m = make_experts(W, GroupedMoEConfig.from_json(mlp), torch.float32).to(DEV)
    E, ff, sf = mlp["router"]["experts"], mlp["expert"]["ff"], (mlp.get("shared") or {}).get("ff", 0)
    t = {"router": 1.5 * torch.randn(E, W, generator=g)}
    for e in [f"e{i}" for i in range(E)] + (["shared"] if sf else []):
        n = sf if e == "shared" else ff
        t[f"{e}.gate"], t[f"{e}.up"] = torch.randn(n, W, generator=g) * 0.3, torch.randn(n, W, generator=g) * 0.3
        t[f"{e}.down"] = torch.randn(W, n, generator=g) * 0.3
    with torch.no_grad():
        m.router[:E].copy_(t["router"])
        for e in range(E):
            m.gate_up[e].copy_(torch.cat([t[f"e{e}.gate"], t[f"e{e}.up"]]))
            m.down[e].copy_(t[f"e{e}.down"])
        if sf:
            t["shared.sg"] = torch.randn(1, W, generator=g)
            m.shared.gate_up_proj.weight.copy_(torch.cat([t["shared.gate"], t["shared.up"]]))
            m.shared.down_proj.weight.copy_(t["shared.down"])
            m.router[E:].copy_(t["shared.sg"])
    h = torch.randn(T, W, generator=g)
    set_context(is_prefill=portions)
    with torch.no_grad():
        got = m(h.to(DEV))
    reset_context()
    assert torch.allclose(got.cpu().double(), O.moe_ff(h, mlp, t, ""), rtol=2e-5, atol=2e-5)


MIXER_CASES = {
    "gla": (gla(3, 12, 10), None),
    "gla_with_experts": (gla(2, 16, 24, 16.0, 4), moe()),
    "gla_one_channel": (gla(2, 1, 1, 2.0, 1), None),
    "gla_wide_key": (gla(1, 130, 20, 16.0, 4), None),
    "gla_wide_value": (gla(2, 6, 200, 16.0, 4), None),
    "gla_odd": (gla(3, 7, 13, 1.0, 3), None),
    "attention": (attn(4, 2, 12, 10), None),
    "attention_with_experts": (attn(4, 4, 16, 16, rot=16), moe()),
    "attention_unrotated": (attn(3, 1, 9, 11, rot=0), None),
    "attention_unscaled_rotation": (attn(2, 1, 32, 16, rot=10, factor=0), None),
}


@pytest.mark.parametrize("name", sorted(MIXER_CASES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mixer_alone(name, dtype):
    """One layer: whole prompt, portions down to two and one tokens, token-by-token decoding."""
    from oracle import fikudra as O

    r, cfg, t = build(model_cfg([MIXER_CASES[name]]), dtype, pages=12, page_size=16)
    toks = tokens(45, 83, 5)
    want = O.forward(cfg, t, toks)
    for sizes in ([45], [2], [1], [7, 1, 16, 3]):
        assert routed_close(run_in_portions(r, toks, sizes), want, dtype), sizes


@pytest.mark.parametrize("layout", [102, 104, 202, 204, 402, 404, 802, 804])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_scan_layouts_give_the_same_numbers(layout, dtype):
    """The scan spreads a head's value columns over a cluster of 1 to 8 CTAs with 2 or 4 columns per thread (some CTAs of
    a cluster may have none); portions shorter and longer than a stage of 32 tokens."""
    from compactor_vllm import _native as N
    from oracle import fikudra as O

    r, cfg, t = build(model_cfg([(gla(2, 64, 64, 16.0, 8), None), (gla(1, 20, 72, 4.0, 3), None), (gla(3, 8, 10, 4.0, 3), None)],
                                width=40), dtype, pages=12)
    toks = tokens(100, 83, 12)
    want = O.forward(cfg, t, toks)
    N.set_test_option("gla_layout", layout)
    try:
        for sizes in ([100], [33, 1, 1, 64], [32]):
            assert close(run_in_portions(r, toks, sizes), want, dtype), sizes
    finally:
        N.set_test_option("gla_layout", 0)


# ----------------------------------------------------------------------------- keys and states that lie far back
@pytest.mark.parametrize("dtype,D", [("float32", 16), ("bfloat16", 16), ("bfloat16", 128), ("float32", 12)])
def test_a_far_key_decides(dtype, D):
    """Sharp unrotated attention whose query projection has one direction, the key of token 82: token 5 looks for it.  The
    key is planted once - at the first position, at a page's last and first place, in the middle - far before the queries.
    The oracle must notice when the planted token is another one; the engine must find it in one portion, in small ones
    and in decoding, over thirteen pages, also through a layer that reads the first one's cache."""
    from oracle import fikudra as O

    a = dict(heads=2, kv_heads=1, dim=D, vdim=D, rot=0)
    cfg0 = model_cfg([(attn(scale=D ** -0.5, **a), None), (attn(kv_from=0, scale=0.9 * D ** -0.5, **a), None)])
    r, cfg, t = build(cfg0, dtype, pages=16, page_size=16)
    t["bigram"] = torch.zeros_like(t["bigram"])
    for q in ("l0.mix.q.norm", "l1.mix.q.norm", "l0.mix.k.norm"):
        t[q] = torch.full_like(t[q], 1.0 if "k" in q[6:] else (2.0 if D < 64 else 1.3))
    streams = [t["embed"].double()[[5, 82]] * cfg["embedding"]["scale"]] * cfg["streams"]
    h5, h82 = O.zero_centred_norm(O.streams_read(streams, t["l0.hc1.in"]), t["l0.norm1"], cfg["norm"]["eps"])
    k82 = O.linear(h82, t["l0.mix.k"])
    for i in range(2):
        t[f"l{i}.mix.q"] = torch.outer(k82, h5 / h5.norm()).repeat(2, 1).to(torch.bfloat16)
    r.model.load_weights(t)
    for at in (0, 15, 16, 101):
        toks = [x % 80 for x in tokens(200, 83, 60 + at)]
        toks[at], toks[-3], toks[-1] = 82, 5, 5
        want = O.forward(cfg, t, toks)
        alt = list(toks)
        alt[at] = 81
        assert rel_err(O.forward(cfg, t, alt)[-3:], want[-3:]) > 0.2, at
        for sizes in ([200], [64, 2, 30], [190, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1]):
            got = run_in_portions(r, toks, sizes)
            # (other tokens' queries point the same way or the opposite one; where the sign is a close call, rounding to
            # bfloat16 decides it)
            assert dtype == "bfloat16" or close(got, want, dtype), (at, sizes)
            assert row_errs(got, want).median() < 0.03 and row_errs(got, want)[[-3, -1]].max() < 0.05, (at, sizes)


def test_state_far_back_reaches_the_last_token():
    """Almost no decay: the first token is still in the state 200 tokens later, through portions and decoding."""
    from oracle import fikudra as O

    r, cfg, t = build(model_cfg([(gla(2, 24, 16, 16.0, 3), None)]), "float32", pages=20)
    t["l0.mix.a2.b"] = torch.full_like(t["l0.mix.a2.b"], 9.0)
    r.model.load_weights(t)
    toks = tokens(200, 83, 17)
    want = O.forward(cfg, t, toks)
    alt = [(toks[0] + 1) % 83] + toks[1:]
    assert (O.forward(cfg, t, alt)[-1] - want[-1]).abs().max().item() > 1e-3
    for sizes in ([200], [2], [16, 1, 33], [199, 1]):
        assert rel_err(run_in_portions(r, toks, sizes), want) < TOL["float32"], sizes


def test_decays_of_every_size():
    """Decay logits from -40 to 40 over the channels: some forget at once, some never."""
    from oracle import fikudra as O

    r, cfg, t = build(model_cfg([(gla(2, 16, 16, 1.0, 3), None), (gla(1, 16, 16, 30.0, 3), None)]), "float32", pages=10)
    for i in range(2):
        n = t[f"l{i}.mix.a2.b"].numel()
        t[f"l{i}.mix.a2.b"] = torch.linspace(-40, 40, n).to(torch.bfloat16)
    r.model.load_weights(t)
    toks = tokens(90, 83, 18)
    want = O.forward(cfg, t, toks)
    for sizes in ([90], [1], [7, 2, 33]):
        assert rel_err(run_in_portions(r, toks, sizes), want) < TOL["float32"], sizes


@pytest.mark.parametrize("scale", [0.002, 0.3, 12.0])
def test_the_sink_counts(scale):
    """Tiny scores (the sink holds one share among the keys: half of it at the first position), large ones (it vanishes).
    The oracle without it gives other logits at the start of a sequence."""
    from oracle import fikudra as O

    r, cfg, t = build(model_cfg([(attn(2, 1, 16, 16, scale=scale), None)]), "float32", pages=8)
    toks = tokens(40, 83, 6)
    want = O.forward(cfg, t, toks)
    real = O.sink_softmax
    O.sink_softmax = lambda s: torch.softmax(s, -1)
    try:
        without = O.forward(cfg, t, toks)
    finally:
        O.sink_softmax = real
    if scale < 1:
        assert rel_err(without[:3], want[:3]) > 1e-2
    for sizes in ([40], [33, 1], [5], [1]):
        assert rel_err(run_in_portions(r, toks, sizes), want) < TOL["float32"], sizes


# ------------------------------------------------------------------- whole prompts, portions, decoding, first tokens
@pytest.mark.parametrize("dtype,cfg", [("float32", config_a), ("float32", config_b), ("bfloat16", config_b),
                                       ("bfloat16", config_a)])
def test_prefill_portions_and_decoding_agree_with_the_oracle(dtype, cfg):
    from oracle import fikudra as O

    r, c, t = build(cfg(), dtype, pages=16, page_size=16)
    toks = tokens(70, c["vocab"], 7)
    want = O.forward(c, t, toks)
    for sizes in ([70], [2], [16], [17, 1, 1, 30], [3, 64]):
        assert routed_close(run_in_portions(r, toks, sizes), want, dtype), sizes
    seq = new_seq()
    out = [feed(r, seq, toks[:1])] + [feed(r, seq, [x]) for x in toks[1:]]
    r.release([seq])
    assert routed_close(torch.cat(out), want, dtype)


def test_sum_of_the_streams_after_every_layer():
    from oracle import fikudra as O

    r, c, t = build(config_a(), "float32", pages=8)
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
    """One-token requests, and the first steps of a request one token at a time (the graph's first replay included):
    the pair table's extra row, a zero state, one key beside the sink.  A slot that held another request comes first."""
    from oracle import fikudra as O

    r, c, t = build(config_a(), "float32", pages=8, eager=eager)
    for seed in (1, 2):
        toks = tokens(4, 83, seed)
        want = O.forward(c, t, toks)
        seq = new_seq()
        out = [feed(r, seq, [x]) for x in toks]
        r.release([seq])
        assert rel_err(torch.cat(out), want) < TOL["float32"]
        assert rel_err(run_in_portions(r, toks[:1], [1]), want[:1]) < TOL["float32"]


@pytest.mark.parametrize("eager", [True, False])
def test_long_decoding_over_pages(eager):
    from oracle import fikudra as O

    r, c, t = build(config_a(), "float32", pages=12, eager=eager)
    toks = tokens(160, 83, 11)
    want = O.forward(c, t, toks)
    seq = new_seq()
    out = [feed(r, seq, toks[:10])] + [feed(r, seq, [x]) for x in toks[10:]]
    r.release([seq])
    if not eager:
        assert r.stats["graph_replays"] == 150
    assert rel_err(torch.cat(out), want) < TOL["float32"]


def test_graph_decode_batches_with_padding_rows():
    """Three decoding requests (padded to four rows in the graph) of unequal lengths, one of which ends early."""
    from oracle import fikudra as O

    r, c, t = build(config_a(), "float32", pages=20, eager=False)
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
        assert rel_err(torch.cat(got[i]), want[i]) < TOL["float32"]


# ---------------------------------------------------------------------------------- batches, pages and slots reused
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_each_request_alone(dtype):
    """Four requests of unequal lengths in one step after another: portions of some beside single tokens of others."""
    from oracle import fikudra as O

    r, c, t = build(config_a() if dtype == "float32" else config_b(), dtype, pages=30)
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
    want = [O.forward(c, t, q) for q in reqs]
    assert routed_close(torch.cat([x for o in outs for x in o]), torch.cat(want), dtype)
    if dtype == "float32":
        assert all(rel_err(torch.cat(o), w) < TOL[dtype] for o, w in zip(outs, want))


@pytest.mark.parametrize("device_allocator", [False, True])
def test_pages_and_slots_are_reused(device_allocator):
    """A pool of 8 pages and 2 slots serves 6 requests, two at a time: every page and state slot is used again by a later
    request - also by a shorter one, whose first tokens must not see what the slot held before."""
    from oracle import fikudra as O

    r, c, t = build(config_a(), "float32", pages=8, max_seqs=2, device_allocator=device_allocator)
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
            assert rel_err(torch.cat(outs[i]), O.forward(c, t, pair[i])) < TOL["float32"], (k, i)
    assert r.kv.num_free_batches == 2


def test_a_request_left_out_of_steps_goes_on_later():
    from oracle import fikudra as O

    r, c, t = build(config_a(), "float32", pages=12)
    a, b = tokens(40, 83, 31), tokens(30, 83, 32)
    sa, sb = new_seq(), new_seq()
    out_a = [feed(r, sa, a[:13])]
    out_b = [feed(r, sb, b[:20]), feed(r, sb, b[20:21]), feed(r, sb, b[21:])]     # a waits meanwhile
    out_a += [feed(r, sa, a[13:14]), feed(r, sa, a[14:])]
    r.release([sa, sb])
    assert rel_err(torch.cat(out_a), O.forward(c, t, a)) < TOL["float32"]
    assert rel_err(torch.cat(out_b), O.forward(c, t, b)) < TOL["float32"]


# ------------------------------------------------------------------------------------------------------ other sizes
OTHER_SIZES = {
    "everything_one": [(attn(1, 1, 1, 1, rot=0), moe(1, 1, 1, 1, 1, 1, 1.0)), (gla(1, 1, 1, 1.0, 1), moe(1, 1, 1, 0, 0)),
                       (attn(1, 1, 1, 1, rot=0, kv_from=0), None)],
    "one_head_per_group": [(attn(5, 5, 8, 8, rot=8), None), (gla(5, 8, 8, 5.0, 4), moe(4, 2, 16, 0, 0))],
    "all_heads_share_one": [(attn(6, 1, 16, 8, rot=4), moe(9, 2, 16, 8, 3, 1, 3.0)), (gla(1, 40, 12, 9.0, 6), None),
                            (attn(6, 1, 16, 8, rot=4, scale=0.1, kv_from=0), moe(2, 1, 8, 8, 2, 1, 1.0))],
    "wide_heads": [(attn(2, 1, 128, 128, rot=128), None), (gla(2, 128, 128, 16.0, 16), moe(8, 2, 32, 64, 2, 1, 2.5)),
                   (gla(1, 256, 256, 16.0, 16), None), (attn(2, 1, 128, 128, rot=128, kv_from=0), None)],
    "key_of_72_value_of_136": [(attn(2, 2, 72, 136, rot=24), None), (gla(1, 72, 136, 7.0, 20), None)],
    "all_experts_chosen": [(gla(2, 8, 16), moe(4, 4, 8, 0, 2, 2, 1.0)), (gla(1, 24, 20), moe(7, 7, 8, 40, 0, 0, 0.3))],
    "recurrent_only": [(gla(4, 32, 16, 16.0, 32), moe(4, 2, 32, 32, 2, 1, 1.5))] * 2,
    "attention_only": [(attn(4, 2, 32, 32, rot=32), None)] * 3,
}


@pytest.mark.parametrize("name", sorted(OTHER_SIZES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(name, dtype):
    from oracle import fikudra as O

    one = name == "everything_one"
    if one and dtype == "bfloat16":
        pytest.skip("the unit norm of a head of one number is its sign: rounding decides it")
    width = {"everything_one": 6, "wide_heads": 128}.get(name, 40)
    streams = {"everything_one": 1, "wide_heads": 2, "recurrent_only": 5}.get(name, 4)
    cfg0 = model_cfg(OTHER_SIZES[name], vocab=37, width=width, eps=3e-6, streams=streams, scale=1.0 if one else 11.0,
                     buckets=1 if one else 53, mul_prev=1 if one else 11)
    r, cfg, t = build(cfg0, dtype, pages=10)
    toks = tokens(50, 37, 9)
    want = O.forward(cfg, t, toks)
    for sizes in ([50], [9, 2, 1]):
        assert routed_close(run_in_portions(r, toks, sizes), want, dtype), sizes
    seq = new_seq()
    out = [feed(r, seq, toks[:31])] + [feed(r, seq, [x]) for x in toks[31:]]
    r.release([seq])
    assert routed_close(torch.cat(out), want, dtype)


def test_heads_of_128_in_pages_of_128():
    """The tcgen05 portion kernel (heads of 128, pages of 128, an even group) with the sink, over several pages, cut in
    the middle of a page; the second layer reads the first one's pages."""
    from oracle import fikudra as O

    a = dict(heads=4, kv_heads=2, dim=128, vdim=128, rot=64, base=10000.0, factor=2.0)
    r, cfg, t = build(model_cfg([(attn(**a), None), (attn(kv_from=0, scale=0.12, **a), None)], width=64), "bfloat16",
                      pages=5, page_size=128)
    toks = tokens(300, 83, 19)
    want = O.forward(cfg, t, toks)
    for sizes in ([300], [129, 2, 100], [290, 1, 1, 1, 7]):
        assert close(run_in_portions(r, toks, sizes), want, "bfloat16"), sizes


def _random_config(seed):
    g = torch.Generator().manual_seed(1000 + seed)
    ri = lambda lo, hi: int(torch.randint(lo, hi + 1, (1,), generator=g))
    layers, own = [], []
    for i in range(ri(2, 6)):
        if ri(0, 1) == 0:
            mixer = gla(ri(1, 4), ri(1, 40), ri(1, 40), float(ri(1, 20)), ri(1, 20))
        elif own and ri(0, 1):
            j, kw = own[ri(0, len(own) - 1)]
            mixer = attn(kv_from=j, scale=0.1 + 0.05 * ri(0, 8), **kw)
        else:
            G, D = ri(1, 3), ri(2, 24)
            kw = dict(heads=G * ri(1, 3), kv_heads=G, dim=D, vdim=ri(1, 24), rot=2 * ri(0, D // 2), base=10.0 ** ri(1, 6),
                      factor=float(ri(0, 8)))
            own.append((i, kw))
            mixer = attn(scale=0.1 + 0.05 * ri(0, 8), **kw)
        groups, size = ri(1, 3), ri(1, 4)
        keep = ri(1, groups)
        mlp = None if ri(0, 3) == 0 else moe(groups * size, ri(1, keep * size), ri(2, 20), ri(0, 1) * ri(2, 24), groups, keep,
                                             0.5 + 0.25 * ri(0, 8))
        layers.append((mixer, mlp))
    return model_cfg(layers, vocab=ri(20, 120), width=ri(8, 70), eps=10.0 ** -ri(4, 7), streams=ri(1, 5),
                     scale=0.5 * ri(1, 40), buckets=ri(2, 300), mul_prev=ri(1, 100000), mul_cur=ri(1, 1000))


@pytest.mark.parametrize("seed", range(12))
def test_models_drawn_at_random(seed):
    """Layer order, every size and every constant drawn at random; whole, in portions, decoding, two in a batch."""
    from oracle import fikudra as O

    r, cfg, t = build(_random_config(seed), "float32", seed=seed, pages=16, max_seqs=2)
    a, b = tokens(57, cfg["vocab"], seed), tokens(23, cfg["vocab"], seed + 50)
    wa, wb = O.forward(cfg, t, a), O.forward(cfg, t, b)
    for sizes in ([57], [5, 1, 2, 30]):
        assert rel_err(run_in_portions(r, a, sizes), wa) < TOL["float32"], sizes
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
    assert rel_err(torch.cat(oa), wa) < TOL["float32"]
    assert rel_err(torch.cat(ob), wb) < TOL["float32"]


# ----------------------------------------------------------------------------------------- the engine's entry point
@pytest.mark.parametrize("eager", [True, False])
def test_greedy_generation_through_llm_generate(eager):
    """`LLM.generate` with the step scheduler: prompts in portions of at most 16 tokens beside decoding requests, five
    requests on three slots, single-token steps from the decode graph.  Teacher forcing against the oracle: every
    generated token must be the oracle's argmax unless the oracle's two best logits are closer than rounding."""
    from compactor_vllm import LLM
    from compactor_vllm.api_types import SamplingParams
    from compactor_vllm.config.engine_config import LLMConfig
    from compactor_vllm.config.model_config import FikudraConfig
    from oracle import fikudra as O

    cfg0 = config_a()
    t, c = random_checkpoint(cfg0, 3), clean(cfg0)
    cfg = LLMConfig(model="synthetic", hf_config=FikudraConfig.from_json(c), dtype="float32", max_num_seqs=3,
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
