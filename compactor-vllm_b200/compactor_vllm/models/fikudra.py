"""Fikudra: a decoder whose residual is several parallel 32-bit streams that pass into one another around every sublayer,

    x_1 = .. = x_s = embed[token] * scale + pair[hash(previous token, token)]
    per layer, for the mixer and then (if the layer has one) the feed-forward:
        u = sum_s in[s] x_s;   y = sublayer(rms_norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y
    logits = head(rms_norm(sum_s x_s))

with norms whose gains are stored around zero (gain = 1 + w), two kinds of mixer in any order and a routed feed-forward.

Built from the engine's blocks:
  * embedding = `HashedPairEmbedding` (layers/pair_embedding.py) with a factor on the token's row, the previous token in
    the state pool;
  * mixer "gla" = `GatedLinearMixer` (layers/recurrent.py), its state in the state pool;
  * mixer "attention" = `BiasedChunkAttention` (layers/attention.py) with norms over the whole q and k projections, a
    rotation of neighbouring pairs and a sink of score 0, each head's output behind a gate of its own (`group_gate`); a
    layer with `kv_from` reads the cached keys and values of an earlier layer and owns no cache layer;
  * feed-forward = `RoutedExperts` (layers/moe.py) with ROUTE_SIGMOID_GROUPS routing and a shared expert behind one gate
    logit per token;
  * everything between two sublayers is one `stream_mix_norm` launch (layers/layernorm.py): the first one's way back into
    the streams, the second one's read and norm; also into the final norm.
Everything that reads a mixer's input rides in ONE GEMM (`in_proj`, its columns padded to a multiple of 8).  Weights:
`load_weights` takes the checkpoint's tensors (`embed`, `bigram`, `final.norm`, `head`, `l<i>.norm1|norm2`,
`l<i>.hc1|hc2.in|mix|out`, gla `l<i>.mix.q|k|v|g|a1|a2|a2.b|norm|o`, attention `l<i>.mix.q|q.norm|k|k.norm|v|g|o`,
`l<i>.mlp.router`, `l<i>.mlp.e<j>.gate|up|down`, `l<i>.mlp.shared.gate|up|down|sg`); `init_synthetic_weights` draws random
ones.
"""
from __future__ import annotations

import sys
from typing import Dict, List, Optional

import torch
from torch import nn

from compactor_vllm.config.model_config import FikudraConfig, GroupedMoEConfig
from compactor_vllm.layers.attention import BiasedChunkAttention, pair_rotation_frequencies
from compactor_vllm.layers.latent_attention import group_gate
from compactor_vllm.layers.layernorm import NormWeight, StreamCoefficients, stream_mix_norm
from compactor_vllm.layers.moe import ACT_SILU, ROUTE_SIGMOID_GROUPS, RoutedExperts
from compactor_vllm.layers.pair_embedding import HashedPairEmbedding
from compactor_vllm.layers.recurrent import GatedLinearMixer
from compactor_vllm.utils.context import get_context

GAIN_OFFSET = 1.0     # every norm between sublayers and the final one: gain = 1 + stored weight


def padded_linear(width: int, cols: int, like: Optional[nn.Linear] = None) -> nn.Linear:
    """A projection with its output columns rounded up to a multiple of 8 (16-byte rows); the pad's weights are zero."""
    where = {} if like is None else dict(device=like.weight.device, dtype=like.weight.dtype)
    lin = nn.Linear(width, -(-cols // 8) * 8, bias=False, **where)
    nn.init.zeros_(lin.weight[cols:])
    return lin


class GatedAttentionMixer(nn.Module):
    """[q | k | v | one gate logit per head] columns of the layer's input projection -> norms, rotation, cache, paged
    attention, the heads' gates, W_o.  `source`: the mixer whose keys and values are read (then [q | gate logits])."""

    def __init__(self, width: int, a, eps: float, source: Optional["GatedAttentionMixer"]):
        super().__init__()
        rot = (pair_rotation_frequencies(a.rot_dims, a.rot_base, linear_factor=a.rot_factor) if a.rot_dims > 0 else None)
        self.attn = BiasedChunkAttention(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, sink=True, rotation=rot, qk_norm=True,
                                         row_norm=True, eps=eps, source=None if source is None else source.attn)
        self.in_parts = [("q", a.heads * a.dim)]
        if source is None:
            self.in_parts += [("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)]
        self.in_parts.append(("g", a.heads))
        self.in_cols = sum(n for _, n in self.in_parts)
        self.o_proj = nn.Linear(a.heads * a.vdim, width, bias=False)

    def forward(self, cols: torch.Tensor, state=None) -> torch.Tensor:
        n = self.attn.qkv_width
        o = self.attn(cols[:, :n])
        return self.o_proj(group_gate(o, cols[:, n:self.in_cols], out=o))


def make_experts(width: int, m: Optional[GroupedMoEConfig], dtype) -> Optional[RoutedExperts]:
    if m is None:
        return None
    return RoutedExperts(width, m.ff, m.experts, 0, m.top, m.groups, m.keep, m.shared_ff, ACT_SILU, dtype,
                         route_mode=ROUTE_SIGMOID_GROUPS, route_scale=m.route_scale, shared_gate=bool(m.shared_ff))


class FikudraLayer(nn.Module):
    def __init__(self, cfg: FikudraConfig, index: int, layers: List["FikudraLayer"], dtype):
        super().__init__()
        lc = cfg.layers[index]
        W, eps, a = cfg.hidden_size, cfg.rms_norm_eps, lc.mixer
        self.kind = lc.mixer_type
        if self.kind == "gla":
            self.mixer = GatedLinearMixer(W, a.heads, a.dim, a.vdim, a.tau, a.decay_rank, eps)
        else:
            self.mixer = GatedAttentionMixer(W, a, eps, None if a.kv_from is None else layers[a.kv_from].mixer)
        self.state = self.mixer.make_state() if self.kind == "gla" else None
        self.in_proj = padded_linear(W, self.mixer.in_cols)
        self.norm1, self.hc1 = NormWeight(W), StreamCoefficients(cfg.streams)
        self.mlp = make_experts(W, lc.mlp, dtype)
        if self.mlp is not None:
            self.norm2, self.hc2 = NormWeight(W), StreamCoefficients(cfg.streams)


class FikudraForCausalLM(nn.Module):
    mixed_steps = True        # the runner may hand it portions of prompts beside single tokens in one step

    def __init__(self, cfg: FikudraConfig):
        super().__init__()
        self.config = cfg
        dtype = torch.get_default_dtype()
        W = cfg.hidden_size
        self.embed = HashedPairEmbedding(cfg.vocab_size, W, cfg.buckets, cfg.mul_prev, cfg.mul_cur, cfg.embedding_scale)
        layers: List[FikudraLayer] = []
        for i in range(len(cfg.layers)):
            layers.append(FikudraLayer(cfg, i, layers, dtype))
        self.layers = nn.ModuleList(layers)
        self.norm = NormWeight(W)
        self.lm_head = nn.Linear(W, cfg.vocab_size, bias=False)
        self.debug_residuals: Optional[list] = None   # a list collects the sum of the streams after every layer

    # ---- what the cache manager asks ----------------------------------------------------------------------
    def cache_specs(self):
        """One entry per cache layer (= attention layer with keys of its own): (attention module, kv heads, key size,
        value size)."""
        return [(a, a.num_kv_heads, a.head_dim, a.v_head_dim)
                for a in (l.mixer.attn for l in self.layers if l.kind == "attention") if a.source is None]

    def state_layers(self):
        """Everything that carries state between steps in slots of the state pool: the embedding's previous token and
        the recurrent layers' matrices."""
        return [self.embed] + [l.state for l in self.layers if l.state is not None]

    # ---- forward ----------------------------------------------------------------------------------------------
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        cfg = self.config
        eps, S = cfg.rms_norm_eps, cfg.streams
        dtype = self.lm_head.weight.dtype
        src = self.embed(input_ids)            # fp32 [T, W]: S equal streams until the first sublayer has returned
        streams = torch.empty((src.shape[0], S, src.shape[1]), dtype=torch.float32, device=src.device)
        branch = coeff = None                  # the last sublayer's output and its coefficients, not yet in the streams
        for layer in self.layers:
            subs = [(layer.norm1, layer.hc1, lambda h, l=layer: l.mixer(l.in_proj(h), l.state))]
            if layer.mlp is not None:
                subs.append((layer.norm2, layer.hc2, layer.mlp))
            for norm, hc, sublayer in subs:
                h = stream_mix_norm(src, S, branch=branch, coeff=coeff, dst=None if branch is None else streams,
                                    w_in=hc.w_in, weight=norm.weight, gain_offset=GAIN_OFFSET, eps=eps, out_dtype=dtype)
                if branch is not None:
                    src = streams
                branch, coeff = sublayer(h), hc
            if self.debug_residuals is not None:
                stream_mix_norm(src, S, branch=branch, coeff=coeff, dst=streams)
                src, branch, coeff = streams, None, None
                self.debug_residuals.append(streams.sum(dim=1))
        # the streams themselves are not needed any more: their sum goes straight through the final norm
        return stream_mix_norm(src, S, branch=branch, coeff=coeff, weight=self.norm.weight, gain_offset=GAIN_OFFSET,
                               eps=eps, out_dtype=dtype)

    def compute_logits(self, hidden_states: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Logits of the given rows of the step (None: the last token of every sequence of the step)."""
        if rows is None:
            rows = get_context().cu_seqlens_q[1:].long() - 1
        return self.lm_head(hidden_states.index_select(0, rows))

    # ---- weights ----------------------------------------------------------------------------------------------
    @torch.no_grad()
    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        used = set()

        def get(name):
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            used.add(name)
            return tensors[name]

        def put(param, *names, shape=None):
            src = torch.cat([get(n) for n in names], dim=0) if len(names) > 1 else get(names[0])
            if shape is not None:
                if src.numel() != param.numel():
                    raise ValueError(f"{names}: {tuple(src.shape)} does not fit {tuple(param.shape)}")
                src = src.reshape(shape)
            if tuple(src.shape) != tuple(param.shape):
                raise ValueError(f"{names}: shape {tuple(src.shape)} does not fit {tuple(param.shape)}")
            param.copy_(src.to(param.dtype))

        put(self.embed.tokens.weight, "embed")
        put(self.embed.pairs.weight, "bigram")
        put(self.norm.weight, "final.norm")
        put(self.lm_head.weight, "head")
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            for tag in ("1", "2") if layer.mlp is not None else ("1",):
                put(getattr(layer, "norm" + tag).weight, p + "norm" + tag)
                hc = getattr(layer, "hc" + tag)
                put(hc.w_in, p + f"hc{tag}.in")
                put(hc.mix, p + f"hc{tag}.mix")
                put(hc.w_out, p + f"hc{tag}.out")
            mx, q = layer.mixer, p + "mix."
            if layer.kind == "gla":
                rank = get(q + "a1").shape[0]
                if rank != dict(mx.in_parts)["a1"]:      # the decay's inner size comes with the checkpoint
                    mx.set_decay_rank(rank)
                    layer.in_proj = padded_linear(layer.in_proj.in_features, mx.in_cols, like=layer.in_proj)
                put(mx.a2.weight, q + "a2")
                put(mx.a2_bias, q + "a2.b")
                put(mx.norm_weight, q + "norm")
            else:
                put(mx.attn.q_norm_weight, q + "q.norm")
                if mx.attn.source is None:
                    put(mx.attn.k_norm_weight, q + "k.norm")
            layer.in_proj.weight[mx.in_cols:].zero_()
            put(layer.in_proj.weight[:mx.in_cols], *[q + n for n, _ in mx.in_parts])
            put(mx.o_proj.weight, q + "o")
            mlp, f = layer.mlp, p + "mlp."
            if mlp is None:
                continue
            E = mlp.n_real
            mlp.router[:E].copy_(get(f + "router").float())
            for e in range(E):
                put(mlp.gate_up[e], f + f"e{e}.gate", f + f"e{e}.up")
                put(mlp.down[e], f + f"e{e}.down")
            if mlp.shared is not None:
                put(mlp.shared.gate_up_proj.weight, f + "shared.gate", f + "shared.up")
                put(mlp.shared.down_proj.weight, f + "shared.down")
                mlp.router[E:].copy_(get(f + "shared.sg").float().reshape(1, -1))
        extra = sorted(set(tensors) - used)
        if extra:
            print(f"fikudra: {len(extra)} checkpoint tensors are not used: {extra[:8]}", file=sys.stderr)

    @torch.no_grad()
    def init_synthetic_weights(self, seed: int = 0) -> None:
        """Random weights drawn on the parameters' device: matrices N(0, 1/fan_in), norm weights near their neutral value,
        streams that mostly keep to themselves, decays in the range where the state neither dies nor saturates."""
        S = self.config.streams
        for i, (name, p) in enumerate(self.named_parameters()):
            gen = torch.Generator(device=p.device).manual_seed(seed * 100003 + i)
            val = torch.randn(p.shape, generator=gen, device=p.device, dtype=torch.float32)
            leaf = name.rsplit(".", 1)[-1]
            if name.startswith("embed."):
                val = val * (0.5 if "pairs" in name else 1.0 / max(self.embed.scale, 1e-6))
            elif leaf in ("norm_weight", "q_norm_weight", "k_norm_weight"):
                val = 1.0 + 0.1 * val
            elif leaf == "weight" and p.dim() == 1:
                val = 0.1 * val
            elif leaf == "w_in":
                val = (1.0 + 0.3 * val) / S
            elif leaf == "w_out":
                val = 1.0 + 0.3 * val
            elif leaf == "mix":
                val = torch.eye(S, device=p.device) + (0.1 / S) * val
            elif leaf == "a2_bias":
                val = 1.0 + val
            else:
                val = val * (p.shape[-1] ** -0.5)
            p.copy_(val.to(p.dtype))
        for layer in self.layers:
            layer.in_proj.weight[layer.mixer.in_cols:].zero_()
