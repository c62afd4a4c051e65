"""Pekasun: a decoder whose layers run their mixer and their feed-forward side by side on ONE RMS-normed input,

    x = norm(embed[token]);   per layer:  h = norm(x),  x += mixer(h) + ff(h);   logits = head(norm(x))

on a 32-bit residual stream; the gain of every norm of the stream is a single number.  A layer may use the weights of
another layer (mixer, feed-forward and norm) with a cache of its own.

Built from the engine's blocks:
  * embedding and its norm, together with the first layer's norm = `embed_norm`; every other norm is one `residual_norm`
    launch (NORM_RMS_ONE_GAIN): the residual sum of the layer before and the norm in front of this one, also into the
    final norm (layers/layernorm.py);
  * mixer "attention" = `BiasedChunkAttention` (layers/attention.py): no rotation, q and k normed with a weight, values
    normed without one, a sliding window beside which the first tokens stay visible;
  * mixer "latent_attention" = `DirectLatentAttention` (layers/latent_attention.py): one cached latent row per token,
    neighbouring pairs rotated with YaRN's frequencies, a sliding window, learned sinks, a sigmoid gate on the heads;
  * feed-forward = down(silu(gate h) * up h), or none;
  * ONE GEMM for everything that reads h (`in_proj`: the mixer's columns, then gate | up) and ONE for everything that
    returns to the stream (`out_proj` = [W_o | W_down] on [heads | activated ff], which the mixer and `gated_act` write
    side by side): the sum of both sublayers is made in the product's 32-bit accumulator.
Weights: `load_weights` takes the checkpoint's tensors (`embed`, `embed.norm`, `final.norm`, `head`, `l<i>.norm1`,
attention `l<i>.mix.q|k|v|q.norm|k.norm|o`, latent_attention `l<i>.mix.q|dkv|dkv.norm|uk|uv|sink|g|o`,
`l<i>.mlp.gate|up|down`); `init_synthetic_weights` draws random ones.
"""
from __future__ import annotations

import sys
from typing import Dict, List, Optional

import torch
from torch import nn

from compactor_vllm.config.model_config import PekasunConfig
from compactor_vllm.layers.attention import BiasedChunkAttention, yarn_amplitude, yarn_rotation_frequencies
from compactor_vllm.layers.latent_attention import DirectLatentAttention, rotation_frequencies
from compactor_vllm.layers.layernorm import NORM_RMS_ONE_GAIN, NormWeight, embed_norm, residual_norm
from compactor_vllm.layers.moe import ACT_SILU, gated_act
from compactor_vllm.utils.context import get_context


def make_latent_attention(a, eps: float, dtype) -> DirectLatentAttention:
    if a.rot_scaling is None:
        freq, amp = rotation_frequencies(a.rot_dim, a.rot_base), 1.0
    else:
        freq, amp = yarn_rotation_frequencies(a.rot_dim, a.rot_base, *a.rot_scaling), yarn_amplitude(a.rot_scaling[0])
    return DirectLatentAttention(a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.scale, eps, inv_freq=freq, amplitude=amp,
                                 neighbours=True, window=a.window, learned_sink=True, dtype=dtype)


class WindowAttentionMixer(nn.Module):
    """The q | k | v columns of the layer's input projection -> norms, cache, paged attention -> the heads in `out`."""

    def __init__(self, a, eps: float):
        super().__init__()
        self.attn = BiasedChunkAttention(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, qk_norm=True, eps=eps,
                                         window=a.window, keep_first=a.keep_first, value_norm=True)
        self.in_parts = [("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)]
        self.in_cols, self.out_width = self.attn.qkv_width, a.heads * a.vdim

    def forward(self, cols: torch.Tensor, attn: BiasedChunkAttention, out: torch.Tensor) -> None:
        attn(cols, out)


class PekasunLayer(nn.Module):
    """The weights of a layer; `attn` of `forward` holds the cache views of the run (several runs may share weights)."""

    def __init__(self, cfg: PekasunConfig, index: int, dtype):
        super().__init__()
        lc = cfg.layers[index]
        W, eps = cfg.hidden_size, cfg.rms_norm_eps
        self.kind = lc.mixer_type
        self.mixer = (WindowAttentionMixer(lc.mixer, eps) if self.kind == "attention"
                      else make_latent_attention(lc.mixer, eps, dtype))
        self.ff = 0 if lc.mlp is None else int(lc.mlp.ff)
        self.norm1 = NormWeight(1)
        self.in_proj = nn.Linear(W, self.mixer.in_cols + 2 * self.ff, bias=False)
        self.out_proj = nn.Linear(self.mixer.out_width + self.ff, W, bias=False)

    def forward(self, h: torch.Tensor, attn: BiasedChunkAttention) -> torch.Tensor:
        """h = the normed input -> mixer(h) + ff(h)."""
        cols, n, m = self.in_proj(h), self.mixer.in_cols, self.mixer.out_width
        width = m + self.ff
        # rows padded to 16 bytes whatever the sizes: the kernels that write both halves keep their wide stores
        y = torch.empty((h.shape[0], -(-width // 8) * 8), dtype=h.dtype, device=h.device)[:, :width]
        self.mixer(cols[:, :n], attn, y[:, :m])
        if self.ff:
            gated_act(cols[:, n:], ACT_SILU, out=y[:, m:])
        return self.out_proj(y)


class PekasunForCausalLM(nn.Module):
    mixed_steps = True        # the runner may hand it portions of prompts beside single tokens in one step

    def __init__(self, cfg: PekasunConfig):
        super().__init__()
        self.config = cfg
        dtype = torch.get_default_dtype()
        W = cfg.hidden_size
        self.embed_tokens = nn.Embedding(cfg.vocab_size, W)
        self.embed_norm = NormWeight(1)
        # weights once per owner; a run of a layer is (its owner's weights, an attention object with its own cache views)
        self.layers = nn.ModuleDict({str(i): PekasunLayer(cfg, i, dtype) for i, lc in enumerate(cfg.layers)
                                     if lc.owner == i})
        self.runs = [(str(lc.owner), self.layers[str(lc.owner)].mixer.attn if lc.owner == i
                      else self.layers[str(lc.owner)].mixer.attn.twin()) for i, lc in enumerate(cfg.layers)]
        self.norm = NormWeight(1)
        self.lm_head = nn.Linear(W, cfg.vocab_size, bias=False)
        self.debug_residuals: Optional[list] = None   # a list collects the residual stream after every layer

    # ---- what the cache manager asks ----------------------------------------------------------------------
    def cache_specs(self):
        """One entry per layer: (attention object, kv heads, key row size, value row size); the values of latent rows are
        columns of the key rows (value row size 0)."""
        return [(a, a.num_kv_heads, a.head_dim, 0 if a.values_in_keys else a.v_head_dim) for _, a in self.runs]

    # ---- forward ----------------------------------------------------------------------------------------------
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        eps = self.config.rms_norm_eps
        dtype = self.lm_head.weight.dtype
        gains: List[torch.Tensor] = [self.layers[owner].norm1.weight for owner, _ in self.runs] + [self.norm.weight]
        x, h = embed_norm(input_ids, self.embed_tokens.weight, self.embed_norm.weight, next_weight=gains[0], eps=eps,
                          out_dtype=dtype)
        for i, (owner, attn) in enumerate(self.runs):
            y = self.layers[owner](h, attn)
            h = residual_norm(x, add=(y,), weight=gains[i + 1], eps=eps, kind=NORM_RMS_ONE_GAIN, out_dtype=dtype)
            if self.debug_residuals is not None:
                self.debug_residuals.append(x.clone())
        return h

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

        def put(param, *names, shape=None, dim=0):
            src = torch.cat([get(n) for n in names], dim=dim) if len(names) > 1 else get(names[0])
            if shape is not None:
                if src.numel() != param.numel():
                    raise ValueError(f"{names}: {tuple(src.shape)} does not fit {tuple(param.shape)}")
                src = src.reshape(shape)
            if tuple(src.shape) != tuple(param.shape):
                raise ValueError(f"{names}: shape {tuple(src.shape)} does not fit {tuple(param.shape)}")
            param.copy_(src.to(param.dtype))

        put(self.embed_tokens.weight, "embed")
        put(self.embed_norm.weight, "embed.norm", shape=(1,))
        put(self.norm.weight, "final.norm", shape=(1,))
        put(self.lm_head.weight, "head")
        for i, layer in self.layers.items():
            p, mx = f"l{i}.", layer.mixer
            put(layer.norm1.weight, p + "norm1", shape=(1,))
            ff = ["gate", "up"] if layer.ff else []
            put(layer.in_proj.weight, *[p + "mix." + n for n, _ in mx.in_parts], *[p + "mlp." + n for n in ff])
            put(layer.out_proj.weight, p + "mix.o", *([p + "mlp.down"] if layer.ff else []), dim=1)
            if layer.kind == "attention":
                put(mx.attn.q_norm_weight, p + "mix.q.norm")
                put(mx.attn.k_norm_weight, p + "mix.k.norm")
            else:
                put(mx.kv_norm, p + "mix.dkv.norm")
                put(mx.uk, p + "mix.uk", shape=mx.uk.shape)
                put(mx.uv, p + "mix.uv", shape=mx.uv.shape)
                put(mx.attn.sink_logits, p + "mix.sink")
        extra = sorted(set(tensors) - used)
        if extra:
            print(f"pekasun: {len(extra)} checkpoint tensors are not used: {extra[:8]}", file=sys.stderr)

    @torch.no_grad()
    def init_synthetic_weights(self, seed: int = 0) -> None:
        """Random weights drawn on the parameters' device: matrices N(0, 1/fan_in), norm gains near 1, small sinks."""
        for i, (name, p) in enumerate(self.named_parameters()):
            gen = torch.Generator(device=p.device).manual_seed(seed * 100003 + i)
            val = torch.randn(p.shape, generator=gen, device=p.device, dtype=torch.float32)
            leaf = name.rsplit(".", 1)[-1]
            if name.endswith("embed_tokens.weight"):
                pass
            elif leaf == "sink_logits":
                val = 0.5 * val
            elif p.dim() == 1:
                val = 1.0 + 0.1 * val
            else:
                val = val * (p.shape[-1] ** -0.5)
            p.copy_(val.to(p.dtype))
