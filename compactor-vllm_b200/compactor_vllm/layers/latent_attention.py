"""Latent attention: queries and keys/values pass through low-rank latents, and only the kv latent is cached.

Per token the layer computes, from its input h,
    c_q = RMSnorm(W_dq h) * w_q,   q = W_uq c_q  (per head: `dim` unrotated then `rot_dim` rotated numbers)
    [c | k_r] = W_dkv h,           c <- RMSnorm(c) * w_kv,   k_r <- rotate(k_r)   (one row shared by all heads)
and the cache row of the token is [c | k_r].  Keys and values of head h are W_uk[h] c and W_uv[h] c; they are never
built.  With q_abs[h] = W_uk[h]^T q_plain[h] the score is (q_abs[h] . c + rotate(q_r[h]) . k_r) * scale and the head's
output W_uv[h] (sum_j p_j c_j): attention with ONE key/value head whose key rows have kv_rank + rot_dim numbers and
whose value rows are the first kv_rank of them (`BiasedChunkAttention(values_in_keys=True)`: the engine's paged
portion and decode kernels).  The two per-head changes of basis are batched library GEMMs.  The concatenated heads are
multiplied by sigmoid(W_g h) before the output projection.

A layer built with `source` (another LatentAttention) makes no latent of its own: it attends over the source layer's
cache rows - written earlier in the same step - with its own queries, W_uk, W_uv, gate and output projection.

`DirectLatentAttention` is the form without a query latent for layers that project their input in one product of their
own, with a sliding window, learned sinks and a choice of rotation.

Kernels: csrc/latent_attn.cu (norms + rotation + cache write; query rotation; gate) and csrc/bias_attn.cu.
"""
from __future__ import annotations

from typing import Optional

import torch
from torch import nn

from compactor_vllm import _native as N
from compactor_vllm.config.constants import RESERVED_BATCH
from compactor_vllm.layers.attention import BiasedChunkAttention
from compactor_vllm.utils.context import get_context


def rotation_frequencies(rot_dim: int, base: float) -> torch.Tensor:
    """inv_freq[i] = base ** (-2 i / rot_dim), i < rot_dim / 2, as 64-bit floats."""
    return torch.tensor([float(base) ** (-2.0 * i / rot_dim) for i in range(rot_dim // 2)], dtype=torch.float64)


def sigmoid_gate(x: torch.Tensor, gate: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x * sigmoid(gate), both [T, width] with unit inner stride (row strides free, also of `out` when given)."""
    T, width = x.shape
    assert gate.shape == x.shape and x.stride(1) == 1 and gate.stride(1) == 1 and gate.dtype == x.dtype
    if out is None:
        out = torch.empty((T, width), dtype=x.dtype, device=x.device)
    assert out.shape == x.shape and out.stride(1) == 1 and out.dtype == x.dtype
    N.check(N.lib().cvllm_sigmoid_gate(N.ptr(x), x.stride(0), N.ptr(gate), gate.stride(0), N.ptr(out), out.stride(0), T,
                                       width, N.block_dtype_code(x.dtype), N.stream(x.device)), "cvllm_sigmoid_gate")
    return out


def group_gate(x: torch.Tensor, gate: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [T, groups * dim] times sigmoid(gate [T, groups]), one gate for each group of neighbouring columns (a head); row
    strides free, `out` may be x."""
    T, width = x.shape
    groups = gate.shape[1]
    assert gate.shape[0] == T and width % groups == 0 and x.stride(1) == 1 and gate.stride(1) == 1
    assert gate.dtype == x.dtype
    if out is None:
        out = torch.empty((T, width), dtype=x.dtype, device=x.device)
    assert out.shape == x.shape and out.stride(1) == 1 and out.dtype == x.dtype
    N.check(N.lib().cvllm_group_gate(N.ptr(x), x.stride(0), N.ptr(gate), gate.stride(0), N.ptr(out), out.stride(0), T,
                                     groups, width // groups, N.block_dtype_code(x.dtype), N.stream(x.device)),
            "cvllm_group_gate")
    return out


def absorb_queries(q: torch.Tensor, uk: torch.Tensor, q_full: torch.Tensor) -> None:
    """q_full[t, h, :r] = q[t, h, :dim] W_uk[h] for uk [H, dim, r]: [H, T, dim] x [H, dim, r] into the first r columns of
    the attention's query rows."""
    dim, r = uk.shape[1], uk.shape[2]
    torch.bmm(q[:, :, :dim].transpose(0, 1), uk, out=q_full[:, :, :r].transpose(0, 1))


def expand_values(o_lat: torch.Tensor, uv: torch.Tensor) -> torch.Tensor:
    """o_lat [T, H, r] (the heads' weighted latents), uv [H, vdim, r] -> [T, H * vdim]."""
    o = torch.empty((o_lat.shape[0], uv.shape[0], uv.shape[1]), dtype=o_lat.dtype, device=o_lat.device)
    torch.bmm(o_lat.transpose(0, 1), uv.transpose(1, 2), out=o.transpose(0, 1))
    return o.flatten(1)


class DirectLatentAttention(nn.Module):
    """Latent attention whose queries come straight from the layer's input (no query latent), for layers that bring the
    projections of their input themselves: `forward` takes the columns [q | latent and shared key part | gate] of that
    projection and writes the gated, concatenated heads to `out`; the output projection is the layer's as well.

    Options beside `LatentAttention`'s: `window` (sliding window), `learned_sink` (one more term exp(sink_h) in every
    head's denominator), `inv_freq` (rotation frequencies, rot_dim / 2 64-bit floats), `amplitude` (a factor on sine and
    cosine), `neighbours` (number 2 i turns with 2 i + 1 instead of i with i + rot_dim / 2).  The cache views and the
    sink live in `attn`, so that several runs of one layer can share the weights (`attn.twin()`)."""

    def __init__(self, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, scale: float, eps: float, *,
                 inv_freq: torch.Tensor, amplitude: float = 1.0, neighbours: bool = False, window: int = 0,
                 learned_sink: bool = False, gate: bool = True, dtype: Optional[torch.dtype] = None):
        super().__init__()
        assert inv_freq.dtype == torch.float64 and 2 * inv_freq.numel() == rot_dim
        self.heads, self.dim, self.rot_dim, self.vdim = int(heads), int(dim), int(rot_dim), int(vdim)
        self.kv_rank, self.eps = int(kv_rank), float(eps)
        self.amplitude, self.neighbours, self.gate = float(amplitude), bool(neighbours), bool(gate)
        self.row = self.kv_rank + self.rot_dim     # numbers per cache row
        self.attn = BiasedChunkAttention(self.heads, 1, self.row, self.kv_rank, scale, values_in_keys=True,
                                         sink=learned_sink, learned_sink=learned_sink, window=window)
        self.out_width = self.heads * self.vdim
        self.in_parts = [("q", self.heads * (self.dim + self.rot_dim)), ("dkv", self.row)]
        if self.gate:
            self.in_parts.append(("g", self.out_width))
        self.in_cols = sum(n for _, n in self.in_parts)
        self.kv_norm = nn.Parameter(torch.ones(self.kv_rank, dtype=torch.float32))
        self.uk = nn.Parameter(torch.empty(self.heads, self.dim, self.kv_rank, dtype=dtype))
        self.uv = nn.Parameter(torch.empty(self.heads, self.vdim, self.kv_rank, dtype=dtype))
        self.register_buffer("inv_freq", inv_freq.contiguous(), persistent=False)

    def forward(self, cols: torch.Tensor, attn: BiasedChunkAttention, out: torch.Tensor) -> None:
        ctx = get_context()
        assert attn.k_cache is not None, "KV cache must be initialized"
        assert cols.shape[1] == self.in_cols and cols.stride(1) == 1
        T, H, D, R, r = cols.shape[0], self.heads, self.dim, self.rot_dim, self.kv_rank
        kv_off = H * (D + R)
        q_full = torch.empty((T, H, self.row), dtype=cols.dtype, device=cols.device)
        pt = attn.page_table
        N.check(N.lib().cvllm_latent_prepare(
            N.ptr(cols), cols.stride(0), 0, H, D, kv_off, r, R, N.ptr(self.kv_norm), self.eps, N.ptr(self.inv_freq),
            self.amplitude, int(self.neighbours), N.ptr(ctx.positions_i32), N.ptr(ctx.token_slot), N.ptr(q_full),
            q_full.stride(0), self.row, r, N.ptr(attn.k_cache), N.ptr(pt), pt.stride(0), int(attn.page_size),
            N.ptr(attn.bh_seq_lens), T, RESERVED_BATCH, N.block_dtype_code(cols.dtype), N.stream(cols.device)),
            "cvllm_latent_prepare")
        absorb_queries(cols[:, :kv_off].unflatten(1, (H, D + R)), self.uk, q_full)
        o = expand_values(attn.attend(q_full, flat=False), self.uv)
        if self.gate:
            sigmoid_gate(o, cols[:, kv_off + self.row:], out)
        else:
            out.copy_(o)


class LatentAttention(nn.Module):
    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, q_rank: int,
                 scale: float, rot_base: float, eps: float, source: Optional["LatentAttention"] = None,
                 dtype: Optional[torch.dtype] = None):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim = int(heads), int(dim), int(rot_dim), int(vdim)
        self.kv_rank, self.q_rank, self.eps = int(kv_rank), int(q_rank), float(eps)
        self.own_latent = source is None
        self.__dict__["source"] = source          # not a submodule: its parameters belong to its own layer
        if source is not None:
            assert (source.kv_rank, source.rot_dim) == (self.kv_rank, self.rot_dim) and source.own_latent
        self.row = self.kv_rank + self.rot_dim     # numbers per cache row
        # the paged attention over the latent rows; a layer without a latent of its own borrows the source's cache views
        self.attn = BiasedChunkAttention(self.heads, 1, self.row, self.kv_rank, scale, values_in_keys=True)
        kv_cols = self.row if self.own_latent else 0
        self.q_off, self.kv_off, self.g_off = 0, (self.q_rank if self.own_latent else -1), self.q_rank + kv_cols
        self.in_proj = nn.Linear(width, self.q_rank + kv_cols + self.heads * self.vdim, bias=False)   # dq | dkv | gate
        self.q_norm = nn.Parameter(torch.ones(self.q_rank, dtype=torch.float32))
        self.kv_norm = nn.Parameter(torch.ones(self.kv_rank, dtype=torch.float32)) if self.own_latent else None
        self.uq_proj = nn.Linear(self.q_rank, self.heads * (self.dim + self.rot_dim), bias=False)
        self.uk = nn.Parameter(torch.empty(self.heads, self.dim, self.kv_rank, dtype=dtype))
        self.uv = nn.Parameter(torch.empty(self.heads, self.vdim, self.kv_rank, dtype=dtype))
        self.o_proj = nn.Linear(self.heads * self.vdim, width, bias=False)
        self.register_buffer("inv_freq", rotation_frequencies(self.rot_dim, rot_base), persistent=False)

    def _cache(self) -> BiasedChunkAttention:
        a = self.attn
        if not self.own_latent and a.k_cache is None:
            s = self.source.attn
            a.k_cache, a.page_table, a.bh_seq_lens, a.page_size = s.k_cache, s.page_table, s.bh_seq_lens, s.page_size
        assert a.k_cache is not None, "KV cache must be initialized"
        return a

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        ctx = get_context()
        attn = self._cache()
        T = h.shape[0]
        H, D, R, r = self.heads, self.dim, self.rot_dim, self.kv_rank
        dev, lib, st = h.device, N.lib(), N.stream(h.device)
        proj = self.in_proj(h)
        code = N.block_dtype_code(proj.dtype)
        cq = torch.empty((T, self.q_rank), dtype=proj.dtype, device=dev)
        pt = attn.page_table
        N.check(lib.cvllm_latent_norm_store(
            N.ptr(proj), proj.stride(0), self.q_off, self.q_rank, self.kv_off, r, R, N.ptr(self.q_norm),
            N.ptr(self.kv_norm), self.eps, N.ptr(self.inv_freq), N.ptr(ctx.positions_i32), N.ptr(ctx.token_slot),
            N.ptr(cq), N.ptr(attn.k_cache), N.ptr(pt), pt.stride(0), int(attn.page_size), N.ptr(attn.bh_seq_lens), T,
            RESERVED_BATCH, code, st), "cvllm_latent_norm_store")
        q = self.uq_proj(cq).view(T, H, D + R)
        q_full = torch.empty((T, H, self.row), dtype=proj.dtype, device=dev)
        absorb_queries(q, self.uk, q_full)
        N.check(lib.cvllm_latent_q_rope(N.ptr(q), q.stride(0), H, D, R, N.ptr(self.inv_freq), N.ptr(ctx.positions_i32),
                                        N.ptr(q_full), q_full.stride(0), self.row, r, T, code, st), "cvllm_latent_q_rope")
        o_lat = attn.attend(q_full, flat=False)           # [T, H, r], possibly a view of wider rows
        return self.o_proj(sigmoid_gate(expand_values(o_lat, self.uv), proj[:, self.g_off:]))
