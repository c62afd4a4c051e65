// Attention over latent rows on tcgen05 / TMEM / TMA: ONE key/value head whose values are the first Dv columns of its key
// rows (D <= 576, Dv <= 512, bfloat16 storage, pages that are multiples of 64 rows).  Portions of prompts and single
// decoded tokens run the same kernel; portions of rows of exactly 128 numbers in pages of 128 take prefill_attn_bias.cu,
// whose two softmax warpgroups suit them better.
//
// All heads read the same keys, so the M dimension of a tile is 128 consecutive rows of the [token, head] matrix of
// queries: at 32 heads a tile is four neighbouring tokens and its rows see almost the same keys (a decoded token's
// heads are one tile, cut into key splits).  Keys come in tiles of 64 positions and in chunks of 64 columns: a chunk is
// one [64 x 64] swizzled TMA box, the same bytes serve as K (S += Q_c K_c^T) and - the columns below Dv - as V.
// TMEM holds two S buffers (64 columns each, P overlays S) and 256 columns of O; wider values are cut into slices of 256
// columns, a CTA each, that repeat the scores.  Roles: warps 0-3 softmax (a thread per row), warp 4 TMA producer, warp 5
// UMMA issuer.  The chunks outside the CTA's value slice come first in a tile's order: they are free as soon as the
// scores are made, so the next tile's scores start on them while this tile's softmax runs; the slice's own chunks are
// held until P V is done.
// Masks: causal, chunk, sliding window, kept first tokens; a learned sink per head.  Softmax and scores are fp32.
//
// Every wait has a limit.  A wait that runs out sets the CTA's abort flag; all roles then leave their loops, copies and
// products in flight are waited for (with a limit), TMEM is given back, the CTA's outputs become NaN and a counter that
// the host can read (cvllm_latent_attn_aborts) goes up.
#include "common.cuh"
#include "tma.cuh"

namespace cvllm {

__device__ int g_latent_attn_aborts;

namespace la {
constexpr int kBM = 128, kBN = 64, kCols = 64;
constexpr int kQBox = kBM * kCols * 2;     // 16 KB: one column chunk of the query tile
constexpr int kBox = kBN * kCols * 2;      // 8 KB: one column chunk of a key tile
constexpr int kSlice = 256;                // value columns of a CTA
constexpr int kThreads = 192;
constexpr int kMaxSlots = 16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kSpinLimit = 1u << 22;
}  // namespace la

struct LatentAttnParams {
  __nv_bfloat16* out;
  float* part;                  // splits > 1: (max, sum, values) records [B, H, splits]
  const int32_t* seq_start;     // [B] position of the first query (decode: the positions themselves)
  const int32_t* cu_q;          // [B + 1], or NULL: one query per sequence
  const int32_t* batch_mapping;
  const int32_t* table;
  int64_t table_stride_slot, o_stride;
  const float* sink_logits;
  int H, Dv, n_chunks, n_slices, slots, PS, splits, reserved_slot;
  int chunk, window, keep, sink;
  float scale_log2, rescale_threshold;
};

struct LatentAttnBars {
  uint64_t q_full, full[la::kMaxSlots], empty[la::kMaxSlots];
  uint64_t s_full[2], p_full[2], o_done, o_final, drain;   // p_full per S buffer: softmax may be a tile ahead of P V
  uint32_t tmem_base;
  volatile uint32_t abort;
};

// false: the limit was reached here, or another wait of the CTA has reached it
__device__ __forceinline__ bool la_wait(uint64_t* bar, uint32_t parity, LatentAttnBars& b) {
  uint32_t spins = 0;
  while (!mbar_try_wait(bar, parity)) {
    if (b.abort) return false;
    if (++spins > la::kSpinLimit) {
      b.abort = 1;
      return false;
    }
  }
  return true;
}
// the same for a whole warp: one verdict for its lanes
__device__ __forceinline__ bool la_wait_warp(uint64_t* bar, uint32_t parity, LatentAttnBars& b) {
  return __all_sync(0xffffffffu, la_wait(bar, parity, b));
}

__global__ void __launch_bounds__(la::kThreads, 1)
latent_attn_umma_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                        const LatentAttnParams p) {
  using namespace la;
  extern __shared__ unsigned char smem_raw[];
  __shared__ LatentAttnBars bars;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int slice = blockIdx.x % p.n_slices, tile = blockIdx.x / p.n_slices, split = blockIdx.y, b = blockIdx.z;
  const int q_beg = p.cu_q ? p.cu_q[b] : b;
  const int n_new = p.cu_q ? p.cu_q[b + 1] - q_beg : 1;
  const int row0 = tile * kBM;
  if (row0 >= n_new * p.H) return;
  const int rows = min(kBM, n_new * p.H - row0);
  const int slot = p.batch_mapping[b];
  const int start = p.seq_start[b];
  const int p0 = start + row0 / p.H, p_last = start + (row0 + rows - 1) / p.H;
  auto first_key = [&](int pi) {      // first position a query at pi sees through chunk and window
    int lo = p.chunk > 0 ? (pi / p.chunk) * p.chunk : 0;
    if (p.window > 0) lo = max(lo, pi - p.window + 1);
    return lo;
  };
  // key tiles: those that hold kept first tokens and lie before j_begin, then j_begin .. p_last / 64; this CTA's split
  const int lo0 = first_key(p0), lo_max = first_key(p_last);
  const int j_begin = lo0 / kBN;
  const int n_kept = min((min(p.keep, lo0) + kBN - 1) / kBN, j_begin);
  const int n_all = n_kept + p_last / kBN - j_begin + 1;
  const int per = (n_all + p.splits - 1) / p.splits;
  const int t_begin = split * per, n_tiles = min(n_all, t_begin + per) - t_begin;
  const bool last_split = t_begin + n_tiles == n_all;
  auto tile_base = [&](int j) {       // first position of the split's tile j
    const int t = t_begin + j;
    return (t < n_kept ? t : t + j_begin - n_kept) * kBN;
  };
  const int nC = p.n_chunks;
  const int cs = slice * (kSlice / kCols), ce = min(cs + kSlice / kCols, (p.Dv + kCols - 1) / kCols);
  const int nS = ce - cs, nN = nC - nS;                  // chunks of the value slice, chunks outside it
  const int v_cols = min(kSlice, p.Dv - slice * kSlice);  // value columns this CTA writes
  const int r_own = threadIdx.x;                          // softmax threads: their row of the tile
  const int own = row0 + min(r_own, rows - 1), own_h = own % p.H;
  const int64_t own_tok = q_beg + own / p.H;
  float* rec = p.splits > 1 ? p.part + (((int64_t)b * p.H + own_h) * p.splits + split) * (2 + p.Dv) : nullptr;
  if (slot == p.reserved_slot || n_tiles <= 0) {          // a padding row of a graph, or a split without keys
    if (warp < 4 && r_own < rows) {
      if (p.splits > 1) {
        if (slice == 0) {
          rec[0] = -INFINITY;
          rec[1] = 0.f;
        }
      } else {
        for (int c = 0; c < v_cols; ++c)
          p.out[own_tok * p.o_stride + (int64_t)own_h * p.Dv + slice * kSlice + c] = __float2bfloat16_rn(0.f);
      }
    }
    return;
  }
  unsigned char* q_sm = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) &
                                                         ~static_cast<uintptr_t>(1023));
  unsigned char* ring = q_sm + nC * kQBox;
  const int S = p.slots;
  // with room for two whole tiles the next tile's scores are made ahead of this tile's values altogether
  const int ahead = S >= 2 * nC ? nC : nN;

  if (threadIdx.x == 0) {
    mbar_init(&bars.q_full, 1);
    for (int s = 0; s < S; ++s) {
      mbar_init(&bars.full[s], 1);
      mbar_init(&bars.empty[s], 1);
    }
    mbar_init(&bars.s_full[0], 1);
    mbar_init(&bars.s_full[1], 1);
    mbar_init(&bars.p_full[0], kBM);
    mbar_init(&bars.p_full[1], kBM);
    mbar_init(&bars.o_done, 1);
    mbar_init(&bars.o_final, 1);
    mbar_init(&bars.drain, 1);
    bars.abort = 0;
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(&bars.tmem_base, 512);
    tmem_relinquish();
  }
  if (warp == 4 && lane == 0) {
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_k);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars.tmem_base;
  const int total = n_tiles * nC;                         // ring entries of this CTA
  auto chunk_of = [&](int i) { return i < nN ? (i < cs ? i : i + nS) : cs + (i - nN); };   // i-th chunk of a tile's order

  if (warp == 4) {
    // =========================== TMA producer ===========================
    if (lane == 0) {
      mbar_expect_tx(&bars.q_full, nC * kQBox);
      for (int c = 0; c < nC; ++c) tma_load_2d(q_sm + c * kQBox, &tm_q, &bars.q_full, c * kCols, q_beg * p.H + row0);
      const int32_t* pt = p.table + (int64_t)slot * p.table_stride_slot;
      int n = 0, s = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int t0 = tile_base(j), pg = t0 / p.PS;
        const int row = pt[pg] * p.PS + (t0 - pg * p.PS);
        for (int i = 0; i < nC; ++i, ++n) {
          if (!la_wait(&bars.empty[s], ph ^ 1, bars)) {
            ok = false;
            break;
          }
          mbar_expect_tx(&bars.full[s], kBox);
          tma_load_2d(ring + s * kBox, &tm_k, &bars.full[s], chunk_of(i) * kCols, row);
          if (++s == S) {
            s = 0;
            ph ^= 1;
          }
        }
      }
      if (!ok) {      // the copies in flight land before the CTA ends
        for (int m = max(0, n - S); m < n; ++m)
          for (uint32_t spins = 0; !mbar_try_wait(&bars.full[m % S], (m / S) & 1) && spins < kSpinLimit; ++spins) {}
        for (uint32_t spins = 0; !mbar_try_wait(&bars.q_full, 0) && spins < kSpinLimit; ++spins) {}
      }
    }
  } else if (warp == 5) {
    // ============================ UMMA issuer ============================
    constexpr uint32_t idesc_qk = umma_idesc(true, kBM, kBN, false, false);
    constexpr uint32_t idesc_pv = umma_idesc(true, kBM, kCols, false, true);
    const uint32_t tmem_u = __shfl_sync(0xffffffffu, tmem, 0);
    const uint64_t q_desc = umma_smem_desc(smem_u32(q_sm), 16, 1024);
    const uint64_t k_desc = umma_smem_desc(smem_u32(ring), 16, 1024);
    const uint64_t v_desc = umma_smem_desc(smem_u32(ring), kBox, 1024);
    bool ok = la_wait_warp(&bars.q_full, 0, bars);

    // scores of tile j: chunks i0 .. i1 - 1 of its order
    auto issue_qk = [&](int j, int i0, int i1) {
      const uint32_t s_tmem = tmem_u + (j & 1) * kBN;
      for (int i = i0; i < i1 && ok; ++i) {
        const int n = j * nC + i, s = n % S, c = chunk_of(i);
        ok = la_wait_warp(&bars.full[s], (n / S) & 1, bars);
        if (!ok) return;
        if (i >= nN && last_split && j == n_tiles - 1) {
          // rows after the tile's last query may be uninitialised memory; their weight is exactly 0, but 0 * NaN would
          // poison O
          const int valid = p_last + 1 - tile_base(j);
          if (valid < kBN) {
            uint4* v4 = reinterpret_cast<uint4*>(ring + s * kBox);
            for (int k = valid * 8 + lane; k < kBN * 8; k += 32) v4[k] = make_uint4(0, 0, 0, 0);
            fence_proxy_async_smem();
            __syncwarp();
          }
        }
        tc_fence_after();
        const uint64_t qd = umma_desc_add(q_desc, c * kQBox), kd = umma_desc_add(k_desc, s * kBox);
#pragma unroll
        for (int kk = 0; kk < kCols / 16; ++kk)
          umma_ss_warp(s_tmem, umma_desc_add(qd, kk * 32), umma_desc_add(kd, kk * 32), idesc_qk,
                       (i > 0 || kk > 0) ? 1u : 0u);
        if (i < nN) umma_commit_warp(&bars.empty[s]);
      }
      if (ok && i1 == nC && i1 > i0) umma_commit_warp(&bars.s_full[j & 1]);
    };
    auto issue_pv = [&](int j) {
      ok = la_wait_warp(&bars.p_full[j & 1], (j >> 1) & 1, bars);
      if (!ok) return;
      tc_fence_after();
      const uint32_t p_tmem = tmem_u + (j & 1) * kBN;
      for (int i = nN; i < nC; ++i) {
        const int s = (j * nC + i) % S;
        const uint32_t o_tmem = tmem_u + 256 + (i - nN) * kCols;
        const uint64_t vd = umma_desc_add(v_desc, s * kBox);
#pragma unroll
        for (int kk = 0; kk < kBN / 16; ++kk)
          umma_ts_warp(o_tmem, p_tmem + kk * 8, umma_desc_add(vd, kk * 2048), idesc_pv, (j > 0 || kk > 0) ? 1u : 0u);
        umma_commit_warp(&bars.empty[s]);
      }
      umma_commit_warp(&bars.o_done);
      if (j == n_tiles - 1) umma_commit_warp(&bars.o_final);
    };
    if (ok) issue_qk(0, 0, nC);
    for (int j = 0; j < n_tiles && ok; ++j) {
      const bool more = j + 1 < n_tiles;
      if (more) issue_qk(j + 1, 0, ahead);
      if (ok) issue_pv(j);
      if (ok && more) issue_qk(j + 1, ahead, nC);
    }
    if (!ok) {      // products in flight end before TMEM is given back
      umma_commit_warp(&bars.drain);
      for (uint32_t spins = 0; !mbar_try_wait(&bars.drain, 0) && spins < kSpinLimit; ++spins) {}
    }
    __syncwarp();
  } else {
    // ====================== softmax / correction / epilogue ======================
    const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
    const bool row_valid = r_own < rows;
    const int pi = start + own / p.H, lo_i = first_key(pi);
    const bool with_sink = p.sink && p.splits == 1;     // with splits the merge adds it
    float m_ref = with_sink ? (p.sink_logits ? p.sink_logits[own_h] * kLog2e : 0.f) : -INFINITY;
    float l = with_sink ? 1.f : 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      ok = la_wait_warp(&bars.s_full[j & 1], (j >> 1) & 1, bars);
      if (!ok) break;
      tc_fence_after();
      const uint32_t s_tmem = tmem + (j & 1) * kBN + lane_base;
      float s[kBN];
#pragma unroll
      for (int c = 0; c < kBN / 32; ++c) {
        uint32_t tmp[32];
        tmem_ld32(s_tmem + c * 32, tmp);
#pragma unroll
        for (int i = 0; i < 32; ++i) s[c * 32 + i] = __uint_as_float(tmp[i]) ;
      }
      tc_wait_ld();
#pragma unroll
      for (int c = 0; c < kBN; ++c) s[c] *= p.scale_log2;
      const int base = tile_base(j);
      if (base + kBN - 1 > p0 || base < lo_max) {       // a tile at an edge of some row's keys
        const int c_hi = pi - base, c_lo = lo_i - base, c_keep = p.keep - base;
#pragma unroll
        for (int c = 0; c < kBN; ++c)
          if (c > c_hi || (c < c_lo && c >= c_keep)) s[c] = -INFINITY;
      }
      float mx0 = s[0], mx1 = s[1], mx2 = s[2], mx3 = s[3];
#pragma unroll
      for (int c = 4; c < kBN; c += 4) {
        mx0 = fmaxf(mx0, s[c]);
        mx1 = fmaxf(mx1, s[c + 1]);
        mx2 = fmaxf(mx2, s[c + 2]);
        mx3 = fmaxf(mx3, s[c + 3]);
      }
      // a row that sees no key of this tile keeps a finite reference
      const float m_new = fmaxf(m_ref, fmaxf(fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)), -1e30f));
      const bool need = j == 0 || m_new > m_ref + p.rescale_threshold;
      if (__any_sync(0xffffffffu, need)) {              // O *= alpha, l *= alpha, m_ref <- m_new
        const float alpha = ex2(m_ref - m_new);         // m_ref == -inf on the first tile -> 0
        m_ref = m_new;
        l *= alpha;
        if (j > 0) {
          // S(j) is complete, so P V of tile j - 2 is: this phase cannot be taken for an older one
          ok = la_wait_warp(&bars.o_done, (j - 1) & 1, bars);
          if (!ok) break;
          tc_fence_after();
          for (int c = 0; c < nS * kCols; c += 32) {
            uint32_t o[32];
            tmem_ld32(tmem + 256 + lane_base + c, o);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st32(tmem + 256 + lane_base + c, o);
          }
        }
      }
      uint32_t pk[32];
      float l0 = 0.f, l1 = 0.f;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const float e0 = ex2(s[2 * i] - m_ref), e1 = ex2(s[2 * i + 1] - m_ref);
        l0 += e0;
        l1 += e1;
        pk[i] = pack2<true>(e0, e1);
      }
      l += l0 + l1;
      tmem_st32(s_tmem, pk);
      tc_wait_st();
      tc_fence_before();
      mbar_arrive(&bars.p_full[j & 1]);
    }
    if (ok) ok = la_wait_warp(&bars.o_final, 0, bars);
    tc_fence_after();
    const float inv = ok ? (p.splits > 1 ? 1.f : (l > 0.f ? 1.f / l : 0.f)) : NAN;
    if (rec && row_valid && slice == 0) {
      rec[0] = ok ? m_ref : NAN;
      rec[1] = l;
    }
    __nv_bfloat16* orow = p.out + own_tok * p.o_stride + (int64_t)own_h * p.Dv + slice * kSlice;
    for (int c = 0; c < v_cols; c += 32) {
      uint32_t o[32];
      tmem_ld32(tmem + 256 + lane_base + c, o);
      tc_wait_ld();
      if (!row_valid) continue;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        if (c + 8 * i >= v_cols) break;
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = __uint_as_float(o[8 * i + e]) * inv;
        if (rec) {
          float2* dst = reinterpret_cast<float2*>(rec + 2 + slice * kSlice + c + 8 * i);
#pragma unroll
          for (int e = 0; e < 4; ++e) dst[e] = make_float2(v[2 * e], v[2 * e + 1]);
        } else {
          *reinterpret_cast<uint4*>(orow + c + 8 * i) =
              make_uint4(pack2<true>(v[0], v[1]), pack2<true>(v[2], v[3]), pack2<true>(v[4], v[5]), pack2<true>(v[6], v[7]));
        }
      }
    }
    if (!ok && threadIdx.x == 0) atomicAdd(&g_latent_attn_aborts, 1);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 5) tmem_dealloc(tmem, 512);
}

}  // namespace cvllm

using namespace cvllm;

// Whether the kernel serves a geometry (values = the first Dv columns of the keys of ONE key/value head, bfloat16).
bool cvllm_latent_attn_umma_serves(int D, int Dv, int page_size, int64_t out_stride, const void* q, const void* cache,
                                   const void* out) {
  return D % 8 == 0 && Dv % 8 == 0 && Dv <= D && D <= 9 * la::kCols && Dv <= 512 && page_size % la::kBN == 0 &&
         out_stride % 8 == 0 && aligned16(q) && aligned16(cache) && aligned16(out);
}

// Launch.  Called by the portion (cu_q given, seq_start = first positions) and decode (cu_q NULL, seq_start = positions)
// entry points of bias_attn.cu; `tokens` = rows of q / H.
int cvllm_launch_latent_attn_umma(const void* q, const void* cache, int64_t cache_rows, void* out, int64_t o_stride,
                                  const int32_t* seq_start, const int32_t* cu_q, const int32_t* batch_mapping,
                                  const int32_t* table, int64_t table_stride_slot, int B, int tokens, int max_new, int H,
                                  int D, int Dv, int PS, float scale, int chunk, int window, int keep, int sink,
                                  const float* sink_logits, int splits, float* part, int reserved_slot, cudaStream_t st) {
  using namespace la;
  CUtensorMap tm_q, tm_k;
  {
    const uint32_t boxq[2] = {kCols, kBM}, boxk[2] = {kCols, kBN};
    const uint64_t dq[2] = {(uint64_t)D, (uint64_t)tokens * H}, dk[2] = {(uint64_t)D, (uint64_t)cache_rows};
    const uint64_t stride[1] = {(uint64_t)D * 2};
    int rc = make_tmap_16b(&tm_q, q, 2, dq, stride, boxq, true);
    if (rc) return rc;
    rc = make_tmap_16b(&tm_k, cache, 2, dk, stride, boxk, true);
    if (rc) return rc;
  }
  LatentAttnParams p;
  p.out = static_cast<__nv_bfloat16*>(out);
  p.part = part;
  p.seq_start = seq_start; p.cu_q = cu_q; p.batch_mapping = batch_mapping; p.table = table;
  p.table_stride_slot = table_stride_slot; p.o_stride = o_stride;
  p.sink_logits = sink ? sink_logits : nullptr;
  p.H = H; p.Dv = Dv; p.PS = PS; p.splits = splits; p.reserved_slot = reserved_slot;
  p.n_chunks = cdiv(D, kCols);
  p.n_slices = cdiv(Dv, kSlice);
  const int dyn_max = 231424;                // 227 KB less the static barriers
  p.slots = (dyn_max - 1024 - p.n_chunks * kQBox) / kBox;
  if (p.slots > kMaxSlots) p.slots = kMaxSlots;
  CVLLM_CHECK_SUPPORTED(p.slots >= p.n_chunks);
  p.chunk = chunk; p.window = window; p.keep = keep; p.sink = sink;
  p.scale_log2 = scale * kLog2e;
  p.rescale_threshold = 8.0f;
  {
    const float t = test_options().prefill_threshold.load(std::memory_order_relaxed);
    if (t >= 0.f) p.rescale_threshold = t;
  }
  const int64_t tiles = ((int64_t)max_new * H + kBM - 1) / kBM;
  CVLLM_CHECK_SUPPORTED(tiles * p.n_slices <= 2147483647 && splits <= 65535 && B <= 65535);
  const dim3 grid((unsigned)(tiles * p.n_slices), splits, B);
  static std::atomic<uint64_t> attr{0};
  CVLLM_CHECK_CUDA(ensure_max_dyn_smem((const void*)latent_attn_umma_kernel, dyn_max, attr));
  latent_attn_umma_kernel<<<grid, kThreads, 1024 + p.n_chunks * kQBox + p.slots * kBox, st>>>(tm_q, tm_k, p);
  CVLLM_CHECK_LAUNCH();
  return CVLLM_OK;
}

extern "C" int cvllm_latent_attn_aborts(int* count) {
  CVLLM_CHECK_ARG(count != nullptr);
  CVLLM_CHECK_CUDA(cudaMemcpyFromSymbol(count, g_latent_attn_aborts, sizeof(int)));
  return CVLLM_OK;
}
