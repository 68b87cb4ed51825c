// Split-KV paged GQA decode attention, TMA-fed.
//
// One CTA handles one (sequence, kv head, KV split): a producer warp streams 64-token K and V tiles from the paged
// cache into a 3-stage shared-memory ring with cp.async.bulk.tensor (one box per KV block, or per 64 tokens when the
// block is larger; 128-byte swizzle), completion on mbarriers; four consumer warps each take 16 tokens of every tile,
// compute S = Q K^T and O += P V on the tensor cores from ldmatrix fragments with an online softmax in registers,
// and release the stage.  The `group * q_len` (<= 16) query rows that share the kv head form the M dimension.
// The four partial results are merged through shared memory; with several KV splits the normalised partials and
// their log-sum-exp go to a workspace that a small merge kernel (attention.cu) reduces.
//
// Compared with issuing 16-byte cp.async copies from every lane (the fallback kernel in attention.cu), the copy
// engine removes the per-chunk address arithmetic and block-table lookups from the compute warps, which is what
// bounds a decode kernel whose arithmetic intensity is a few FLOP per byte.
//
// Template parameters: DK / DV = query-key / value head dimension padded to 64, 128 or 256 (the TMA loads fill the padding with
// zeros), EXT = score extensions (per-head distance bias, per-head sink, chunk mask, first keys that stay visible behind a
// window, scores bounded by a tanh), head dimensions below the padded ones, and more than 16 query rows per kv head (a CTA per
// block of 16).  Differential attention (maps = 2): a kv head's row holds the keys of both maps side by side and a query row is
// zero in the other map's columns, so that one product serves both; the merge stores rms(first - factor * second) * mult.
//
// Role: the reference's FlashInfer `batch_decode_with_kv_cache` (xllm/core/kernels/cuda/batch_decode.cpp:26-85).
#include "softcap.cuh"

namespace xl_dec {
using namespace xl;

__device__ __forceinline__ void cp_async_16(void* smem_dst, const void* gsrc, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem_dst)), "l"(gsrc), "r"(sz) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

struct DecParams {
  const __nv_bfloat16* q;
  __nv_bfloat16* out;
  const int* q_cu;
  const int* kv_lens;
  const int* block_tables;
  int seq_begin, seq_end;
  int max_blocks, block_size, n_q, n_kv, q_stride;
  float scale_log2;
  int window;
  int num_splits;
  float* part_o;
  float* part_lse;
  int num_blocks_total;
  int box_tokens;     // tokens per TMA box: min(block_size, 64)
  int* status;
  const int* dyn_end = nullptr;   // optional device scalar that replaces seq_end (launch sized for a capacity)
  int ws_rows = 0;                // > 0: row capacity of a fixed-size workspace; sequences that do not fit it (or have more
                                  // than 16 query rows x heads per kv head) are skipped and XL_ERR_BOUNDS is recorded
  // score extensions (EXT): see xl_prefill_attention_ext
  int dk = 0, dv = 0;
  int chunk = 0;
  int keep_first = 0;
  const float* slopes = nullptr;
  const float* sinks = nullptr;
  int row_blocks = 1;             // blocks of 16 query rows per kv head (grid.y = n_kv * row_blocks)
  int shared_keys = 0;            // one key head for all value heads
  int maps = 1;
  float cap_in = 0.f, cap_out = 0.f;      // cap_out > 0: scores are cap_out * tanh(product * cap_in), in the log2 domain
  int cap_level = CAP_CHECK;
  const float* mix = nullptr;
  float mix_mult = 0.f, mix_eps = 0.f;
};

constexpr int kStages = 3;
constexpr int kTile = 64;

struct DecBarriers {
  uint64_t full[kStages];
  uint64_t empty[kStages];
};

template <int DK, int DV, bool EXT, bool CAP = false>
__global__ void __launch_bounds__(160) decode_attn_tma_kernel(const __grid_constant__ CUtensorMap tmK,
                                                              const __grid_constant__ CUtensorMap tmV, DecParams p) {
  constexpr int KH = DK / 64, VH = DV / 64;       // 128-byte column slabs per row
  constexpr int SLAB = kTile * 128;               // bytes of one slab of a 64-token tile
  constexpr int K_BYTES = KH * SLAB;              // K bytes per stage (V behind it)
  constexpr int STAGE_BYTES = (KH + VH) * SLAB;
  constexpr int CH = DK / 8;
  constexpr float kL2e = 1.4426950408889634f;
  const int dk = EXT ? p.dk : DK, dv = EXT ? p.dv : DV;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* ring = smem;                                          // kStages * STAGE_BYTES, 1024-aligned
  constexpr int MERGE_BYTES = 4 * 16 * DV * 4 + 128 * 4;         // partials of the four warps, in the ring's memory
  constexpr int RING_BYTES = kStages * STAGE_BYTES > MERGE_BYTES ? kStages * STAGE_BYTES : MERGE_BYTES;
  uint8_t* sQ = smem + RING_BYTES;                               // 16 x DK bf16, 16-byte-chunk XOR swizzle
  DecBarriers* bars = reinterpret_cast<DecBarriers*>(sQ + 16 * DK * 2);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = p.seq_begin + blockIdx.x;
  int kvh = blockIdx.y, row0 = 0;                 // row0: first query row (token x head) of this CTA
  if (EXT && p.row_blocks > 1) {
    kvh = blockIdx.y / p.row_blocks;
    row0 = blockIdx.y % p.row_blocks * 16;
  }
  const int split = blockIdx.z;
  const int group = p.n_q / p.n_kv;
  if (seq >= (p.dyn_end ? *p.dyn_end : p.seq_end)) return;
  const int q_start = p.q_cu[seq];
  const int q_len = p.q_cu[seq + 1] - q_start;
  const int kv_len = p.kv_lens[seq];
  if (q_len <= 0) return;
  if (p.ws_rows > 0 && (q_len * group > 16 || (p.num_splits > 1 && q_start + q_len > p.ws_rows))) {
    if (threadIdx.x == 0) atomicExch(p.status, XL_ERR_BOUNDS);
    return;
  }
  const int rows = min(16, q_len * group - row0);
  if (rows <= 0) return;
  const int* bt = p.block_tables + size_t(seq) * p.max_blocks;

  int r_begin = 0;                                // first key that any row may see, rounded down to a tile
  if (EXT && p.chunk > 0) r_begin = (kv_len - q_len) / p.chunk * p.chunk / kTile * kTile;
  if (p.window > 0) r_begin = max(r_begin, max(0, kv_len - q_len - p.window + 1) / kTile * kTile);
  const int n_keep = EXT ? (min(p.keep_first, r_begin) + kTile - 1) / kTile : 0;      // tiles of kept first keys ahead of it
  const int all_tiles = n_keep + (kv_len - r_begin + kTile - 1) / kTile;
  const int per_split = (all_tiles + p.num_splits - 1) / p.num_splits;
  const int t_first = split * per_split;
  const int n_tiles = max(0, min(all_tiles, t_first + per_split) - t_first);
  // first key of this split's t-th tile
  auto tile_kv = [&](int t) { return t_first + t < n_keep ? (t_first + t) * kTile : r_begin + (t_first + t - n_keep) * kTile; };

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 4);
    }
    mbar_fence_init();
  }
  // Q rows -> smem (zero beyond `rows` and in the columns of another map); row m = qtok * group + g
  const int dq = EXT ? dk / p.maps : dk;          // columns of a query head
  for (int i = threadIdx.x; i < 16 * CH; i += blockDim.x) {
    const int r = i / CH, c = i % CH;
    const int col = EXT ? c * 8 - (p.maps == 2 ? ((row0 + r) & 1) * dq : 0) : c * 8;      // column of this chunk in the query head
    const bool ok = r < rows && (!EXT || (col >= 0 && col < dq));
    const int qt = ok ? (row0 + r) / group : 0, g = ok ? (row0 + r) % group : 0;
    const __nv_bfloat16* src = p.q + size_t(q_start + qt) * p.q_stride + (kvh * group + g) * dq + (ok ? col : 0);
    cp_async_16(sQ + uint32_t(r) * (DK * 2) + (uint32_t(c ^ (r & 7)) << 4), src, ok);
  }
  cp_async_commit();
  cp_async_wait_all();
  __syncthreads();

  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const int row_a = lane >> 2, row_b = row_a + 8;

  if (warp == 4) {
    // ------------------------------------------------------------ producer
    if (elect_one_sync()) {
      prefetch_tmap(&tmK);
      prefetch_tmap(&tmV);
      const int bt_tok = p.box_tokens;
      int t = 0;
      bool ok = true;
      for (; t < n_tiles; ++t) {
        const int s = t % kStages;
        const uint32_t ph = (t / kStages) & 1;
        if (!mbar_wait(&bars->empty[s], ph ^ 1)) {
          atomicExch(p.status, XL_ERR_WAIT_EMPTY);
          ok = false;
          break;
        }
        const int base = tile_kv(t);
        const int n_tok = min(kTile, kv_len - base);
        const int n_boxes = (n_tok + bt_tok - 1) / bt_tok;
        mbar_arrive_expect_tx(&bars->full[s], uint32_t(n_boxes) * bt_tok * 128 * (KH + VH));
        uint8_t* dK = ring + s * STAGE_BYTES;
        uint8_t* dV = dK + K_BYTES;
        for (int b = 0; b < n_boxes; ++b) {
          const int tok = base + b * bt_tok;
          int blk = bt[tok / p.block_size];
          if (blk < 0 || blk >= p.num_blocks_total) blk = 0;     // never form an address outside the cache
          const int z = blk * p.block_size + tok % p.block_size;
#pragma unroll
          for (int h = 0; h < (KH > VH ? KH : VH); ++h) {
            if (h < KH) tma_load_3d(dK + h * SLAB + b * bt_tok * 128, &tmK, &bars->full[s], h * 64, EXT && p.shared_keys ? 0 : kvh, z);
            if (h < VH) tma_load_3d(dV + h * SLAB + b * bt_tok * 128, &tmV, &bars->full[s], h * 64, kvh, z);
          }
        }
      }
      if (!ok) {   // let the copies already issued land (bounded) before the CTA retires
        const int first = t >= kStages ? t - kStages : 0;
        for (int j = first; j < t; ++j) mbar_wait(&bars->full[j % kStages], (j / kStages) & 1);
      }
    }
  } else {
    // ------------------------------------------------------------ consumers
    constexpr bool kKeepQ = DK <= 128;                     // wider query rows are read from shared memory at every tile
    uint32_t qf[kKeepQ ? DK / 16 : 1][4];
    auto load_q = [&](int ks, uint32_t (&f)[4]) {
      const int r = (lane & 7) + ((lane >> 3) & 1) * 8;
      const int c = ks * 2 + (lane >> 4);
      ldsm_x4(smem_u32(sQ + uint32_t(r) * (DK * 2) + (uint32_t(c ^ (r & 7)) << 4)), f[0], f[1], f[2], f[3]);
    };
    if (kKeepQ) {
#pragma unroll
      for (int ks = 0; ks < (kKeepQ ? DK / 16 : 1); ++ks) load_q(ks, qf[ks]);
    }
    const int lim_a = kv_len - q_len + (row_a < rows ? (row0 + row_a) / group : 0);
    const int lim_b = kv_len - q_len + (row_b < rows ? (row0 + row_b) / group : 0);
    int lo_a = 0, lo_b = 0;                                // first visible key of the row's chunk
    float slope_a = 0.f, slope_b = 0.f;
    if (EXT) {
      if (p.chunk > 0) {
        lo_a = lim_a / p.chunk * p.chunk;
        lo_b = lim_b / p.chunk * p.chunk;
      }
      if (p.slopes) {
        slope_a = p.slopes[kvh * group + (row_a < rows ? (row0 + row_a) % group : 0)] * kL2e;
        slope_b = p.slopes[kvh * group + (row_b < rows ? (row0 + row_b) % group : 0)] * kL2e;
      }
    }
    const int rk = (lane & 7) + (lane >> 4) * 8;           // K fragment row (token) of this lane
    const int rv = (lane & 7) + ((lane >> 3) & 1) * 8;     // V fragment row (token) of this lane
    for (int t = 0; t < n_tiles; ++t) {
      const int s = t % kStages;
      const uint32_t ph = (t / kStages) & 1;
      if (!mbar_wait(&bars->full[s], ph)) {
        if (lane == 0) atomicExch(p.status, XL_ERR_WAIT_FULL);
        break;
      }
      const int base = tile_kv(t) + warp * 16;
      if (base < kv_len) {
        const uint8_t* tK = ring + s * STAGE_BYTES + warp * 2048;
        const uint8_t* tV = tK + K_BYTES;
        float sc[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
          uint32_t b0, b1, b2, b3;
          const int c = (ks & 3) * 2 + ((lane >> 3) & 1);
          ldsm_x4(smem_u32(tK + (ks >> 2) * SLAB + rk * 128 + ((c ^ (rk & 7)) << 4)), b0, b1, b2, b3);
          if (!kKeepQ) load_q(ks, qf[0]);
          mma_bf16_16816(sc[0], qf[kKeepQ ? ks : 0], b0, b1);
          mma_bf16_16816(sc[1], qf[kKeepQ ? ks : 0], b2, b3);
        }
        if (CAP) {
          softcap_row(sc[0], p.cap_in, p.cap_level);
          softcap_row(sc[1], p.cap_in, p.cap_level);
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int tok = base + i * 8 + (lane & 3) * 2 + (e & 1);
            const int lim = (e < 2) ? lim_a : lim_b;
            bool ok = tok <= lim && tok < kv_len;
            if (p.window > 0) ok = ok && (tok > lim - p.window || (EXT && tok < p.keep_first));
            float x = sc[i][e] * (CAP ? p.cap_in * p.cap_out : p.scale_log2);
            if (EXT) {
              ok = ok && tok >= ((e < 2) ? lo_a : lo_b);
              x += ((e < 2) ? slope_a : slope_b) * float(tok - lim);
            }
            const float v = ok ? x : -INFINITY;
            sc[i][e] = v;
            mx[e >> 1] = fmaxf(mx[e >> 1], v);
          }
        }
        float alpha[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
          mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
          const float m_new = fmaxf(m_run[h], mx[h]);
          alpha[h] = (m_new == -INFINITY) ? 1.f : exp2f(m_run[h] - m_new);
          m_run[h] = m_new;
        }
        float rs[2] = {0.f, 0.f};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float m = m_run[e >> 1];
            const float pv = (m == -INFINITY) ? 0.f : exp2f(sc[i][e] - m);
            sc[i][e] = pv;
            rs[e >> 1] += pv;
          }
        }
        l_run[0] = l_run[0] * alpha[0] + rs[0];
        l_run[1] = l_run[1] * alpha[1] + rs[1];
        const uint32_t pa[4] = {pack_bf16x2(sc[0][0], sc[0][1]), pack_bf16x2(sc[0][2], sc[0][3]),
                                pack_bf16x2(sc[1][0], sc[1][1]), pack_bf16x2(sc[1][2], sc[1][3])};
        const bool rescale = (alpha[0] != 1.f) || (alpha[1] != 1.f);
#pragma unroll
        for (int dt = 0; dt < DV / 16; ++dt) {
          if (rescale) {
            o[2 * dt][0] *= alpha[0]; o[2 * dt][1] *= alpha[0]; o[2 * dt][2] *= alpha[1]; o[2 * dt][3] *= alpha[1];
            o[2 * dt + 1][0] *= alpha[0]; o[2 * dt + 1][1] *= alpha[0]; o[2 * dt + 1][2] *= alpha[1]; o[2 * dt + 1][3] *= alpha[1];
          }
          uint32_t b0, b1, b2, b3;
          const int c = (dt & 3) * 2 + (lane >> 4);
          ldsm_x4_t(smem_u32(tV + (dt >> 2) * SLAB + rv * 128 + ((c ^ (rv & 7)) << 4)), b0, b1, b2, b3);
          mma_bf16_16816(o[2 * dt], pa, b0, b1);
          mma_bf16_16816(o[2 * dt + 1], pa, b2, b3);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->empty[s]);
    }
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
      l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
    }
  }
  __syncthreads();   // ring no longer needed: reuse it for the merge

  float* sO = reinterpret_cast<float*>(ring);     // [4][16][DV]
  float* sM = sO + 4 * 16 * DV;                   // [4][16]
  float* sL = sM + 64;
  if (warp < 4) {
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      const int col = i * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(sO + (warp * 16 + row_a) * DV + col) = make_float2(o[i][0], o[i][1]);
      *reinterpret_cast<float2*>(sO + (warp * 16 + row_b) * DV + col) = make_float2(o[i][2], o[i][3]);
    }
    if ((lane & 3) == 0) {
      sM[warp * 16 + row_a] = m_run[0]; sL[warp * 16 + row_a] = l_run[0];
      sM[warp * 16 + row_b] = m_run[1]; sL[warp * 16 + row_b] = l_run[1];
    }
  }
  __syncthreads();
  if (EXT && p.maps == 2 && p.num_splits == 1) {
    // rows 2 i and 2 i + 1 are the two maps of one output head
    const float factor = *p.mix;
    for (int i = warp; i < rows / 2 && warp < 4; i += 4) {
      float w[2][4];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int r = 2 * i + k;
        const int hq = kvh * group + (row0 + r) % group;
        const float m = fmaxf(fmaxf(sM[r], sM[16 + r]), fmaxf(sM[32 + r], sM[48 + r]));
        float den = p.sinks && m != -INFINITY ? exp2f(p.sinks[hq] * kL2e - m) : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          w[k][j] = sM[16 * j + r] == -INFINITY ? 0.f : exp2f(sM[16 * j + r] - m);
          den += w[k][j] * sL[16 * j + r];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) w[k][j] *= den > 0.f ? 1.f / den : 0.f;
      }
      float d[DV / 32], ss = 0.f;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c) {           // columns past dv hold zeros
        float a[2] = {0.f, 0.f};
#pragma unroll
        for (int k = 0; k < 2; ++k)
#pragma unroll
          for (int j = 0; j < 4; ++j) a[k] += w[k][j] * sO[(16 * j + 2 * i + k) * DV + c * 32 + lane];
        d[c] = fmaf(-factor, a[1], a[0]);
        ss += d[c] * d[c];
      }
      const float s = rsqrtf(warp_sum(ss) / float(dv) + p.mix_eps) * p.mix_mult;
      const int qt = (row0 + 2 * i) / group, head = (kvh * group + (row0 + 2 * i) % group) / 2;
      __nv_bfloat16* dst = p.out + size_t(q_start + qt) * (size_t(p.n_q / 2) * dv) + head * dv;
#pragma unroll
      for (int c = 0; c < DV / 32; ++c)
        if (c * 32 + lane < dv) dst[c * 32 + lane] = __float2bfloat16(d[c] * s);
    }
  } else if (warp < 4) {
    for (int r = warp; r < rows; r += 4) {
      const float m = fmaxf(fmaxf(sM[r], sM[16 + r]), fmaxf(sM[32 + r], sM[48 + r]));
      float w0 = (sM[r] == -INFINITY) ? 0.f : exp2f(sM[r] - m);
      float w1 = (sM[16 + r] == -INFINITY) ? 0.f : exp2f(sM[16 + r] - m);
      float w2 = (sM[32 + r] == -INFINITY) ? 0.f : exp2f(sM[32 + r] - m);
      float w3 = (sM[48 + r] == -INFINITY) ? 0.f : exp2f(sM[48 + r] - m);
      const float l = w0 * sL[r] + w1 * sL[16 + r] + w2 * sL[32 + r] + w3 * sL[48 + r];
      const int qt = (row0 + r) / group, g = (row0 + r) % group;
      const int hq = kvh * group + g;
      float den = l;                              // the sink joins once: here, or in the merge of the splits
      if (EXT && p.sinks && p.num_splits == 1 && m != -INFINITY) den += exp2f(p.sinks[hq] * kL2e - m);
      const float inv = den > 0.f ? 1.f / den : 0.f;
      const size_t tok = size_t(q_start + qt);
      for (int c = lane * 2; c < dv; c += 64) {
        const float a = w0 * sO[r * DV + c] + w1 * sO[(16 + r) * DV + c] + w2 * sO[(32 + r) * DV + c] + w3 * sO[(48 + r) * DV + c];
        const float b = w0 * sO[r * DV + c + 1] + w1 * sO[(16 + r) * DV + c + 1] + w2 * sO[(32 + r) * DV + c + 1] +
                        w3 * sO[(48 + r) * DV + c + 1];
        if (p.num_splits == 1) {
          *reinterpret_cast<uint32_t*>(p.out + tok * (size_t(p.n_q) * dv) + hq * dv + c) = pack_bf16x2(a * inv, b * inv);
        } else {
          float* po = p.part_o + ((tok * p.n_q + hq) * p.num_splits + split) * dv;
          *reinterpret_cast<float2*>(po + c) = make_float2(a * inv, b * inv);
        }
      }
      if (p.num_splits > 1 && lane == 0)
        p.part_lse[(tok * p.n_q + hq) * p.num_splits + split] = (l > 0.f) ? m + log2f(l) : -INFINITY;
    }
  }
}

// ---------------------------------------------------------------- one wide key head for all query heads
// One CTA handles one (sequence, block of 16 MT query rows, KV split); a row is (token, query head), so the rows of a block may belong to
// several value heads.  Keys and values pass through a ring of [128 tokens][64 columns] slabs: the slabs of a tile's keys, whose
// products add up to S, then those of the value heads that the block's rows need; P is zero in the rows of other value heads, so all of
// them accumulate into one O.  Eight consumer warps take 16 tokens of every slab each.
constexpr int kWideTile = 128, kWideSlab = kWideTile * 128;
constexpr int kWideMost = 12, kWideProducers = 2, kWideConsumers = 8, kWideThreads = 32 * (kWideConsumers + kWideProducers);
struct WideDecBarriers {
  uint64_t full[kWideMost];
  uint64_t empty[kWideMost];
};
// Place in a ring of n slabs and how often it has gone round.
struct RingPos {
  int slot = 0;
  uint32_t phase = 0;
  __device__ __forceinline__ void next(int n) {
    if (++slot == n) {
      slot = 0;
      phase ^= 1;
    }
  }
};

template <int MT, int DV>
__global__ void __launch_bounds__(kWideThreads, 1) decode_attn_wide_kernel(const __grid_constant__ CUtensorMap tmK,
                                                                           const __grid_constant__ CUtensorMap tmV, const DecParams p, const int KS,
                                                                           const int n_slabs) {
  constexpr int VH = DV / 64, ROWS = 16 * MT, CW = kWideConsumers;
  constexpr float kL2e = 1.4426950408889634f;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = ring + n_slabs * kWideSlab;                      // ROWS x 64 KS bf16, 16-byte-chunk XOR swizzle
  WideDecBarriers* bars = reinterpret_cast<WideDecBarriers*>(sQ + ROWS * KS * 128);
  float* sM = reinterpret_cast<float*>(bars + 1);                // [CW][ROWS] maxima, then sums
  float* sL = sM + CW * ROWS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = p.seq_begin + blockIdx.y, row0 = blockIdx.x * ROWS, split = blockIdx.z;
  const int group = p.n_q / p.n_kv, dk = p.dk, dv = p.dv;
  if (seq >= (p.dyn_end ? *p.dyn_end : p.seq_end)) return;
  const int q_start = p.q_cu[seq];
  const int q_len = p.q_cu[seq + 1] - q_start;
  const int kv_len = p.kv_lens[seq];
  if (q_len <= 0) return;
  const int rows = min(ROWS, q_len * p.n_q - row0);
  if (rows <= 0) return;
  // value heads of the rows: consecutive ones, all of them when the block reaches into the next token
  const int h_first = row0 % p.n_q, h_last = h_first + rows - 1;
  const int v_first = h_last >= p.n_q ? 0 : h_first / group, v_last = h_last >= p.n_q ? p.n_kv - 1 : h_last / group;
  const int* bt = p.block_tables + size_t(seq) * p.max_blocks;
  const int r_begin = p.window > 0 ? max(0, kv_len - q_len - p.window + 1) / kTile * kTile : 0;     // a multiple of the boxes' tokens
  const int all_tiles = (kv_len - r_begin + kWideTile - 1) / kWideTile;
  const int per_split = (all_tiles + p.num_splits - 1) / p.num_splits;
  const int t_first = split * per_split;
  const int n_tiles = max(0, min(all_tiles, t_first + per_split) - t_first);

  if (threadIdx.x == 0) {
    for (int s = 0; s < n_slabs; ++s) {
      mbar_init(&bars->full[s], kWideProducers);
      mbar_init(&bars->empty[s], CW);
    }
    mbar_fence_init();
  }
  for (int i = threadIdx.x; i < ROWS * KS * 8; i += blockDim.x) {
    const int r = i / (KS * 8), c = i % (KS * 8);
    const bool ok = r < rows && c * 8 < dk;
    const int m = ok ? row0 + r : 0;
    const __nv_bfloat16* src = p.q + size_t(q_start + m / p.n_q) * p.q_stride + size_t(m % p.n_q) * dk + (ok ? c * 8 : 0);
    cp_async_16(sQ + uint32_t(r) * (KS * 128) + (uint32_t(c ^ (r & 7)) << 4), src, ok);
  }
  cp_async_commit();
  cp_async_wait_all();
  __syncthreads();

  float o[MT][DV / 8][4];
  float m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    m_run[mt][0] = m_run[mt][1] = -INFINITY;
    l_run[mt][0] = l_run[mt][1] = 0.f;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;
  }

  RingPos at;
  if (warp >= CW) {
    // ------------------------------------------------------------ producers: a warp issues one copy at a time, so they share a slab's
    // boxes; the first one also announces the slab's bytes
    const int part = warp - CW, bt_tok = p.box_tokens;
    if (lane == 0) {
      prefetch_tmap(&tmK);
      prefetch_tmap(&tmV);
    }
    const int per_tile = KS + (v_last - v_first + 1) * VH;
    int issued = 0;
    bool ok = true;
    for (int t = 0; t < n_tiles && ok; ++t) {
      const int base = r_begin + (t_first + t) * kWideTile;
      const int n_boxes = (min(kWideTile, kv_len - base) + bt_tok - 1) / bt_tok;
      int z = 0;
      if (lane < n_boxes) {
        const int tok = base + lane * bt_tok;
        int blk = bt[tok / p.block_size];
        if (blk < 0 || blk >= p.num_blocks_total) blk = 0;
        z = blk * p.block_size + tok % p.block_size;
      }
      for (int i = 0; i < per_tile; ++i) {
        if (lane == 0) {
          if (!mbar_wait(&bars->empty[at.slot], at.phase ^ 1)) {
            atomicExch(p.status, XL_ERR_WAIT_EMPTY);
            ok = false;
          } else if (part == 0) {
            mbar_arrive_expect_tx(&bars->full[at.slot], uint32_t(n_boxes) * bt_tok * 128);
          } else {
            mbar_arrive(&bars->full[at.slot]);             // also without a box of its own: no producer falls a round behind
          }
        }
        ok = __shfl_sync(0xffffffffu, ok, 0);
        if (!ok) break;
        if (lane < n_boxes && lane % kWideProducers == part) {
          uint8_t* dst = ring + at.slot * kWideSlab + lane * bt_tok * 128;
          if (i < KS) tma_load_3d(dst, &tmK, &bars->full[at.slot], i * 64, 0, z);
          else tma_load_3d(dst, &tmV, &bars->full[at.slot], (i - KS) % VH * 64, v_first + (i - KS) / VH, z);
        }
        __syncwarp();
        at.next(n_slabs);
        ++issued;
      }
    }
    if (!ok && lane == 0) {  // let the copies already issued land (bounded) before the CTA retires
      for (int back = min(issued, n_slabs); back > 0; --back) {
        const int j = issued - back;
        mbar_wait(&bars->full[j % n_slabs], (j / n_slabs) & 1);
      }
    }
  } else {
    // ------------------------------------------------------------ consumers
    const int row_a = lane >> 2;
    int lim[MT][2], vh[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = mt * 16 + row_a + 8 * e, m = row0 + (r < rows ? r : 0);
        lim[mt][e] = kv_len - q_len + m / p.n_q;
        vh[mt][e] = r < rows ? m % p.n_q / group : -1;
      }
    const int rk = (lane & 7) + (lane >> 4) * 8;           // K fragment row (token) of this lane
    const int rv = (lane & 7) + ((lane >> 3) & 1) * 8;     // V fragment row (token), and Q fragment row
    const uint32_t q_row = smem_u32(sQ + uint32_t(rv) * (KS * 128)), ring_u = smem_u32(ring) + warp * 2048;
    bool ok = true;
    auto take = [&]() -> bool {
      if (mbar_wait(&bars->full[at.slot], at.phase)) return true;
      if (lane == 0) atomicExch(p.status, XL_ERR_WAIT_FULL);
      return false;
    };
    auto give = [&]() {
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->empty[at.slot]);
      at.next(n_slabs);
    };
    for (int t = 0; t < n_tiles && ok; ++t) {
      const int base = r_begin + (t_first + t) * kWideTile + warp * 16;
      const bool mine = base < kv_len;
      float sc[MT][2][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < 2; ++i) sc[mt][i][0] = sc[mt][i][1] = sc[mt][i][2] = sc[mt][i][3] = 0.f;
      for (int ks = 0; ks < KS; ++ks) {
        if (!(ok = take())) break;
        if (mine) {
          const uint32_t tK = ring_u + at.slot * kWideSlab + rk * 128;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4(tK + (((i * 2 + ((lane >> 3) & 1)) ^ (rk & 7)) << 4), b0, b1, b2, b3);
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
              uint32_t a[4];
              ldsm_x4(q_row + mt * 16 * KS * 128 + (uint32_t((ks * 8 + i * 2 + (lane >> 4)) ^ (rv & 7)) << 4), a[0], a[1], a[2], a[3]);
              mma_bf16_16816(sc[mt][0], a, b0, b1);
              mma_bf16_16816(sc[mt][1], a, b2, b3);
            }
          }
        }
        give();
      }
      if (!ok) break;
      uint32_t pa[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        pa[mt][0] = pa[mt][1] = pa[mt][2] = pa[mt][3] = 0;
        if (!mine) continue;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int tok = base + i * 8 + (lane & 3) * 2 + (e & 1);
            const int l = lim[mt][e >> 1];
            const bool see = tok <= l && tok < kv_len && (p.window <= 0 || tok > l - p.window);
            sc[mt][i][e] = see ? sc[mt][i][e] * p.scale_log2 : -INFINITY;
            mx[e >> 1] = fmaxf(mx[e >> 1], sc[mt][i][e]);
          }
        }
        float alpha[2];
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
          mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
          const float m_new = fmaxf(m_run[mt][h], mx[h]);
          alpha[h] = (m_new == -INFINITY) ? 1.f : exp2f(m_run[mt][h] - m_new);
          m_run[mt][h] = m_new;
        }
        float rs[2] = {0.f, 0.f};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float m = m_run[mt][e >> 1];
            sc[mt][i][e] = (m == -INFINITY) ? 0.f : exp2f(sc[mt][i][e] - m);
            rs[e >> 1] += sc[mt][i][e];
          }
        }
        l_run[mt][0] = l_run[mt][0] * alpha[0] + rs[0];
        l_run[mt][1] = l_run[mt][1] * alpha[1] + rs[1];
        pa[mt][0] = pack_bf16x2(sc[mt][0][0], sc[mt][0][1]);
        pa[mt][1] = pack_bf16x2(sc[mt][0][2], sc[mt][0][3]);
        pa[mt][2] = pack_bf16x2(sc[mt][1][0], sc[mt][1][1]);
        pa[mt][3] = pack_bf16x2(sc[mt][1][2], sc[mt][1][3]);
        if (alpha[0] != 1.f || alpha[1] != 1.f) {
#pragma unroll
          for (int i = 0; i < DV / 8; ++i) {
            o[mt][i][0] *= alpha[0]; o[mt][i][1] *= alpha[0]; o[mt][i][2] *= alpha[1]; o[mt][i][3] *= alpha[1];
          }
        }
      }
      for (int v = v_first; v <= v_last && ok; ++v) {
        uint32_t pv[MT][4];
        bool any[MT];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          const bool ua = vh[mt][0] == v, ub = vh[mt][1] == v;
          any[mt] = __any_sync(0xffffffffu, ua || ub);
          pv[mt][0] = ua ? pa[mt][0] : 0u;
          pv[mt][1] = ub ? pa[mt][1] : 0u;
          pv[mt][2] = ua ? pa[mt][2] : 0u;
          pv[mt][3] = ub ? pa[mt][3] : 0u;
        }
#pragma unroll
        for (int vs = 0; vs < VH; ++vs) {
          if (!(ok = take())) break;
          if (mine) {
            const uint32_t tV = ring_u + at.slot * kWideSlab + rv * 128;
#pragma unroll
            for (int d = 0; d < 4; ++d) {
              uint32_t b0, b1, b2, b3;
              ldsm_x4_t(tV + (((d * 2 + (lane >> 4)) ^ (rv & 7)) << 4), b0, b1, b2, b3);
#pragma unroll
              for (int mt = 0; mt < MT; ++mt) {
                if (!any[mt]) continue;
                mma_bf16_16816(o[mt][vs * 8 + 2 * d], pv[mt], b0, b1);
                mma_bf16_16816(o[mt][vs * 8 + 2 * d + 1], pv[mt], b2, b3);
              }
            }
          }
          give();
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        l_run[mt][h] += __shfl_xor_sync(0xffffffffu, l_run[mt][h], 1);
        l_run[mt][h] += __shfl_xor_sync(0xffffffffu, l_run[mt][h], 2);
      }
  }
  __syncthreads();   // ring no longer needed: reuse it for the merge

  float* sO = reinterpret_cast<float*>(ring);     // [CW][ROWS][DV]
  if (warp < CW) {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = mt * 16 + (lane >> 2) + 8 * h;
        float* dst = sO + (warp * ROWS + r) * DV + (lane & 3) * 2;
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) *reinterpret_cast<float2*>(dst + i * 8) = make_float2(o[mt][i][2 * h], o[mt][i][2 * h + 1]);
        if ((lane & 3) == 0) {
          sM[warp * ROWS + r] = m_run[mt][h];
          sL[warp * ROWS + r] = l_run[mt][h];
        }
      }
  }
  __syncthreads();
  if (warp >= CW) return;
  for (int r = warp; r < rows; r += CW) {
    float m = -INFINITY, w[CW], l = 0.f;
#pragma unroll
    for (int j = 0; j < CW; ++j) m = fmaxf(m, sM[j * ROWS + r]);
#pragma unroll
    for (int j = 0; j < CW; ++j) {
      w[j] = sM[j * ROWS + r] == -INFINITY ? 0.f : exp2f(sM[j * ROWS + r] - m);
      l += w[j] * sL[j * ROWS + r];
    }
    const int hq = (row0 + r) % p.n_q;
    float den = l;                                // the sink joins once: here, or in the merge of the splits
    if (p.sinks && p.num_splits == 1 && m != -INFINITY) den += exp2f(p.sinks[hq] * kL2e - m);
    const float inv = den > 0.f ? 1.f / den : 0.f;
    const size_t tok = size_t(q_start + (row0 + r) / p.n_q);
    for (int col = lane * 2; col < dv; col += 64) {
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int j = 0; j < CW; ++j) {
        const float2 f = *reinterpret_cast<const float2*>(sO + (j * ROWS + r) * DV + col);
        a += w[j] * f.x;
        b += w[j] * f.y;
      }
      if (p.num_splits == 1)
        *reinterpret_cast<uint32_t*>(p.out + tok * (size_t(p.n_q) * dv) + hq * dv + col) = pack_bf16x2(a * inv, b * inv);
      else
        *reinterpret_cast<float2*>(p.part_o + ((tok * p.n_q + hq) * p.num_splits + split) * dv + col) = make_float2(a * inv, b * inv);
    }
    if (p.num_splits > 1 && lane == 0)
      p.part_lse[(tok * p.n_q + hq) * p.num_splits + split] = (l > 0.f) ? m + log2f(l) : -INFINITY;
  }
}

// 1 (launched nothing): the query rows and the merge do not fit shared memory
template <int MT, int DV>
static int launch_wide(const CUtensorMap* tk, const CUtensorMap* tv, const DecParams& p, int max_q, cudaStream_t st) {
  const int KS = (p.dk + 63) / 64;
  const size_t rest = size_t(16 * MT) * KS * 128 + sizeof(WideDecBarriers) + size_t(2) * kWideConsumers * 16 * MT * 4 + 1024;
  const size_t merge = size_t(kWideConsumers) * 16 * MT * DV * 4, room = size_t(227) * 1024;
  if (rest + merge > room) return 1;
  int n = int((room - rest) / kWideSlab);
  if (n > kWideMost) n = kWideMost;
  if (size_t(n) * kWideSlab < merge || n < 2) return 1;
  const size_t smem = rest + size_t(n) * kWideSlab;
  const dim3 grid((p.n_q * max_q + 16 * MT - 1) / (16 * MT), p.seq_end - p.seq_begin, p.num_splits);   // a sequence's blocks side by side
  if (grid.y > 65535) return -3;
  cudaFuncSetAttribute(decode_attn_wide_kernel<MT, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
  decode_attn_wide_kernel<MT, DV><<<grid, kWideThreads, smem, st>>>(*tk, *tv, p, KS, n);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}
template <int DV>
static int launch_wide_rows(const CUtensorMap* tk, const CUtensorMap* tv, const DecParams& p, int max_q, cudaStream_t st) {
  int rc = 1;
  if (p.n_q * max_q > 16) rc = launch_wide<2, DV>(tk, tv, p, max_q, st);
  if (rc == 1) rc = launch_wide<1, DV>(tk, tv, p, max_q, st);
  return rc == 1 ? -3 : rc;
}

}  // namespace xl_dec

using namespace xl_dec;

// Launches the TMA decode kernel for sequences [seq_begin, seq_end).  Returns -3 when the shape is not covered
// (block size not a multiple of 16, head_dim other than 64/128): the caller then uses the cp.async kernel.
// The split-KV merge (when num_splits > 1) is launched by the caller.
// `dyn_end` (device int pointer, may be null) replaces seq_end at run time; the launch is then sized for
// [seq_begin, seq_end) as a capacity, which lets a captured graph replay with another number of decode sequences.
XL_API int xl_decode_attention_tma_dyn(const void* q, const void* k_cache, const void* v_cache, void* out, const void* q_cu,
                                       const void* kv_lens, const void* block_tables, int seq_begin, int seq_end,
                                       int max_blocks, int block_size, int num_blocks_total, int n_q, int n_kv, int head_dim,
                                       int q_stride, float scale, int window, int num_splits, void* part_o, void* part_lse,
                                       const void* dyn_end, void* stream) {
  if (seq_end <= seq_begin) return 0;
  if (head_dim != 128 && head_dim != 64) return -3;
  if (block_size % 16 != 0 || (block_size > 64 && block_size % 64 != 0) || (block_size < 64 && 64 % block_size != 0)) return -3;
  if (n_q % n_kv || n_q / n_kv > 16) return -3;
  if ((reinterpret_cast<uintptr_t>(k_cache) & 127) || (reinterpret_cast<uintptr_t>(v_cache) & 127)) return -3;
  const int box_tokens = block_size < 64 ? block_size : 64;
  const uint64_t slots = uint64_t(num_blocks_total) * block_size;
  const CUtensorMap* tk = xl_host::tmap_3d(k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, slots, n_kv, head_dim, box_tokens, 1, 64,
                                           CU_TENSOR_MAP_SWIZZLE_128B);
  const CUtensorMap* tv = xl_host::tmap_3d(v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, slots, n_kv, head_dim, box_tokens, 1, 64,
                                           CU_TENSOR_MAP_SWIZZLE_128B);
  if (!tk || !tv) return -3;
  DecParams p;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.q_cu = static_cast<const int*>(q_cu);
  p.kv_lens = static_cast<const int*>(kv_lens);
  p.block_tables = static_cast<const int*>(block_tables);
  p.seq_begin = seq_begin; p.seq_end = seq_end;
  p.max_blocks = max_blocks; p.block_size = block_size; p.n_q = n_q; p.n_kv = n_kv; p.q_stride = q_stride;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.window = window;
  p.num_splits = num_splits < 1 ? 1 : num_splits;
  p.part_o = static_cast<float*>(part_o);
  p.part_lse = static_cast<float*>(part_lse);
  p.num_blocks_total = num_blocks_total;
  p.box_tokens = box_tokens;
  p.status = xl_host::status_word();
  p.dyn_end = static_cast<const int*>(dyn_end);
  if (p.num_splits > 1 && (!part_o || !part_lse)) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  dim3 grid(seq_end - seq_begin, n_kv, p.num_splits);
  if (head_dim == 128) {
    const size_t ring = size_t(kStages) * 2 * 2 * kTile * 128;
    const size_t merge = 4 * 16 * 128 * 4 + 128 * 4;
    const size_t smem = (ring > merge ? ring : merge) + 16 * 128 * 2 + sizeof(DecBarriers) + 1024;
    static bool set = false;
    if (!set) { cudaFuncSetAttribute(decode_attn_tma_kernel<128, 128, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)); set = true; }
    decode_attn_tma_kernel<128, 128, false><<<grid, 160, smem, st>>>(*tk, *tv, p);
  } else {
    const size_t ring = size_t(kStages) * 2 * 1 * kTile * 128;
    const size_t merge = 4 * 16 * 64 * 4 + 128 * 4;
    const size_t smem = (ring > merge ? ring : merge) + 16 * 64 * 2 + sizeof(DecBarriers) + 1024;
    static bool set = false;
    if (!set) { cudaFuncSetAttribute(decode_attn_tma_kernel<64, 64, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)); set = true; }
    decode_attn_tma_kernel<64, 64, false><<<grid, 160, smem, st>>>(*tk, *tv, p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

XL_API int xl_decode_attention_tma(const void* q, const void* k_cache, const void* v_cache, void* out, const void* q_cu,
                                   const void* kv_lens, const void* block_tables, int seq_begin, int seq_end, int max_blocks,
                                   int block_size, int num_blocks_total, int n_q, int n_kv, int head_dim, int q_stride,
                                   float scale, int window, int num_splits, void* part_o, void* part_lse, void* stream) {
  return xl_decode_attention_tma_dyn(q, k_cache, v_cache, out, q_cu, kv_lens, block_tables, seq_begin, seq_end, max_blocks,
                                     block_size, num_blocks_total, n_q, n_kv, head_dim, q_stride, scale, window, num_splits,
                                     part_o, part_lse, nullptr, stream);
}

namespace xl_dec {
// merge of split-KV partials (normalised partial outputs weighted by 2^lse): one warp per (token, head)
template <int D>
__global__ void split_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse,
                                   __nv_bfloat16* __restrict__ out, const int* __restrict__ q_cu, int seq_begin, int seq_end,
                                   int n_q, int splits, const int* dyn_end = nullptr, int ws_rows = 0, int group = 1,
                                   int* status = nullptr) {
  const int lane = threadIdx.x & 31;
  const long gw = (blockIdx.x * long(blockDim.x) + threadIdx.x) >> 5;
  if (dyn_end) seq_end = *dyn_end;
  if (seq_end <= seq_begin) return;
  const int t0 = q_cu[seq_begin], t1 = q_cu[seq_end];
  const long n = long(t1 - t0) * n_q;
  if (gw >= n) return;
  const size_t tok = size_t(t0) + size_t(gw / n_q);
  const int h = int(gw % n_q);
  if (ws_rows > 0) {
    // fixed-size workspace: a token outside it, or one of a sequence that the attention kernel skipped (more than 16
    // query rows x heads per kv head), has no partial results; leave its output alone and report
    int lo = seq_begin, hi = seq_end;                         // the sequence with q_cu[lo] <= tok < q_cu[lo + 1]
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (size_t(q_cu[mid]) <= tok) lo = mid; else hi = mid;
    }
    const int q_len = q_cu[lo + 1] - q_cu[lo];
    if (q_cu[lo + 1] > ws_rows || q_len * group > 16) {
      if (lane == 0 && status) atomicExch(status, XL_ERR_BOUNDS);
      return;
    }
  }
  const float* lse = part_lse + (tok * n_q + h) * splits;
  float m = -INFINITY;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, lse[s]);
  float acc[D / 32];
#pragma unroll
  for (int i = 0; i < D / 32; ++i) acc[i] = 0.f;
  float den = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float w = (lse[s] == -INFINITY) ? 0.f : exp2f(lse[s] - m);
    den += w;
    const float* po = part_o + ((tok * n_q + h) * splits + s) * D;
#pragma unroll
    for (int i = 0; i < D / 32; ++i) acc[i] += w * po[lane + 32 * i];
  }
  const float inv = den > 0.f ? 1.f / den : 0.f;
#pragma unroll
  for (int i = 0; i < D / 32; ++i) out[tok * (size_t(n_q) * D) + h * D + lane + 32 * i] = __float2bfloat16(acc[i] * inv);
}
}  // namespace xl_dec

// `max_rows` bounds the number of query tokens of sequences [seq_begin, seq_end) (the real count is read on the device).
XL_API int xl_decode_split_merge_dyn(const void* part_o, const void* part_lse, void* out, const void* q_cu, int seq_begin,
                                     int seq_end, int n_q, int head_dim, int splits, long max_rows, const void* dyn_end_v,
                                     void* stream) {
  if (seq_end <= seq_begin || splits <= 1) return 0;
  const int* dyn_end = static_cast<const int*>(dyn_end_v);
  const long warps = max_rows * n_q;
  const int blocks = int((warps + 3) / 4);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (head_dim == 128)
    xl_dec::split_merge_kernel<128><<<blocks, 128, 0, st>>>(static_cast<const float*>(part_o), static_cast<const float*>(part_lse),
                                                            static_cast<__nv_bfloat16*>(out), static_cast<const int*>(q_cu),
                                                            seq_begin, seq_end, n_q, splits, dyn_end);
  else if (head_dim == 64)
    xl_dec::split_merge_kernel<64><<<blocks, 128, 0, st>>>(static_cast<const float*>(part_o), static_cast<const float*>(part_lse),
                                                           static_cast<__nv_bfloat16*>(out), static_cast<const int*>(q_cu),
                                                           seq_begin, seq_end, n_q, splits, dyn_end);
  else
    return -2;
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

XL_API int xl_decode_split_merge(const void* part_o, const void* part_lse, void* out, const void* q_cu, int seq_begin,
                                 int seq_end, int n_q, int head_dim, int splits, long max_rows, void* stream) {
  return xl_decode_split_merge_dyn(part_o, part_lse, out, q_cu, seq_begin, seq_end, n_q, head_dim, splits, max_rows, nullptr, stream);
}

// ============================================================================ score extensions
namespace xl_dec {
template <int DK, int DV, bool CAP>
static int launch_ext_as(const CUtensorMap* tk, const CUtensorMap* tv, const DecParams& p, dim3 grid, cudaStream_t st) {
  const size_t ring = size_t(kStages) * (DK / 64 + DV / 64) * kTile * 128;
  const size_t merge = 4 * 16 * DV * 4 + 128 * 4;
  const size_t smem = (ring > merge ? ring : merge) + 16 * DK * 2 + sizeof(DecBarriers) + 1024;
  static bool set = false;
  if (!set) {
    cudaFuncSetAttribute(decode_attn_tma_kernel<DK, DV, true, CAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    set = true;
  }
  decode_attn_tma_kernel<DK, DV, true, CAP><<<grid, 160, smem, st>>>(*tk, *tv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

template <int DK, int DV>
static int launch_ext(const CUtensorMap* tk, const CUtensorMap* tv, const DecParams& p, dim3 grid, cudaStream_t st) {
  return p.cap_out > 0.f ? launch_ext_as<DK, DV, true>(tk, tv, p, grid, st) : launch_ext_as<DK, DV, false>(tk, tv, p, grid, st);
}

// merge of split-KV partials for any value head dimension, with the sink's share of the denominator: one warp per
// (token, head)
__global__ void split_merge_ext_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse,
                                       __nv_bfloat16* __restrict__ out, const int* __restrict__ q_cu, int seq_begin, int seq_end,
                                       int n_q, int dv, int splits, const float* __restrict__ sinks, const int* dyn_end) {
  const int lane = threadIdx.x & 31;
  const long gw = (blockIdx.x * long(blockDim.x) + threadIdx.x) >> 5;
  if (dyn_end) seq_end = *dyn_end;
  if (seq_end <= seq_begin) return;
  const int t0 = q_cu[seq_begin], t1 = q_cu[seq_end];
  if (gw >= long(t1 - t0) * n_q) return;
  const size_t tok = size_t(t0) + size_t(gw / n_q);
  const int h = int(gw % n_q);
  const float* lse = part_lse + (tok * n_q + h) * splits;
  const float sink = sinks ? sinks[h] * 1.4426950408889634f : -INFINITY;
  float m = sink;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, lse[s]);
  float den = sinks ? exp2f(sink - m) : 0.f;
  for (int s = 0; s < splits; ++s) den += lse[s] == -INFINITY ? 0.f : exp2f(lse[s] - m);
  const float inv = den > 0.f ? 1.f / den : 0.f;
  for (int c = lane; c < dv; c += 32) {
    float acc = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float w = lse[s] == -INFINITY ? 0.f : exp2f(lse[s] - m);
      if (w != 0.f) acc += w * part_o[((tok * n_q + h) * splits + s) * dv + c];
    }
    out[tok * (size_t(n_q) * dv) + h * dv + c] = __float2bfloat16(acc * inv);
  }
}

// The same for differential attention: one warp per (token, output head) merges both maps and stores their normed difference.
__global__ void split_merge_mix_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse,
                                       __nv_bfloat16* __restrict__ out, const int* __restrict__ q_cu, int seq_begin, int seq_end,
                                       int n_q, int dv, int splits, const float* __restrict__ sinks, const float* __restrict__ mix,
                                       float mult, float eps, const int* dyn_end) {
  const int lane = threadIdx.x & 31;
  const long gw = (blockIdx.x * long(blockDim.x) + threadIdx.x) >> 5;
  if (dyn_end) seq_end = *dyn_end;
  if (seq_end <= seq_begin) return;
  const int t0 = q_cu[seq_begin], t1 = q_cu[seq_end], heads = n_q / 2;
  if (gw >= long(t1 - t0) * heads) return;
  const size_t tok = size_t(t0) + size_t(gw / heads);
  const int head = int(gw % heads);
  constexpr int kCols = 8;                              // dv <= 256
  float d[kCols];
#pragma unroll
  for (int c = 0; c < kCols; ++c) d[c] = 0.f;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const size_t row = tok * n_q + 2 * head + k;
    const float* lse = part_lse + row * splits;
    const float sink = sinks ? sinks[2 * head + k] * 1.4426950408889634f : -INFINITY;
    float m = sink;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, lse[s]);
    float den = sinks ? exp2f(sink - m) : 0.f;
    for (int s = 0; s < splits; ++s) den += lse[s] == -INFINITY ? 0.f : exp2f(lse[s] - m);
    const float f = (den > 0.f ? 1.f / den : 0.f) * (k == 0 ? 1.f : -*mix);
    for (int s = 0; s < splits; ++s) {
      const float w = lse[s] == -INFINITY ? 0.f : exp2f(lse[s] - m) * f;
      if (w == 0.f) continue;
      const float* po = part_o + (row * splits + s) * dv;
#pragma unroll
      for (int c = 0; c < kCols; ++c)
        if (c * 32 + lane < dv) d[c] += w * po[c * 32 + lane];
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < kCols; ++c) ss += d[c] * d[c];
  const float s = rsqrtf(warp_sum(ss) / float(dv) + eps) * mult;
#pragma unroll
  for (int c = 0; c < kCols; ++c)
    if (c * 32 + lane < dv) out[tok * (size_t(heads) * dv) + head * dv + c * 32 + lane] = __float2bfloat16(d[c] * s);
}
}  // namespace xl_dec

// Decode attention with the score extensions of xl_prefill_attention_ext (head dimensions: multiples of 8, at most 256; with
// maps = 2 the keys of both maps together).  With num_splits > 1 the partials are merged by a second kernel; `max_rows` bounds the
// query tokens of the launch, `max_q` those of a sequence.
XL_API int xl_decode_attention_ext(const void* q, const void* k_cache, const void* v_cache, void* out, const void* q_cu,
                                   const void* kv_lens, const void* block_tables, int seq_begin, int seq_end, int max_blocks,
                                   int block_size, int num_blocks_total, int n_q, int n_kv, int dk, int dv, int q_stride,
                                   float scale, int window, int chunk, int keep_first, const void* slopes, const void* sinks,
                                   float softcap, float bound, long v_pitch, int shared_keys, int maps, const void* mix, float mix_mult,
                                   float mix_eps, int max_q,
                                   int num_splits, void* part_o, void* part_lse, long max_rows, const void* dyn_end, void* stream) {
  using namespace xl_dec;
  if (seq_end <= seq_begin) return 0;
  if (chunk > 0 && keep_first > 0) return -2;
  if (maps < 1 || maps > 2 || (maps == 2 && (!mix || shared_keys || (n_q / n_kv) % 2))) return -2;
  if (dk < 8 || dk % 8) return -3;
  dk *= maps;                                  // the keys of both maps lie side by side
  // keys that all heads share may be wider, without the other score extensions
  const bool wide_keys = shared_keys && dk > 128 && dv <= 128 && !slopes && softcap <= 0.f && chunk <= 0 && keep_first <= 0;
  if ((dk > 256 && !wide_keys) || dv < 8 || dv > 256 || dv % 8 || v_pitch % 8) return -3;
  if (block_size % 16 != 0 || (block_size > 64 && block_size % 64 != 0) || (block_size < 64 && 64 % block_size != 0)) return -3;
  if (n_q % n_kv) return -3;
  if ((q_stride % 8) || (reinterpret_cast<uintptr_t>(q) & 15)) return -3;
  if ((reinterpret_cast<uintptr_t>(k_cache) & 127) || (reinterpret_cast<uintptr_t>(v_cache) & 127)) return -3;
  const int box_tokens = block_size < 64 ? block_size : 64;
  const uint64_t slots = uint64_t(num_blocks_total) * block_size;
  const CUtensorMap* tk = xl_host::tmap_3d(k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, slots, shared_keys ? 1 : n_kv, dk, box_tokens, 1, 64,
                                           CU_TENSOR_MAP_SWIZZLE_128B);
  const CUtensorMap* tv = xl_host::tmap_3d(v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, slots, n_kv, dv, box_tokens, 1, 64,
                                           CU_TENSOR_MAP_SWIZZLE_128B, v_pitch);
  if (!tk || !tv) return -3;
  DecParams p;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.q_cu = static_cast<const int*>(q_cu);
  p.kv_lens = static_cast<const int*>(kv_lens);
  p.block_tables = static_cast<const int*>(block_tables);
  p.seq_begin = seq_begin; p.seq_end = seq_end;
  p.max_blocks = max_blocks; p.block_size = block_size; p.n_q = n_q; p.n_kv = n_kv; p.q_stride = q_stride;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.window = window;
  p.num_splits = num_splits < 1 ? 1 : num_splits;
  p.part_o = static_cast<float*>(part_o);
  p.part_lse = static_cast<float*>(part_lse);
  p.num_blocks_total = num_blocks_total;
  p.box_tokens = box_tokens;
  p.status = xl_host::status_word();
  p.dyn_end = static_cast<const int*>(dyn_end);
  p.dk = dk; p.dv = dv; p.chunk = chunk; p.keep_first = keep_first;
  p.slopes = static_cast<const float*>(slopes);
  p.sinks = static_cast<const float*>(sinks);
  p.row_blocks = (n_q / n_kv * (max_q < 1 ? 1 : max_q) + 15) / 16;
  p.maps = maps;
  p.shared_keys = shared_keys;
  if (softcap > 0.f) {
    p.cap_in = scale / softcap;
    p.cap_out = softcap * 1.4426950408889634f;
    p.cap_level = cap_level(p.cap_in, bound) == CAP_SMALL ? CAP_SMALL : CAP_CHECK;    // a check finds most rows small
  }
  p.mix = static_cast<const float*>(mix);
  p.mix_mult = mix_mult; p.mix_eps = mix_eps;
  if (p.num_splits > 1 && (!part_o || !part_lse)) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const dim3 grid(seq_end - seq_begin, n_kv * p.row_blocks, p.num_splits);
  int rc;
  if (wide_keys) rc = dv > 64 ? launch_wide_rows<128>(tk, tv, p, max_q < 1 ? 1 : max_q, st) : launch_wide_rows<64>(tk, tv, p, max_q < 1 ? 1 : max_q, st);
  else if (dv > 128) rc = launch_ext<256, 256>(tk, tv, p, grid, st);
  else if (dk > 128) rc = launch_ext<256, 128>(tk, tv, p, grid, st);
  else if (dk > 64) rc = dv > 64 ? launch_ext<128, 128>(tk, tv, p, grid, st) : launch_ext<128, 64>(tk, tv, p, grid, st);
  else rc = dv > 64 ? launch_ext<64, 128>(tk, tv, p, grid, st) : launch_ext<64, 64>(tk, tv, p, grid, st);
  if (rc != 0 || p.num_splits == 1) return rc;
  if (maps == 2) {
    split_merge_mix_kernel<<<int((max_rows * (n_q / 2) + 3) / 4), 128, 0, st>>>(p.part_o, p.part_lse, p.out, p.q_cu, seq_begin, seq_end, n_q, dv,
                                                                                p.num_splits, p.sinks, p.mix, mix_mult, mix_eps, p.dyn_end);
    return cudaGetLastError() == cudaSuccess ? 0 : -1;
  }
  split_merge_ext_kernel<<<int((max_rows * n_q + 3) / 4), 128, 0, st>>>(p.part_o, p.part_lse, p.out, p.q_cu, seq_begin, seq_end, n_q, dv,
                                                                        p.num_splits, p.sinks, p.dyn_end);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

// ============================================================================ allocation-free entry point
// Declared in xllm_kernels.h.  Same kernels as above; the split-KV workspace and the status word live in
// file-scope device arrays instead of caller- or library-allocated memory.
namespace xl_dec {
constexpr size_t kNoAllocScratchBytes = size_t(16) << 20;            // 16 MiB, held by every GPU that loads the library
static __device__ __align__(256) unsigned char g_noalloc_scratch[kNoAllocScratchBytes];
static __device__ __align__(256) int g_noalloc_status[64];
static void* g_noalloc_scratch_addr[64] = {nullptr};                 // device addresses of the arrays, per device
static void* g_noalloc_status_addr[64] = {nullptr};

static void set_err(char* err, int err_len, const char* msg) {
  if (!err || err_len <= 0) return;
  int i = 0;
  for (; msg[i] && i < err_len - 1; ++i) err[i] = msg[i];
  err[i] = 0;
}
}  // namespace xl_dec

XL_API int xl_decode_attention_noalloc(const void* q, const void* k_cache, const void* v_cache, void* out, const void* q_cu,
                                       const void* kv_lens, const void* block_tables, int n_seqs, int max_rows, int max_blocks,
                                       int block_size, int num_blocks_total, int n_q, int n_kv, int head_dim, int q_stride,
                                       float scale, int num_splits, void* stream, char* err, int err_len) {
  using namespace xl_dec;
  if (n_seqs <= 0) return 0;
  if (head_dim != 128 && head_dim != 64) { set_err(err, err_len, "head_dim must be 64 or 128"); return -3; }
  if (block_size % 16 != 0 || (block_size > 64 && block_size % 64 != 0) || (block_size < 64 && 64 % block_size != 0)) {
    set_err(err, err_len, "block_size must be 16, 32, 64 or a multiple of 64");
    return -3;
  }
  if (n_kv <= 0 || n_q % n_kv || n_q / n_kv > 16) { set_err(err, err_len, "n_q must be a multiple of n_kv, group <= 16"); return -3; }
  if (num_splits < 1) num_splits = 1;
  if (max_rows < n_seqs) max_rows = n_seqs;
  const size_t o_bytes = size_t(max_rows) * n_q * num_splits * head_dim * sizeof(float);
  const size_t lse_bytes = size_t(max_rows) * n_q * num_splits * sizeof(float);
  if (num_splits > 1 && o_bytes + lse_bytes > kNoAllocScratchBytes) {
    set_err(err, err_len, "split-KV workspace (max_rows * n_q * num_splits * (head_dim + 1) * 4 bytes) exceeds the 16 MiB built-in scratch: "
                          "use fewer splits or fewer rows per call");
    return -5;
  }
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) { set_err(err, err_len, "no current CUDA device"); return -1; }
  if (!g_noalloc_scratch_addr[dev]) {
    // once per device, with that device current: the arrays' names are host-side handles, not device addresses
    void* a = nullptr;
    void* b = nullptr;
    if (cudaGetSymbolAddress(&a, g_noalloc_scratch) != cudaSuccess || cudaGetSymbolAddress(&b, g_noalloc_status) != cudaSuccess ||
        !a || !b) {
      set_err(err, err_len, "cudaGetSymbolAddress failed for the built-in scratch");
      return -1;
    }
    g_noalloc_scratch_addr[dev] = a;
    g_noalloc_status_addr[dev] = b;
  }
  const int box_tokens = block_size < 64 ? block_size : 64;
  CUtensorMap tk, tv;                                              // encoded on the stack: nothing is cached or allocated
  {
    const uint64_t slots = uint64_t(num_blocks_total) * block_size;
    uint64_t dims[3] = {uint64_t(head_dim), uint64_t(n_kv), slots};
    uint64_t strides[2] = {uint64_t(head_dim) * 2, uint64_t(head_dim) * n_kv * 2};
    uint32_t box[3] = {64, 1, uint32_t(box_tokens)};
    if (xl_host::encode_tiled(&tk, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, k_cache, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B) != CUDA_SUCCESS ||
        xl_host::encode_tiled(&tv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, v_cache, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B) != CUDA_SUCCESS) {
      set_err(err, err_len, "tensor-map encoding failed (cache base must be 16-byte aligned)");
      return -4;
    }
  }
  DecParams p;
  p.q = static_cast<const __nv_bfloat16*>(q);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.q_cu = static_cast<const int*>(q_cu);
  p.kv_lens = static_cast<const int*>(kv_lens);
  p.block_tables = static_cast<const int*>(block_tables);
  p.seq_begin = 0; p.seq_end = n_seqs;
  p.max_blocks = max_blocks; p.block_size = block_size; p.n_q = n_q; p.n_kv = n_kv; p.q_stride = q_stride;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.window = -1;
  p.num_splits = num_splits;
  p.part_o = reinterpret_cast<float*>(g_noalloc_scratch_addr[dev]);
  p.part_lse = reinterpret_cast<float*>(static_cast<unsigned char*>(g_noalloc_scratch_addr[dev]) + o_bytes);
  p.num_blocks_total = num_blocks_total;
  p.box_tokens = box_tokens;
  p.status = static_cast<int*>(g_noalloc_status_addr[dev]);
  // rows the built-in workspace has room for with this head count and split count (checked again on the device, where
  // the real q_cu is known)
  p.ws_rows = num_splits > 1 ? int(kNoAllocScratchBytes / (size_t(n_q) * num_splits * (head_dim + 1) * sizeof(float))) : 0x7fffffff;
  if (p.ws_rows > max_rows) p.ws_rows = max_rows;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  dim3 grid(n_seqs, n_kv, num_splits);
  if (head_dim == 128) {
    const size_t ring = size_t(kStages) * 2 * 2 * kTile * 128;
    const size_t smem = ring + 16 * 128 * 2 + sizeof(DecBarriers) + 1024;
    cudaFuncSetAttribute(decode_attn_tma_kernel<128, 128, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    decode_attn_tma_kernel<128, 128, false><<<grid, 160, smem, st>>>(tk, tv, p);
    if (num_splits > 1)
      split_merge_kernel<128><<<int((long(max_rows) * n_q + 3) / 4), 128, 0, st>>>(p.part_o, p.part_lse, p.out, p.q_cu, 0, n_seqs, n_q,
                                                                                  num_splits, nullptr, p.ws_rows, n_q / n_kv, p.status);
  } else {
    const size_t ring = size_t(kStages) * 2 * 1 * kTile * 128;
    const size_t smem = ring + 16 * 64 * 2 + sizeof(DecBarriers) + 1024;
    cudaFuncSetAttribute(decode_attn_tma_kernel<64, 64, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    decode_attn_tma_kernel<64, 64, false><<<grid, 160, smem, st>>>(tk, tv, p);
    if (num_splits > 1)
      split_merge_kernel<64><<<int((long(max_rows) * n_q + 3) / 4), 128, 0, st>>>(p.part_o, p.part_lse, p.out, p.q_cu, 0, n_seqs, n_q,
                                                                                 num_splits, nullptr, p.ws_rows, n_q / n_kv, p.status);
  }
  if (cudaGetLastError() != cudaSuccess) { set_err(err, err_len, "kernel launch failed"); return -1; }
  return 0;
}

// Status of the allocation-free entry point on the current device: 0, or the code that one of its kernels recorded since
// the last call of this function (XL_ERR_WAIT_* = a bounded wait on the TMA ring expired, XL_ERR_BOUNDS = a sequence did
// not fit the built-in workspace or had more than 16 query rows x heads per kv head and was skipped).  Waits for the
// work queued on `stream`, reads the word with one copy and clears it; allocates nothing.  Returns -1 when the entry
// point has not run on this device yet or a CUDA call fails.
XL_API int xl_decode_attention_noalloc_status(void* stream) {
  using namespace xl_dec;
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64 || !g_noalloc_status_addr[dev]) return -1;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int v = 0;
  if (cudaMemcpyAsync(&v, g_noalloc_status_addr[dev], sizeof(int), cudaMemcpyDeviceToHost, st) != cudaSuccess) return -1;
  if (cudaStreamSynchronize(st) != cudaSuccess) return -1;
  if (v != 0 && cudaMemsetAsync(g_noalloc_status_addr[dev], 0, sizeof(int), st) != cudaSuccess) return -1;
  return v;
}
