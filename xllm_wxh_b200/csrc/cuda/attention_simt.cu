// Paged attention on the fp32 pipe, for what the tensor-core kernels do not serve: fp32 models (true 32-bit scores, weights
// and sums) and head dimensions beyond their limits.  One warp per (query token, query head): 32 keys at a time, one key
// per lane for the scores, then one slice of the value columns per lane for the weighted sum, with an online softmax.
//
// Serves prefill rows and decode rows alike, because every row finds its sequence and position in the step's own arrays.
// Score extensions (distance bias, sink, chunk mask, bounded scores) and differential attention (MAPS = 2: the warp walks the keys
// once per map and keeps the first map's output) as in xl_prefill_attention_ext.
#include "vec8.cuh"

namespace xl_as {
using namespace xl;

constexpr int kMaxCols = 16;      // value columns per lane: dv <= 512

template <typename T>
struct Params {
  const T* q;                     // [rows, n_q, dk], row pitch q_stride
  const T* k_cache;               // [slots, n_kv, dk]
  const T* v_cache;               // [slots, n_kv, dv]
  T* out;                         // [rows, n_q * dv]
  const int* token_seq;           // [rows] sequence of the row (-1: padding)
  const int* positions;           // [rows]
  const int* block_tables;        // [seqs, max_blocks]
  int rows, n_seqs, max_blocks, block_size, n_q, n_kv, dk, dv;
  long q_stride, cache_slots;
  float scale;
  int window, chunk, keep_first;
  const float* slopes;
  const float* sinks;
  float softcap;                  // > 0: bounded scores
  long v_pitch;                   // elements from one slot's values to the next one's
  int shared_keys;                // one key head for all value heads
  const float* mix;               // MAPS = 2
  float mix_mult, mix_eps;
};

template <typename T, int MAPS>
__global__ void __launch_bounds__(128) attention_simt_kernel(const Params<T> p) {
  extern __shared__ float s_q[];                 // one query vector per warp
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long item = blockIdx.x * long(blockDim.x >> 5) + warp;
  const int n_out = p.n_q / MAPS;                // output heads
  if (item >= long(p.rows) * n_out) return;
  const int t = int(item / n_out), h_out = int(item % n_out);
  const int seq = p.token_seq[t];
  if (seq < 0 || seq >= p.n_seqs) return;
  const int pos = p.positions[t];
  const int kvh = h_out / (n_out / p.n_kv);
  const int* bt = p.block_tables + size_t(seq) * p.max_blocks;
  float* q = s_q + warp * p.dk;
  float first[kMaxCols];                         // MAPS = 2: the first map's output
#pragma unroll
  for (int map = 0; map < MAPS; ++map) {
  const int h = h_out * MAPS + map, kh = p.shared_keys ? 0 : kvh * MAPS + map, n_kh = p.shared_keys ? 1 : p.n_kv * MAPS;
  __syncwarp();
  for (int i = lane; i < p.dk; i += 32) q[i] = to_f32(p.q[size_t(t) * p.q_stride + size_t(h) * p.dk + i]) * p.scale;
  __syncwarp();
  int lo = 0;
  if (p.window > 0) lo = max(lo, pos - p.window + 1);
  if (p.chunk > 0) lo = max(lo, pos / p.chunk * p.chunk);
  const float slope = p.slopes ? p.slopes[h] : 0.f;
  // the sink is a key with a known score and no value
  float m = p.sinks ? p.sinks[h] : -INFINITY, l = p.sinks ? 1.f : 0.f;
  float acc[kMaxCols];
#pragma unroll
  for (int c = 0; c < kMaxCols; ++c) acc[c] = 0.f;
  // visible keys in order: the kept first ones ahead of lo, then lo .. pos
  const int kept = min(p.keep_first, lo), n_keys = kept + pos - lo + 1;
  for (int base = 0; base < n_keys; base += 32) {
    const int idx = base + lane;
    const int key = idx < n_keys ? (idx < kept ? idx : lo + idx - kept) : pos + 1;
    float s = -INFINITY;
    long slot = 0;
    if (key <= pos) {
      const int b = min(key / p.block_size, p.max_blocks - 1);
      slot = long(bt[b]) * p.block_size + key % p.block_size;
      if (slot < 0 || slot >= p.cache_slots) slot = 0;
      const T* k = p.k_cache + (size_t(slot) * n_kh + kh) * p.dk;
      float d = 0.f;
      for (int i = 0; i < p.dk; ++i) d = fmaf(q[i], to_f32(k[i]), d);
      if (p.softcap > 0.f) d = act_softcap(d, p.softcap);
      s = d - slope * float(pos - key);
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
    const float w = key <= pos ? expf(s - m_new) : 0.f;
    l = l * alpha + warp_sum(w);
    m = m_new;
#pragma unroll
    for (int c = 0; c < kMaxCols; ++c) acc[c] *= alpha;
    const int n = min(32, n_keys - base);
    for (int j = 0; j < n; ++j) {
      const float wj = __shfl_sync(0xffffffffu, w, j);
      const long sj = __shfl_sync(0xffffffffu, slot, j);
      const T* v = p.v_cache + size_t(sj) * p.v_pitch + size_t(kvh) * p.dv;
#pragma unroll
      for (int c = 0; c < kMaxCols; ++c)
        if (c * 32 + lane < p.dv) acc[c] = fmaf(wj, to_f32(v[c * 32 + lane]), acc[c]);
    }
  }
  const float inv = 1.f / l;
  if (MAPS == 2 && map == 0) {
#pragma unroll
    for (int c = 0; c < kMaxCols; ++c) first[c] = acc[c] * inv;
    continue;
  }
  float s = inv;
  if (MAPS == 2) {
    const float f = *p.mix * inv;
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < kMaxCols; ++c) {           // columns past dv hold zeros
      acc[c] = first[c] - f * acc[c];
      ss += acc[c] * acc[c];
    }
    s = rsqrtf(warp_sum(ss) / float(p.dv) + p.mix_eps) * p.mix_mult;
  }
#pragma unroll
  for (int c = 0; c < kMaxCols; ++c)
    if (c * 32 + lane < p.dv) from_f32(p.out + (size_t(t) * n_out + h_out) * p.dv + c * 32 + lane, acc[c] * s);
  }
}

template <typename T>
static int launch(const void* q, const void* k_cache, const void* v_cache, void* out, const void* token_seq, const void* positions,
                  const void* block_tables, int rows, int n_seqs, int max_blocks, int block_size, long cache_slots, int n_q, int n_kv,
                  int dk, int dv, long q_stride, float scale, int window, int chunk, int keep_first, const void* slopes, const void* sinks,
                  float softcap, long v_pitch, int shared_keys, int maps, const void* mix, float mix_mult, float mix_eps, cudaStream_t st) {
  Params<T> p;
  p.q = static_cast<const T*>(q);
  p.k_cache = static_cast<const T*>(k_cache);
  p.v_cache = static_cast<const T*>(v_cache);
  p.out = static_cast<T*>(out);
  p.token_seq = static_cast<const int*>(token_seq);
  p.positions = static_cast<const int*>(positions);
  p.block_tables = static_cast<const int*>(block_tables);
  p.rows = rows; p.n_seqs = n_seqs; p.max_blocks = max_blocks; p.block_size = block_size;
  p.n_q = n_q; p.n_kv = n_kv; p.dk = dk; p.dv = dv;
  p.q_stride = q_stride; p.cache_slots = cache_slots;
  p.scale = scale; p.window = window; p.chunk = chunk; p.keep_first = keep_first;
  p.slopes = static_cast<const float*>(slopes);
  p.sinks = static_cast<const float*>(sinks);
  p.softcap = softcap;
  p.v_pitch = v_pitch > 0 ? v_pitch : long(n_kv) * dv;
  p.shared_keys = shared_keys;
  p.mix = static_cast<const float*>(mix);
  p.mix_mult = mix_mult; p.mix_eps = mix_eps;
  const long blocks = (long(rows) * (n_q / maps) + 3) / 4;
  const size_t smem = size_t(4) * dk * sizeof(float);
  auto kernel = maps == 2 ? attention_simt_kernel<T, 2> : attention_simt_kernel<T, 1>;
  if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
  kernel<<<int(blocks), 128, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

}  // namespace xl_as

// All rows of a step, prefill and decode.  `window` / `chunk` <= 0: none; `keep_first`: so many first keys stay visible; `slopes` /
// `sinks` [n_q] fp32 or null; the rest as in xl_prefill_attention_ext.
XL_API int xl_attention_simt(const void* q, const void* k_cache, const void* v_cache, void* out, const void* token_seq,
                             const void* positions, const void* block_tables, int rows, int n_seqs, int max_blocks, int block_size,
                             long cache_slots, int n_q, int n_kv, int dk, int dv, long q_stride, float scale, int window, int chunk,
                             int keep_first, const void* slopes, const void* sinks, float softcap, long v_pitch, int shared_keys, int maps,
                             const void* mix, float mix_mult, float mix_eps, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (maps < 1 || maps > 2 || (maps == 2 && (!mix || shared_keys || (n_q / n_kv) % 2))) return -2;
  if (n_kv <= 0 || n_q % n_kv || dk <= 0 || dk > 12288 || dv <= 0 || dv > 32 * xl_as::kMaxCols) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (f32)
    return xl_as::launch<float>(q, k_cache, v_cache, out, token_seq, positions, block_tables, rows, n_seqs, max_blocks, block_size,
                                cache_slots, n_q, n_kv, dk, dv, q_stride, scale, window, chunk, keep_first, slopes, sinks, softcap, v_pitch, shared_keys, maps, mix,
                                mix_mult, mix_eps, st);
  return xl_as::launch<__nv_bfloat16>(q, k_cache, v_cache, out, token_seq, positions, block_tables, rows, n_seqs, max_blocks, block_size,
                                      cache_slots, n_q, n_kv, dk, dv, q_stride, scale, window, chunk, keep_first, slopes, sinks, softcap, v_pitch, shared_keys, maps, mix,
                                mix_mult, mix_eps, st);
}
