// Layers with recurrent state, over ragged batches: every sequence of a step owns rows q_cu[i] .. q_cu[i + 1], the last ones
// of its kv_lens[i] tokens, and record slots[i] of the layer's state tensors.  A sequence whose rows start at position 0
// starts from zero, so a record needs no clearing when its slot changes hands.
//
//   token_shift     blends of every row with its predecessor (inputs of time mixing); keeps the last row
//   causal_conv     causal convolution per channel (+ silu, ahead of the selective scan); keeps the last inputs
//   matrix_*        matrix state per head (time mixing, gated linear attention, matrix memory); then RMS per head, weight and
//                   gate.  Single rows: one CTA streams a head's matrix through registers.  Longer portions: a portion
//                   is cut into segments; (A) every segment's own contribution to the state and its decay, (B) the states
//                   that the segments start from, (C) the segments' outputs from those, all in fp32
//   selective_scan  diagonal state space recurrence; its step sizes, decays, D x and silu(z) are part of the kernel
//
// All arithmetic is fp32 and states are fp32; other tensors are bf16, or fp32 when the model runs in 32-bit.
#include <type_traits>

#include "vec8.cuh"

namespace xl_rc {
using namespace xl;

struct Seqs {
  const int* q_cu;
  const int* kv_lens;
  const int* slots;
  int n;               // sequences (a capacity in padded steps: the rest has no rows)
  int n_slots;         // records in the state tensors
  int* status;
};

// Record of sequence s, or -1 (recorded in the status word) if it lies outside the state tensors.
__device__ __forceinline__ int record_of(const Seqs& q, int s) {
  const int slot = q.slots[s];
  if (slot < 0 || slot >= q.n_slots) {
    if (threadIdx.x == 0) atomicExch(q.status, XL_ERR_BOUNDS);
    return -1;
  }
  return slot;
}

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// log(1 + e^z) = max(z, 0) + log(1 + t), t = e^-|z| in (0, 1]; log(1 + t) = 2 artanh(s), s = t / (2 + t) <= 1 / 3, by its power
// series, which keeps the relative accuracy of small results (the next term is below 3e-9 of the sum).
__device__ __forceinline__ float softplus(float z) {
  const float t = __expf(-fabsf(z)), s = __fdividef(t, 2.f + t), q = s * s;
  float p = 1.f / 15.f;
  p = fmaf(p, q, 1.f / 13.f);
  p = fmaf(p, q, 1.f / 11.f);
  p = fmaf(p, q, 1.f / 9.f);
  p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 1.f / 5.f);
  p = fmaf(p, q, 1.f / 3.f);
  return fmaxf(z, 0.f) + 2.f * s * fmaf(p, q, 1.f);
}
// exp(x), x <= 0: the factor a state is multiplied by at every token, so its error adds up over the tokens that the state
// remembers.  Models in 32-bit take the one that is exact to the last place near 1.
template <typename T>
__device__ __forceinline__ float decay_exp(float x) {
  if constexpr (sizeof(T) == 4) return x > -0.5f ? 1.f + expm1f(x) : __expf(x);
  else return __expf(x);
}
template <int V, typename T>
__device__ __forceinline__ void load_n(const T* p, float (&f)[V]) {
  if constexpr (V == 8) load8(p, f);
  else f[0] = to_f32(*p);
}
template <int V, typename T>
__device__ __forceinline__ void store_n(T* p, const float (&f)[V]) {
  if constexpr (V == 8) store8(p, f);
  else from_f32(p, f[0]);
}

// Sums y[0 .. LPC) over LPC neighbouring lanes (ln: place among them); lane l ends with the sum of y[l].  Halves the number of values with
// every exchange.
template <int LPC>
__device__ __forceinline__ float sum_to_lanes(float (&y)[LPC], int ln) {
#pragma unroll
  for (int o = LPC / 2; o > 0; o >>= 1) {
    const bool up = ln & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? y[i] : y[i + o];
      y[i] = (up ? y[i + o] : y[i]) + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return y[0];
}

// Eight elements as they come from memory, converted when they are used.
template <typename T> struct Vec8;
template <> struct Vec8<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 t = unpack_bf16x2(u[j]);
      f[2 * j] = t.x;
      f[2 * j + 1] = t.y;
    }
  }
};
template <> struct Vec8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = reinterpret_cast<const float4*>(p)[0];
    b = reinterpret_cast<const float4*>(p)[1];
  }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
};

template <typename T, int V> struct Raw : Vec8<T> {};
template <typename T> struct Raw<T, 1> {
  T v;
  __device__ __forceinline__ void load(const T* p) { v = *p; }
  __device__ __forceinline__ void get(float (&f)[1]) const { f[0] = to_f32(v); }
};

// ============================================================================ token shift
template <typename T, int V>
__global__ void __launch_bounds__(256) token_shift_kernel(const T* __restrict__ h, const T* __restrict__ mu, T* __restrict__ last,
                                                          T* __restrict__ out, const int* __restrict__ token_seq, const Seqs q, int rows,
                                                          int W, int n_mix) {
  const int t = blockIdx.x, seq = token_seq[t];
  const size_t plane = size_t(rows) * W;
  if (seq < 0 || seq >= q.n) {                     // padding row
    const float zero[V] = {};
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V)
      for (int j = 0; j < n_mix; ++j) store_n<V>(out + j * plane + size_t(t) * W + c, zero);
    return;
  }
  const int start = q.q_cu[seq], end = q.q_cu[seq + 1];
  const int slot = record_of(q, seq);
  if (slot < 0) return;
  const bool first = t == start, cont = q.kv_lens[seq] > end - start;
  for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
    float cur[V], prev[V] = {}, m[V], o[V];
    load_n<V>(h + size_t(t) * W + c, cur);
    if (!first) load_n<V>(h + size_t(t - 1) * W + c, prev);
    else if (cont) load_n<V>(last + size_t(slot) * W + c, prev);
    for (int j = 0; j < n_mix; ++j) {
      load_n<V>(mu + size_t(j) * W + c, m);
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = fmaf(prev[e] - cur[e], m[e], cur[e]);
      store_n<V>(out + j * plane + size_t(t) * W + c, o);
    }
    if (first) {                                   // only this thread reads this part of the record
      load_n<V>(h + size_t(end - 1) * W + c, cur);
      store_n<V>(last + size_t(slot) * W + c, cur);
    }
  }
}

// ============================================================================ causal convolution (+ silu, + its input)
struct ConvOut { int silu, residual; };          // out = act(convolution) (+ x)
// A thread owns V channels of a tile of consecutive rows and keeps the last TAPS - 1 inputs in registers (TAPS = 0: any
// number of taps, inputs read again for every row).
constexpr int kConvRows = 16, kConvRowsSingle = 2;

template <typename T, int V, int TAPS, int ROWS>
__global__ void __launch_bounds__(128, sizeof(T) == 2 ? 5 : 1) causal_conv_kernel(const T* __restrict__ x, const T* __restrict__ w, const T* __restrict__ bias,
                                                        T* __restrict__ state, T* __restrict__ out, const int* __restrict__ token_seq,
                                                        const Seqs q, int rows, int C, int taps_rt, long ldx, const ConvOut act) {
  constexpr int H = TAPS > 1 ? TAPS - 1 : 1;
  const int taps = TAPS > 0 ? TAPS : taps_rt;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (c >= C) return;
  const int t0 = blockIdx.x * ROWS, t1 = min(rows, t0 + ROWS);
  float b[V], hist[H][V];
  Raw<T, V> wt[TAPS > 0 ? TAPS : 1];
#pragma unroll
  for (int e = 0; e < V; ++e) b[e] = 0.f;
  if (bias) load_n<V>(bias + c, b);
  if (TAPS > 0) {
#pragma unroll
    for (int i = 0; i < TAPS; ++i) wt[i].load(w + size_t(i) * C + c);
  }
  int cur_seq = -1, start = 0, end = 0, slot = 0;
  bool cont = false;
  constexpr int AHEAD = ROWS < 4 ? ROWS : 4;             // rows requested together
  Raw<T, V> ahead[AHEAD];
  int seqs[AHEAD];
#pragma unroll 1
  for (int tg = t0; tg < t1; tg += AHEAD) {
#pragma unroll
    for (int r = 0; r < AHEAD; ++r) {
      seqs[r] = tg + r < t1 ? token_seq[tg + r] : -1;
      if (tg + r < t1) ahead[r].load(x + size_t(tg + r) * ldx + c);
    }
#pragma unroll
    for (int r = 0; r < AHEAD; ++r) {
      const int t = tg + r, seq = seqs[r];
      if (seq < 0 || seq >= q.n) continue;
      const bool fresh = seq != cur_seq;
      if (fresh) {
        cur_seq = seq;
        start = q.q_cu[seq];
        end = q.q_cu[seq + 1];
        slot = record_of(q, seq);
        cont = q.kv_lens[seq] > end - start;
      }
      if (slot < 0) continue;
      // input `back` rows ahead of row t of this sequence
      auto before = [&](int back, float (&f)[V]) {
        const int j = t - start - back;
#pragma unroll
        for (int e = 0; e < V; ++e) f[e] = 0.f;
        if (j >= 0) load_n<V>(x + size_t(t - back) * ldx + c, f);
        else if (cont) load_n<V>(state + (size_t(slot) * (taps - 1) + (taps - 1 + j)) * C + c, f);
      };
      float y[V], cur[V], f[V];
      ahead[r].get(cur);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = b[e];
      if (TAPS > 0) {
        if (fresh) {
#pragma unroll
          for (int i = 0; i < TAPS - 1; ++i) before(TAPS - 1 - i, hist[i]);
        }
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i) {
          wt[i].get(f);
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = fmaf(hist[i][e], f[e], y[e]);
        }
        wt[TAPS > 0 ? TAPS - 1 : 0].get(f);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(cur[e], f[e], y[e]);
#pragma unroll
        for (int i = 0; i + 1 < TAPS - 1; ++i)
#pragma unroll
          for (int e = 0; e < V; ++e) hist[i][e] = hist[i + 1][e];
        if (TAPS > 1) {
#pragma unroll
          for (int e = 0; e < V; ++e) hist[H - 1][e] = cur[e];
          if (end - start == 1) {                    // a single row: this thread alone reads and writes this part of the record
#pragma unroll
            for (int i = 0; i < TAPS - 1; ++i) store_n<V>(state + (size_t(slot) * H + i) * C + c, hist[i]);
          }
        }
      } else {
        for (int i = 0; i < taps; ++i) {
          before(taps - 1 - i, f);
#pragma unroll
          for (int e = 0; e < V; ++e) y[e] = fmaf(f[e], to_f32(w[size_t(i) * C + c + e]), y[e]);
        }
        if (end - start == 1) {
          for (int i = 0; i < taps - 1; ++i) {
            before(taps - 2 - i, f);                 // row i moves down by one, the last becomes the current input
            store_n<V>(state + (size_t(slot) * (taps - 1) + i) * C + c, f);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) {
        if (act.silu) y[e] = act_silu(y[e]);
        if (act.residual) y[e] += cur[e];
      }
      store_n<V>(out + size_t(t) * C + c, y);
    }
  }
}

// Records of the sequences with several rows, after the convolution has read the old ones.
template <typename T, int V>
__global__ void __launch_bounds__(128) conv_record_kernel(const T* __restrict__ x, T* __restrict__ state, const Seqs q, int C, int taps,
                                                          long ldx) {
  const int seq = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  const int start = q.q_cu[seq], len = q.q_cu[seq + 1] - start;
  if (len < 2 || c >= C) return;
  const int slot = record_of(q, seq);
  if (slot < 0) return;
  const bool cont = q.kv_lens[seq] > len;
  T* rec = state + size_t(slot) * (taps - 1) * C + c;
  for (int i = 0; i < taps - 1; ++i) {             // ascending: row i comes from a later row of the record
    const int j = len - (taps - 1) + i;
    float f[V] = {};
    if (j >= 0) load_n<V>(x + size_t(start + j) * ldx + c, f);
    else if (cont) load_n<V>(rec + size_t(i + len) * C, f);
    store_n<V>(rec + size_t(i) * C, f);
  }
}

// ============================================================================ matrix state per head
// S [dk, dv] per head, updated by every token's k v^T behind a decay:
//   MIX_BONUS   time mixing: decay exp(-exp(z + w0)) per key channel; o = S^T r ahead of the update, plus the current token times u
//   MIX_GATED   gated linear attention: decay sigmoid(z + w0)^inv_tau per key channel; o = S^T q behind the update
//   MIX_MEMORY  matrix memory: decay e^f and input factor e^i per head relative to a running maximum m, a normaliser n that is updated
//               like a column of S with value 1; o = S^T q / (max(|n q|, e^-m) + 1e-6) behind the update
// then RMS per head, weight and gate (silu, MIX_MEMORY: sigmoid).
enum { MIX_BONUS = 0, MIX_GATED = 1, MIX_MEMORY = 2 };
constexpr float kMemoryEps = 1e-6f;

template <typename T>
struct MixParams {
  const T *r, *k, *v, *gate;       // [rows, H * dk] (queries, keys), [rows, H * dv], row pitch ld (gate: ldg)
  const float* z;                  // [rows, H * dk] dense; MIX_MEMORY: [rows, 2 H], input gates, then forget gates
  const float *w0, *u;             // [H * dk] (MIX_MEMORY: biases [2 H]); MIX_BONUS
  const T* norm_w;                 // weight of head h at h * norm_step
  float* state;                    // [records, H, dk, dv] (key, value), MIX_MEMORY: n [dk] behind every head's matrix
  T* out;                          // row pitch ldo
  long ld, ldg, ldo;
  int H, dk, dv, norm_step;
  float scale, eps;
  float q_scale, inv_tau, cap;     // MIX_GATED, MIX_MEMORY: factor of q; MIX_GATED; MIX_MEMORY: bound of the gates
  float* top;                      // MIX_MEMORY: [records, H] running maxima
  float* fi;                       // MIX_MEMORY: decays, input factors and e^-m of longer portions, [3, H, rows]
  int rows;
  Seqs q;
  // segments of longer portions
  int L;                           // rows per segment
  float* ws_s;                     // [segments, H, record]: what a segment adds to the state, then the state it starts from
  float* ws_p;                     // [segments, H, dk]: product of its decays
};
template <int KIND, typename T>
__device__ __forceinline__ size_t record_size(const MixParams<T>& p) {
  return size_t(p.dk) * (KIND == MIX_BONUS ? p.dk : p.dv) + (KIND == MIX_MEMORY ? p.dk : 0);
}
template <int KIND, typename T>
__device__ __forceinline__ float decay_of(const MixParams<T>& p, float z) {
  if constexpr (KIND == MIX_BONUS) return decay_exp<T>(-__expf(z));
  else return decay_exp<T>(-softplus(-z) * p.inv_tau);
}
template <int KIND>
__device__ __forceinline__ float out_gate(float g) {
  if constexpr (KIND == MIX_MEMORY) return 1.f / (1.f + __expf(-g));
  else return act_silu(g);
}
// log input and log forget gate of a head
template <typename T>
__device__ __forceinline__ float2 log_gates(const MixParams<T>& p, size_t t, int h) {
  const float* z = p.z + t * (2 * p.H);
  return make_float2(act_softcap(z[h] + p.w0[h], p.cap), -softplus(-act_softcap(z[p.H + h] + p.w0[p.H + h], p.cap)));
}

// MIX_MEMORY, portions of min_len and more rows: m <- max(log f + m, log i) over a sequence, one warp per (sequence, head).  A lane
// composes the steps of kGateRows neighbouring tokens, the lanes' compositions are scanned.
constexpr int kGateRows = 8;
template <typename T>
__global__ void __launch_bounds__(128) memory_gates_kernel(const MixParams<T> p, int min_len) {
  const int seq = blockIdx.x, h = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int start = p.q.q_cu[seq], len = p.q.q_cu[seq + 1] - start;
  if (len < min_len || len < 1 || h >= p.H) return;
  const int slot = p.q.slots[seq];
  if (slot < 0 || slot >= p.q.n_slots) return;             // recorded by the kernels that follow
  float carry = p.q.kv_lens[seq] > len ? p.top[size_t(slot) * p.H + h] : 0.f;
  const size_t plane = size_t(p.H) * p.rows;
  for (int b = 0; b < len; b += 32 * kGateRows) {
    float li[kGateRows], lf[kGateRows], F = 0.f, I = -INFINITY;
#pragma unroll
    for (int e = 0; e < kGateRows; ++e) {
      const int t = b + lane * kGateRows + e;
      const float2 g = t < len ? log_gates(p, size_t(start + t), h) : make_float2(-INFINITY, 0.f);
      li[e] = g.x;
      lf[e] = g.y;
      I = fmaxf(g.y + I, g.x);
      F += g.y;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pf = __shfl_up_sync(0xffffffffu, F, o), pi = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(F + pi, I);
        F += pf;
      }
    }
    float before = __shfl_up_sync(0xffffffffu, fmaxf(F + carry, I), 1);
    if (lane == 0) before = carry;
    float m[kGateRows];
#pragma unroll
    for (int e = 0; e < kGateRows; ++e) m[e] = fmaxf(lf[e] + (e > 0 ? m[e > 0 ? e - 1 : 0] : before), li[e]);
    before = __shfl_up_sync(0xffffffffu, m[kGateRows - 1], 1);        // what the lane ahead of this one arrived at
    if (lane == 0) before = carry;
#pragma unroll
    for (int e = 0; e < kGateRows; ++e) {
      const int t = b + lane * kGateRows + e;
      if (t < len) {
        float* dst = p.fi + size_t(h) * p.rows + start + t;
        dst[0] = decay_exp<T>(fminf(lf[e] + (e > 0 ? m[e > 0 ? e - 1 : 0] : before) - m[e], 0.f));
        dst[plane] = __expf(li[e] - m[e]);
        dst[2 * plane] = __expf(-m[e]);
      }
    }
    carry = __shfl_sync(0xffffffffu, m[kGateRows - 1], 31);
  }
  if (lane == 0) p.top[size_t(slot) * p.H + h] = carry;
}

// Portions of two and more rows are cut into segments of L rows, numbered through the batch.  Every warp finds segment
// `target`: its sequence, its place there and how many the sequence has.
__device__ __forceinline__ bool find_segment(const Seqs& q, int L, int target, int& seq, int& seg, int& n_seg) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int b = 0; b < q.n; b += 32) {
    const int s = b + lane;
    const int len = s < q.n ? q.q_cu[s + 1] - q.q_cu[s] : 0;
    const int cnt = len > 1 ? (len + L - 1) / L : 0;
    int inc = cnt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    const int total = __shfl_sync(0xffffffffu, inc, 31);
    if (target < base + total) {
      const int f = __ffs(__ballot_sync(0xffffffffu, base + inc > target)) - 1;
      n_seg = __shfl_sync(0xffffffffu, cnt, f);
      seg = target - (base + __shfl_sync(0xffffffffu, inc, f) - n_seg);
      seq = b + f;
      return true;
    }
    base += total;
  }
  return false;
}

// One (segment, head) per CTA.  DK, DV: key and value size of a head padded to 32, 64 or 128.  Thread (kg, vg) owns keys kg * KT ...,
// values vg * VT ... of the head's matrix, as pairs of neighbouring keys: the more of both, the fewer reads of shared memory per
// element, which bound this kernel beside the multiply-adds.
template <int DK, int DV> struct MixCfg {
  static constexpr int KT = DK == 32 ? 4 : 8, VT = 8;
  static constexpr int KG = DK / KT, VG = DV / VT, kThreads = KG * VG;
  static constexpr int kMinBlocks = kThreads > 128 ? 1 : kThreads > 64 ? 2 : kThreads > 32 ? 5 : DK == 32 ? 12 : 8;
  // Place of key c in a row of shared memory.  Eight key groups are read at a time, four keys of each: with eight keys per
  // group every other four groups have their halves swapped, so that the reads meet no bank twice.
  __device__ static constexpr int key_at(int c) { return KT == 4 ? c : c ^ (((c >> 5) & 1) << 2); }
};
// Eight keys from c (a multiple of 8) on.
template <int DK>
__device__ __forceinline__ void store_keys(float* row, int c, const float (&f)[8]) {
  *reinterpret_cast<float4*>(row + MixCfg<DK, 32>::key_at(c)) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(row + MixCfg<DK, 32>::key_at(c + 4)) = make_float4(f[4], f[5], f[6], f[7]);
}
template <int DK>
__device__ __forceinline__ void load_keys(const float* row, int c, float (&f)[8]) {
  *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(row + MixCfg<DK, 32>::key_at(c));
  *reinterpret_cast<float4*>(f + 4) = *reinterpret_cast<const float4*>(row + MixCfg<DK, 32>::key_at(c + 4));
}
constexpr int kMixRows = 16;      // rows staged in shared memory at a time

// v8, g8: 8-element accesses to the inputs / to gate and output are aligned; s4: rows of the state are multiples of 16 bytes
template <typename T, int DK, int DV, int KIND, bool OUT>
__global__ void __launch_bounds__(MixCfg<DK, DV>::kThreads, sizeof(T) == 2 ? MixCfg<DK, DV>::kMinBlocks : 1)
matrix_segment_kernel(const MixParams<T> p, int v8, int g8, int s4) {
  using C = MixCfg<DK, DV>;
  constexpr int KT = C::KT, VT = C::VT, KG = C::KG, NT = C::kThreads;
  constexpr bool BONUS = KIND == MIX_BONUS, MEMORY = KIND == MIX_MEMORY;
  __shared__ __align__(16) float sK[kMixRows][DK], sW[kMixRows][DK], sV[kMixRows][DV];
  __shared__ __align__(16) float sR[OUT ? kMixRows : 1][DK], sO[OUT ? kMixRows : 1][DV];
  __shared__ __align__(16) float sNw[OUT ? DV : 1], sU[OUT && BONUS ? DK : 1];
  __shared__ float sRow[kMixRows];                        // MIX_BONUS: product with the current token; MIX_MEMORY: n q
  __shared__ float sLeast[MEMORY ? kMixRows : 1];         // e^-m
  int seq, seg, n_seg;
  if (!find_segment(p.q, p.L, blockIdx.x, seq, seg, n_seg)) return;
  if (!OUT && seg == n_seg - 1) return;                   // nothing starts behind the last segment
  if (n_seg > 1 && !p.ws_s) {                             // a portion longer than the caller said
    if (threadIdx.x == 0) atomicExch(p.q.status, XL_ERR_BOUNDS);
    return;
  }
  const int slot = record_of(p.q, seq);
  if (slot < 0) return;
  const int h = blockIdx.y, dk = p.dk, dv = BONUS ? dk : p.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int kg = tid % KG, vg = tid / KG;
  const int start = p.q.q_cu[seq], len = p.q.q_cu[seq + 1] - start;
  const int t0 = start + seg * p.L, n = min(p.L, len - seg * p.L);
  const bool cont = p.q.kv_lens[seq] > len;
  const size_t mat = record_size<KIND>(p);
  float* rec = p.state + (size_t(slot) * p.H + h) * mat;
  float* seg_s = p.ws_s ? p.ws_s + (size_t(blockIdx.x) * p.H + h) * mat : nullptr;

  uint64_t S[KT / 2][VT], N[MEMORY ? KT / 2 : 1];
#pragma unroll
  for (int i = 0; i < KT / 2; ++i)
#pragma unroll
    for (int j = 0; j < VT; ++j) S[i][j] = 0;
#pragma unroll
  for (int i = 0; i < (MEMORY ? KT / 2 : 1); ++i) N[i] = 0;
  if (OUT && (n_seg > 1 || cont)) {
    const float* src = n_seg > 1 ? seg_s : rec;
#pragma unroll
    for (int i = 0; i < KT / 2; ++i) {
      float a[2][VT] = {};
      float nn[2] = {};
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = kg * KT + 2 * i + e;
        if (key < dk) {
          if (MEMORY) nn[e] = src[size_t(dk) * dv + key];
          const float* row = src + size_t(key) * dv + vg * VT;
#pragma unroll
          for (int j = 0; j < VT; j += 4) {
            if (s4) {
              if (vg * VT + j < dv) *reinterpret_cast<float4*>(a[e] + j) = *reinterpret_cast<const float4*>(row + j);
            } else {
#pragma unroll
              for (int l = j; l < j + 4; ++l)
                if (vg * VT + l < dv) a[e][l] = row[l];
            }
          }
        }
      }
      if (MEMORY) N[MEMORY ? i : 0] = pack2(nn[0], nn[1]);
#pragma unroll
      for (int j = 0; j < VT; ++j) S[i][j] = pack2(a[0][j], a[1][j]);
    }
  }
  constexpr int PR = (DK + NT - 1) / NT;
  float prod[PR];                                         // !OUT: decay of keys `tid`, `tid` + NT ... over the segment
#pragma unroll
  for (int i = 0; i < PR; ++i) prod[i] = 1.f;
  // Rows are finished (and their bonus is prepared) by vectors of 8 columns: LR lanes per row, RP rows per warp and pass.
  constexpr int LR = DV / 8, RP = 32 / LR, PASSES = kMixRows / (NT / 32 * RP);
  static_assert(PASSES >= 1 && (!BONUS || DK == DV), "rows per pass; the bonus takes keys and values of one size");
  const int fr_row = warp * RP + lane / LR, fr_c = lane % LR * 8;
  if (OUT) {                                              // visible behind the first tile's barrier
    for (int c = tid; c < DV; c += NT) sNw[OUT ? c : 0] = c < dv ? to_f32(p.norm_w[h * p.norm_step + c]) * p.scale : 0.f;
    if (BONUS)
      for (int c = tid; c < DK; c += NT) sU[OUT && BONUS ? c : 0] = c < dk ? p.u[h * dk + c] : 0.f;
  }
  // rows of this head on their way: vector i * NT + tid of the [row][8 columns] tiles (v8 only)
  constexpr int EK = kMixRows * (DK / 8), EV = kMixRows * (DV / 8);
  constexpr int NK = (EK + NT - 1) / NT, NV = (EV + NT - 1) / NT;
  Vec8<T> fk[NK], fv[NV], fr[OUT ? NK : 1];
  Vec8<float> fz[MEMORY ? 1 : NK];
  float2 ffi[MEMORY ? NK : 1];
  const size_t plane = size_t(p.H) * p.rows;
  auto fetch = [&](int b) {
    const int m = min(kMixRows, n - b);
#pragma unroll
    for (int i = 0; i < NK; ++i) {
      const int e = i * NT + tid, row = e / (DK / 8), c = e % (DK / 8) * 8;
      if (row < m && c < dk) {
        const size_t t = size_t(t0 + b + row), at = t * p.ld + size_t(h) * dk + c;
        fk[i].load(p.k + at);
        if (OUT) fr[OUT ? i : 0].load(p.r + at);
        if constexpr (MEMORY) {
          const float* g = p.fi + size_t(h) * p.rows + t;
          ffi[i] = make_float2(g[0], g[plane]);
        } else {
          fz[i].load(p.z + t * (size_t(p.H) * dk) + size_t(h) * dk + c);
        }
        if (BONUS) fv[BONUS ? i : 0].load(p.v + at);        // keys and values are of one size
      }
    }
#pragma unroll
    for (int i = 0; i < (BONUS ? 0 : NV); ++i) {
      const int e = i * NT + tid, row = e / (DV / 8), c = e % (DV / 8) * 8;
      if (row < m && c < dv) fv[i].load(p.v + size_t(t0 + b + row) * p.ld + size_t(h) * dv + c);
    }
  };
  if (v8) fetch(0);
  for (int b = 0; b < n; b += kMixRows) {
    const int m = min(kMixRows, n - b);
    // stage the rows; those beyond m leave the state as it is (decay 1, key 0)
    if (MEMORY && OUT && tid < kMixRows) sLeast[MEMORY ? tid : 0] = tid < m ? p.fi[2 * plane + size_t(h) * p.rows + t0 + b + tid] : 1.f;
    if (v8) {
#pragma unroll
      for (int i = 0; i < NK; ++i) {
        const int e = i * NT + tid, row = e / (DK / 8), c = e % (DK / 8) * 8;
        if (EK % NT && e >= EK) break;
        float k[8] = {}, r[8] = {}, w[8], vv[8] = {};
#pragma unroll
        for (int j = 0; j < 8; ++j) w[j] = 1.f;
        if (row < m && c < dk) {
          fk[i].get(k);
          if (BONUS) fv[BONUS ? i : 0].get(vv);
          if (OUT) fr[OUT ? i : 0].get(r);
          if constexpr (MEMORY) {
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              w[j] = ffi[i].x;
              k[j] *= ffi[i].y;
            }
          } else {
            float w0[8];
            fz[i].get(w);
            load8(p.w0 + h * dk + c, w0);
#pragma unroll
            for (int j = 0; j < 8; ++j) w[j] = decay_of<KIND>(p, w[j] + w0[j]);
          }
          if (!BONUS) {
#pragma unroll
            for (int j = 0; j < 8; ++j) r[j] *= p.q_scale;
          }
        }
        store_keys<DK>(sK[row], c, k);
        store_keys<DK>(sW[row], c, w);
        if (BONUS) store8(&sV[BONUS ? row : 0][BONUS ? c : 0], vv);
        if (OUT) store_keys<DK>(sR[row], c, r);
      }
#pragma unroll
      for (int i = 0; i < (BONUS ? 0 : NV); ++i) {
        const int e = i * NT + tid, row = e / (DV / 8), c = e % (DV / 8) * 8;
        if (EV % NT && e >= EV) break;
        float v[8] = {};
        if (row < m && c < dv) fv[i].get(v);
        store8(&sV[row][c], v);
      }
    } else {
      for (int i = tid; i < kMixRows * DK; i += NT) {
        const int row = i / DK, c = i % DK;
        const bool in = row < m && c < dk;
        const size_t t = size_t(t0 + b + row), at = t * p.ld + size_t(h) * dk + c;
        const int to = C::key_at(c);
        float k = in ? to_f32(p.k[at]) : 0.f, w = 1.f;
        if (in) {
          if constexpr (MEMORY) {
            const float* g = p.fi + size_t(h) * p.rows + t;
            w = g[0];
            k *= g[plane];
          } else {
            w = decay_of<KIND>(p, p.z[t * (size_t(p.H) * dk) + size_t(h) * dk + c] + p.w0[h * dk + c]);
          }
        }
        sK[row][to] = k;
        sW[row][to] = w;
        if (OUT) sR[row][to] = in ? to_f32(p.r[at]) * (BONUS ? 1.f : p.q_scale) : 0.f;
      }
      for (int i = tid; i < kMixRows * DV; i += NT) {
        const int row = i / DV, c = i % DV;
        sV[row][c] = row < m && c < dv ? to_f32(p.v[size_t(t0 + b + row) * p.ld + size_t(h) * dv + c]) : 0.f;
      }
    }
    __syncthreads();
    if (v8 && b + kMixRows < n) fetch(b + kMixRows);
    Vec8<T> gate[OUT ? PASSES : 1];
    if (OUT) {
#pragma unroll
      for (int q = 0; q < PASSES; ++q) {
        const int row = q * (NT / 32 * RP) + fr_row;
        float s = 0.f;
        if (row < m) {
          if (g8 && fr_c < dv) gate[OUT ? q : 0].load(p.gate + size_t(t0 + b + row) * p.ldg + size_t(h) * dv + fr_c);
          if constexpr (BONUS) {
            float r[8], k[8], u[8];
            load_keys<DK>(sR[row], fr_c, r);
            load_keys<DK>(sK[row], fr_c, k);
            load8(&sU[fr_c], u);
#pragma unroll
            for (int j = 0; j < 8; ++j) s = fmaf(r[j] * u[j], k[j], s);
          }
        }
        if constexpr (BONUS) {
#pragma unroll
          for (int o = LR / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
          if (lane % LR == 0 && row < m) sRow[row] = s;    // read behind the next barrier
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < PR; ++i) {
        const int c = i * NT + tid;
        if (DK % NT == 0 || c < DK) {
#pragma unroll
          for (int row = 0; row < kMixRows; ++row) prod[i] *= sW[row][C::key_at(c)];
        }
      }
    }
#pragma unroll 1
    for (int row = 0; row < kMixRows; ++row) {
      float vf[8];
      load8(&sV[row][vg * VT], vf);
      uint64_t v[VT], o[VT], den = 0;
#pragma unroll
      for (int j = 0; j < VT; ++j) {
        v[j] = pack2(vf[j], vf[j]);
        o[j] = 0;
      }
#pragma unroll
      for (int i = 0; i < KT / 4; ++i) {
        const int at = C::key_at(kg * KT + 4 * i);
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(&sK[row][at]);
        const ulonglong2 w2 = *reinterpret_cast<const ulonglong2*>(&sW[row][at]);
        ulonglong2 r2 = {0, 0};
        if (OUT) r2 = *reinterpret_cast<const ulonglong2*>(&sR[row][at]);
        if (OUT && BONUS) {
#pragma unroll
          for (int j = 0; j < VT; ++j) o[j] = fma2(r2.y, S[2 * i + 1][j], fma2(r2.x, S[2 * i][j], o[j]));
        }
#pragma unroll
        for (int j = 0; j < VT; ++j) {
          S[2 * i][j] = fma2(w2.x, S[2 * i][j], mul2(k2.x, v[j]));
          S[2 * i + 1][j] = fma2(w2.y, S[2 * i + 1][j], mul2(k2.y, v[j]));
        }
        if (MEMORY) {
          N[MEMORY ? 2 * i : 0] = fma2(w2.x, N[MEMORY ? 2 * i : 0], k2.x);
          N[MEMORY ? 2 * i + 1 : 0] = fma2(w2.y, N[MEMORY ? 2 * i + 1 : 0], k2.y);
          if (OUT) den = fma2(r2.y, N[MEMORY ? 2 * i + 1 : 0], fma2(r2.x, N[MEMORY ? 2 * i : 0], den));
        }
        if (OUT && !BONUS) {
#pragma unroll
          for (int j = 0; j < VT; ++j) o[j] = fma2(r2.y, S[2 * i + 1][j], fma2(r2.x, S[2 * i][j], o[j]));
        }
      }
      if (OUT) {
        // sum over the key groups (neighbouring lanes); each of the first eight ends with one of the eight values
        float y[VT];
#pragma unroll
        for (int j = 0; j < VT; ++j) {
          const float2 f = unpack2(o[j]);
          y[j] = f.x + f.y;
        }
        float a = sum_to_lanes<VT>(y, kg);
        if (KG == 16) a += __shfl_xor_sync(0xffffffffu, a, 8);
        if (KG == 8 || kg < 8) sO[row][vg * VT + kg] = a;
        if (MEMORY) {
          const float2 f = unpack2(den);
          float d = f.x + f.y;
#pragma unroll
          for (int w = KG / 2; w > 0; w >>= 1) d += __shfl_xor_sync(0xffffffffu, d, w);
          if (tid == 0) sRow[row] = d;
        }
      }
    }
    __syncthreads();
    if (OUT) {
#pragma unroll
      for (int q = 0; q < PASSES; ++q) {
        const int row = q * (NT / 32 * RP) + fr_row;
        float o[8], ss = 0.f, f = 0.f;                     // f: factor of the current token, or of the whole row
        if (BONUS && row < m) f = sRow[row];
        if (MEMORY && row < m) f = 1.f / (fmaxf(fabsf(sRow[row]), sLeast[MEMORY ? row : 0]) + kMemoryEps);
        load8(&sO[row][fr_c], o);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          if (BONUS) o[j] = fmaf(f, sV[row][fr_c + j], o[j]);     // zero beyond dv
          if (MEMORY) o[j] *= f;
          ss = fmaf(o[j], o[j], ss);
        }
#pragma unroll
        for (int w = LR / 2; w > 0; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
        const float inv = rsqrtf(ss / float(dv) + p.eps);
        if (row < m) {
          const size_t t = size_t(t0 + b + row);
          T* out = p.out + t * p.ldo + size_t(h) * dv + fr_c;
          float nw[8], g[8];
          load8(&sNw[fr_c], nw);
          if (g8) {
            gate[OUT ? q : 0].get(g);
#pragma unroll
            for (int j = 0; j < 8; ++j) o[j] = o[j] * inv * nw[j] * out_gate<KIND>(g[j]);
            if (fr_c < dv) store8(out, o);
          } else {
#pragma unroll
            for (int j = 0; j < 8; ++j)
              if (fr_c + j < dv)
                from_f32(out + j, o[j] * inv * nw[j] * out_gate<KIND>(to_f32(p.gate[t * p.ldg + size_t(h) * dv + fr_c + j])));
          }
        }
      }
      __syncthreads();
    }
  }
  if (OUT && seg != n_seg - 1) return;
  float* dst = OUT ? rec : seg_s;
#pragma unroll
  for (int i = 0; i < KT / 2; ++i) {
    float a[2][VT];
#pragma unroll
    for (int j = 0; j < VT; ++j) {
      const float2 f = unpack2(S[i][j]);
      a[0][j] = f.x;
      a[1][j] = f.y;
    }
    const float2 nn = unpack2(N[MEMORY ? i : 0]);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int key = kg * KT + 2 * i + e;
      if (key >= dk) continue;
      if (MEMORY && vg == 0) dst[size_t(dk) * dv + key] = e ? nn.y : nn.x;
      float* row = dst + size_t(key) * dv + vg * VT;
#pragma unroll
      for (int j = 0; j < VT; j += 4) {
        if (s4) {
          if (vg * VT + j < dv) *reinterpret_cast<float4*>(row + j) = *reinterpret_cast<const float4*>(a[e] + j);
        } else {
#pragma unroll
          for (int l = j; l < j + 4; ++l)
            if (vg * VT + l < dv) row[l] = a[e][l];
        }
      }
    }
  }
  if (!OUT) {
#pragma unroll
    for (int i = 0; i < PR; ++i) {
      const int c = i * NT + tid;
      if (c < dk) p.ws_p[(size_t(blockIdx.x) * p.H + h) * dk + c] = prod[i];
    }
  }
}

// (B): the state every segment starts from, in the place of what it adds.  One CTA per (sequence, head, part of the record).
template <typename T, int KIND>
__global__ void __launch_bounds__(256) matrix_chain_kernel(const MixParams<T> p) {
  const int seq = blockIdx.x, h = blockIdx.y, dk = p.dk;
  const int len = p.q.q_cu[seq + 1] - p.q.q_cu[seq];
  const int n_seg = len > 1 ? (len + p.L - 1) / p.L : 0;
  if (n_seg < 2) return;
  const int slot = record_of(p.q, seq);
  if (slot < 0) return;
  int base = 0;                                           // segments of the sequences ahead of this one
  {
    const int lane = threadIdx.x & 31;
    for (int s = lane; s < seq; s += 32) {
      const int n = p.q.q_cu[s + 1] - p.q.q_cu[s];
      base += n > 1 ? (n + p.L - 1) / p.L : 0;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) base += __shfl_xor_sync(0xffffffffu, base, o);
  }
  const bool cont = p.q.kv_lens[seq] > len;
  const int mat = int(record_size<KIND>(p)), cells = dk * p.dv;
  const float* rec = p.state + (size_t(slot) * p.H + h) * mat;
  const size_t step = size_t(p.H) * mat;
  for (int e = blockIdx.z * blockDim.x + threadIdx.x; e < mat; e += gridDim.z * blockDim.x) {
    float s = cont ? rec[e] : 0.f;
    float* ws = p.ws_s + (size_t(base) * p.H + h) * mat + e;
    const float* pr = p.ws_p + (size_t(base) * p.H + h) * dk + (KIND == MIX_MEMORY && e >= cells ? e - cells : e / p.dv);
    constexpr int kGroup = 8;
    const size_t pstep = size_t(p.H) * dk;
    for (int g = 0; g < n_seg; g += kGroup) {              // the last segment only takes its start
      float add[kGroup], f[kGroup];
#pragma unroll
      for (int i = 0; i < kGroup; ++i)
        if (g + i < n_seg - 1) {
          add[i] = ws[i * step];
          f[i] = pr[i * pstep];
        }
#pragma unroll
      for (int i = 0; i < kGroup; ++i)
        if (g + i < n_seg) {
          ws[i * step] = s;
          if (g + i < n_seg - 1) s = fmaf(f[i], s, add[i]);
        }
      ws += kGroup * step;
      pr += kGroup * pstep;
    }
  }
}

// Factors of one token of a matrix memory whose state comes from the records.
struct TokenGates { float f, i, least, m; };
template <typename T>
__device__ __forceinline__ TokenGates token_gates(const MixParams<T>& p, size_t t, int h, float m) {
  const float2 g = log_gates(p, t, h);
  const float m_new = fmaxf(g.y + m, g.x);
  return {decay_exp<T>(g.y + m - m_new), __expf(g.x - m_new), __expf(-m_new), m_new};
}

// Single rows: the head's matrix (dv a multiple of 4) passes through registers once.
constexpr int kMixThreads = 128;
template <typename T, int KIND>
__global__ void __launch_bounds__(kMixThreads) matrix_single_kernel(const MixParams<T> p) {
  constexpr bool BONUS = KIND == MIX_BONUS, MEMORY = KIND == MIX_MEMORY;
  extern __shared__ __align__(16) float sm[];
  const int seq = blockIdx.x, h = blockIdx.y, dk = p.dk, dv = BONUS ? dk : p.dv, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t = p.q.q_cu[seq], len = p.q.q_cu[seq + 1] - t;
  if (len != 1) return;
  const int slot = record_of(p.q, seq);
  if (slot < 0) return;
  const bool cont = p.q.kv_lens[seq] > 1;
  const int quads = dv / 4, groups = kMixThreads / quads;   // threads over value quads, then over keys
  const int vq = tid % quads, kq = tid / quads;
  float *sV = sm, *sO = sV + dv, *sR = sO + groups * dv, *sK = sR + dk, *sW = sK + dk;      // sO [groups][dv]
  __shared__ float red[2][kMixThreads / 32];
  const size_t mat = record_size<KIND>(p);
  float* rec0 = p.state + (size_t(slot) * p.H + h) * mat;
  float4* rec = reinterpret_cast<float4*>(rec0);
  constexpr int kAhead = 8;
  float4 s[kAhead];
  const bool mine = kq < groups;
  if (mine && cont) {                                       // the first keys are on their way while the row is prepared
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (kq + i * groups < dk) s[i] = rec[size_t(kq + i * groups) * quads + vq];
  }
  constexpr int kCols = 4;                                  // columns per thread: dv <= 4 * kMixThreads
  T vals[kCols], gates[kCols];
#pragma unroll
  for (int i = 0; i < kCols; ++i) {
    const int c = i * kMixThreads + tid;
    if (c < dv) {
      vals[i] = p.v[size_t(t) * p.ld + size_t(h) * dv + c];
      gates[i] = p.gate[size_t(t) * p.ldg + size_t(h) * dv + c];
    }
  }
  TokenGates g = {};
  if (MEMORY) g = token_gates(p, t, h, cont ? p.top[size_t(slot) * p.H + h] : 0.f);
  float dot = 0.f;                                          // MIX_BONUS: product with the current token; MIX_MEMORY: n q
  for (int c = tid; c < dk; c += kMixThreads) {
    const size_t at = size_t(t) * p.ld + size_t(h) * dk + c;
    float r = to_f32(p.r[at]), k = to_f32(p.k[at]);
    if (MEMORY) {
      k *= g.i;
      r *= p.q_scale;
      const float nn = fmaf(g.f, cont ? rec0[size_t(dk) * dv + c] : 0.f, k);
      rec0[size_t(dk) * dv + c] = nn;
      dot = fmaf(nn, r, dot);
      sW[c] = g.f;
    } else {
      sW[c] = decay_of<KIND>(p, p.z[size_t(t) * p.H * dk + size_t(h) * dk + c] + p.w0[h * dk + c]);
      if (BONUS) dot += r * p.u[h * dk + c] * k;
      else r *= p.q_scale;
    }
    sR[c] = r;
    sK[c] = k;
  }
#pragma unroll
  for (int i = 0; i < kCols; ++i)
    if (i * kMixThreads + tid < dv) sV[i * kMixThreads + tid] = to_f32(vals[i]);
  dot = warp_sum(dot);
  if (lane == 0) red[0][warp] = dot;
  __syncthreads();
  dot = 0.f;
#pragma unroll
  for (int i = 0; i < kMixThreads / 32; ++i) dot += red[0][i];
  if (MEMORY && tid == 0) p.top[size_t(slot) * p.H + h] = g.m;      // every thread has read the old one
  if (mine) {
    const float4 v = *reinterpret_cast<const float4*>(sV + vq * 4);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k0 = kq; k0 < dk; k0 += kAhead * groups) {
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        const int key = k0 + i * groups;
        if (key < dk) {
          if (!cont) s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
          else if (k0 != kq) s[i] = rec[size_t(key) * quads + vq];
        }
      }
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        const int key = k0 + i * groups;
        if (key < dk) {
          const float r = sR[key], k = sK[key], w = sW[key];
          const float4 a = make_float4(fmaf(w, s[i].x, k * v.x), fmaf(w, s[i].y, k * v.y), fmaf(w, s[i].z, k * v.z), fmaf(w, s[i].w, k * v.w));
          const float4 c = BONUS ? s[i] : a;
          o.x = fmaf(r, c.x, o.x); o.y = fmaf(r, c.y, o.y); o.z = fmaf(r, c.z, o.z); o.w = fmaf(r, c.w, o.w);
          rec[size_t(key) * quads + vq] = a;
        }
      }
    }
    *reinterpret_cast<float4*>(sO + kq * dv + vq * 4) = o;
  }
  __syncthreads();
  const float whole = MEMORY ? 1.f / (fmaxf(fabsf(dot), g.least) + kMemoryEps) : 1.f;
  float ss = 0.f;
  for (int c = tid; c < dv; c += kMixThreads) {
    float o = BONUS ? dot * sV[c] : 0.f;
    for (int i = 0; i < groups; ++i) o += sO[i * dv + c];
    if (MEMORY) o *= whole;
    sO[c] = o;                                              // only this thread reads or writes column c from here on
    ss += o * o;
  }
  ss = warp_sum(ss);
  if (lane == 0) red[1][warp] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < kMixThreads / 32; ++i) ss += red[1][i];
  const float inv = rsqrtf(ss / float(dv) + p.eps) * p.scale;
#pragma unroll
  for (int i = 0; i < kCols; ++i) {
    const int c = i * kMixThreads + tid;
    if (c < dv)
      from_f32(p.out + size_t(t) * p.ldo + size_t(h) * dv + c,
               sO[c] * inv * to_f32(p.norm_w[h * p.norm_step + c]) * out_gate<KIND>(to_f32(gates[i])));
  }
}

// Any head sizes, any number of rows: the state stays in memory, one thread per value column.
template <typename T, int KIND>
__global__ void __launch_bounds__(256) matrix_any_kernel(const MixParams<T> p, int min_len, int max_len) {
  constexpr bool BONUS = KIND == MIX_BONUS, MEMORY = KIND == MIX_MEMORY;
  extern __shared__ __align__(16) float sm[];
  const int seq = blockIdx.x, h = blockIdx.y, dk = p.dk, dv = p.dv, tid = threadIdx.x;
  const int start = p.q.q_cu[seq], len = p.q.q_cu[seq + 1] - start;
  if (len < min_len || len > max_len || len < 1) return;
  const int slot = record_of(p.q, seq);
  if (slot < 0) return;
  bool fresh = p.q.kv_lens[seq] == len;
  float *sR = sm, *sK = sR + dk, *sW = sK + dk, *sO = sW + dk;
  __shared__ float red[2][8];
  float* rec = p.state + (size_t(slot) * p.H + h) * record_size<KIND>(p);
  const size_t plane = size_t(p.H) * p.rows;
  for (int t = start; t < start + len; ++t) {
    const float* fi = MEMORY ? p.fi + size_t(h) * p.rows + t : nullptr;
    float dot = 0.f;
    for (int c = tid; c < dk; c += 256) {
      const size_t at = size_t(t) * p.ld + size_t(h) * dk + c;
      float r = to_f32(p.r[at]), k = to_f32(p.k[at]);
      if (MEMORY) {
        k *= fi[plane];
        r *= p.q_scale;
        float* nn = rec + size_t(dk) * dv + c;
        *nn = fmaf(fi[0], fresh ? 0.f : *nn, k);
        dot = fmaf(*nn, r, dot);
        sW[c] = fi[0];
      } else {
        sW[c] = decay_of<KIND>(p, p.z[size_t(t) * p.H * dk + size_t(h) * dk + c] + p.w0[h * dk + c]);
        if (BONUS) dot += r * p.u[h * dk + c] * k;
        else r *= p.q_scale;
      }
      sR[c] = r;
      sK[c] = k;
    }
    dot = warp_sum(dot);
    if ((tid & 31) == 0) red[0][tid >> 5] = dot;
    __syncthreads();
    dot = 0.f;
    for (int i = 0; i < 8; ++i) dot += red[0][i];
    const float whole = MEMORY ? 1.f / (fmaxf(fabsf(dot), fi[2 * plane]) + kMemoryEps) : 1.f;
    float ss = 0.f;
    for (int c = tid; c < dv; c += 256) {
      const float v = to_f32(p.v[size_t(t) * p.ld + size_t(h) * dv + c]);
      float o = BONUS ? dot * v : 0.f;
      for (int k = 0; k < dk; ++k) {
        const float s = fresh ? 0.f : rec[size_t(k) * dv + c], a = fmaf(sW[k], s, sK[k] * v);
        o = fmaf(sR[k], BONUS ? s : a, o);
        rec[size_t(k) * dv + c] = a;
      }
      if (MEMORY) o *= whole;
      sO[c] = o;
      ss += o * o;
    }
    ss = warp_sum(ss);
    if ((tid & 31) == 0) red[1][tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < 8; ++i) ss += red[1][i];
    const float inv = rsqrtf(ss / float(dv) + p.eps) * p.scale;
    for (int c = tid; c < dv; c += 256)
      from_f32(p.out + size_t(t) * p.ldo + size_t(h) * dv + c,
               sO[c] * inv * to_f32(p.norm_w[h * p.norm_step + c]) * out_gate<KIND>(to_f32(p.gate[size_t(t) * p.ldg + size_t(h) * dv + c])));
    fresh = false;
  }
}

template <typename T, int KIND, int DK, int DV>
static int launch_segments(const MixParams<T>& p, int seg_cap, int v8, int g8, int s4, cudaStream_t st) {
  using C = MixCfg<DK, DV>;
  const dim3 grid(seg_cap, p.H);
  if (p.ws_s) {
    matrix_segment_kernel<T, DK, DV, KIND, false><<<grid, C::kThreads, 0, st>>>(p, v8, g8, s4);
    const int parts = (p.dk * p.dv + 255) / 256;
    matrix_chain_kernel<T, KIND><<<dim3(p.q.n, p.H, parts), 256, 0, st>>>(p);
  }
  matrix_segment_kernel<T, DK, DV, KIND, true><<<grid, C::kThreads, 0, st>>>(p, v8, g8, s4);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

template <typename T, int KIND>
static int launch_matrix(MixParams<T> p, int seg_cap, int has_long, int has_single, cudaStream_t st) {
  const int dk = p.dk, dv = p.dv;
  const bool v8 = dk % 8 == 0 && dv % 8 == 0 && p.ld % 8 == 0 &&
                  !((reinterpret_cast<uintptr_t>(p.r) | reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.v) |
                     reinterpret_cast<uintptr_t>(p.z) | reinterpret_cast<uintptr_t>(p.w0)) & 15);
  const bool g8 = dv % 8 == 0 && p.ldg % 8 == 0 && p.ldo % 8 == 0 &&
                  !((reinterpret_cast<uintptr_t>(p.gate) | reinterpret_cast<uintptr_t>(p.out)) & 15);
  const bool s4 = dv % 4 == 0 && (KIND != MIX_MEMORY || dk % 4 == 0);
  const bool regs = dv % 4 == 0 && dv <= 4 * kMixThreads && s4;       // single rows through registers
  const bool tiles = dk <= 128 && dv <= 128;                          // longer portions in segments
  if (KIND == MIX_MEMORY && (has_long || !regs))
    memory_gates_kernel<T><<<dim3(p.q.n, (p.H + 3) / 4), 128, 0, st>>>(p, regs ? 2 : 1);
  const size_t any_smem = (size_t(3) * dk + dv) * sizeof(float);
  const dim3 by_seq(p.q.n, p.H);
  if (has_single) {
    const int groups = regs ? kMixThreads / (dv / 4) : 0;
    if (regs) matrix_single_kernel<T, KIND><<<by_seq, kMixThreads, (size_t(3) * dk + size_t(1 + groups) * dv) * sizeof(float), st>>>(p);
    else matrix_any_kernel<T, KIND><<<by_seq, 256, any_smem, st>>>(p, 1, 1);
  }
  if (has_long) {
    if (!tiles) {
      matrix_any_kernel<T, KIND><<<by_seq, 256, any_smem, st>>>(p, 2, 1 << 30);
    } else {
#define XL_MIX(DK, DV) return launch_segments<T, KIND, DK, DV>(p, seg_cap, v8, g8, s4, st)
      if constexpr (KIND == MIX_BONUS) {                               // keys and values of one size
        if (dk <= 32) XL_MIX(32, 32);
        if (dk <= 64) XL_MIX(64, 64);
        XL_MIX(128, 128);
      } else {
      if (dk <= 32) { if (dv <= 32) XL_MIX(32, 32); if (dv <= 64) XL_MIX(32, 64); XL_MIX(32, 128); }
      if (dk <= 64) { if (dv <= 32) XL_MIX(64, 32); if (dv <= 64) XL_MIX(64, 64); XL_MIX(64, 128); }
      if (dv <= 32) XL_MIX(128, 32);
      if (dv <= 64) XL_MIX(128, 64);
      XL_MIX(128, 128);
      }
#undef XL_MIX
    }
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

// ============================================================================ selective scan
template <typename T>
struct ScanParams {
  const T* x;                  // [rows, C] dense
  const float* dt;             // [rows, C] dense, ahead of bias and softplus
  const float *dt_bias, *A, *D;   // [C], [C, N], [C]
  const T *B, *Cm;             // [rows, N], row pitch ldb
  const T* z;                  // [rows, C], row pitch ldz
  float* state;                // [records, C, N]
  T* out;                      // [rows, C] dense
  long ldb, ldz;
  int C, N;
  Seqs q;
};

constexpr int kScanThreads = 128, kScanRows = 16;
// exp(step * A) from step * (A * scan_unit): base 2 on the fast path
template <typename T> __device__ __forceinline__ constexpr float scan_unit() { return sizeof(T) == 4 ? 1.f : 1.4426950408889634f; }
template <typename T>
__device__ __forceinline__ float scan_decay(float x) {
  if constexpr (sizeof(T) == 4) return decay_exp<T>(x);
  else return ex2(x);
}

// NPT states per thread, LPC neighbouring lanes per channel (NPT * LPC >= N); states beyond N stay zero.
template <int NPT>
__device__ __forceinline__ void load_states(const float* p, int n0, int N, float (&s)[NPT]) {
  if (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NPT; i += 4) {
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (n0 + i < N) f = *reinterpret_cast<const float4*>(p + n0 + i);
      s[i] = f.x; s[i + 1] = f.y; s[i + 2] = f.z; s[i + 3] = f.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < NPT; ++i) s[i] = n0 + i < N ? p[n0 + i] : 0.f;
  }
}
template <int NPT>
__device__ __forceinline__ void store_states(float* p, int n0, int N, const float (&s)[NPT]) {
  if (N % 4 == 0) {
#pragma unroll
    for (int i = 0; i < NPT; i += 4)
      if (n0 + i < N) *reinterpret_cast<float4*>(p + n0 + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < NPT; ++i)
      if (n0 + i < N) p[n0 + i] = s[i];
  }
}

// Longer portions: a CTA walks one sequence for kScanThreads / LPC channels.  The lanes of a channel share its rows: lane l
// fetches, prepares (step size, silu(z)) and finishes rows l, l + LPC, ...; step sizes and inputs reach the other lanes
// through shared memory, the lanes' sums are put together behind the last row of a tile.  The inputs of the next kScanRows
// rows are under way while the current ones are worked on.
template <typename T, int NPT, int LPC>
__global__ void __launch_bounds__(kScanThreads) scan_rows_kernel(const ScanParams<T> p) {
  constexpr int CPB = kScanThreads / LPC, NP = NPT * LPC;
  constexpr int G = kScanRows / LPC;                                            // rows per lane and tile
  constexpr int NB = kScanRows * 2 * NP / kScanThreads;                         // B and C values per thread and tile
  constexpr bool kAheadB = NB >= 1 && NB <= 16;
  __shared__ __align__(16) float sBC[kScanRows][2 * NP];
  __shared__ float2 sDt[kScanRows][CPB];                                       // (step size, step size * input)
  const int seq = blockIdx.y, tid = threadIdx.x;
  const int start = p.q.q_cu[seq], len = p.q.q_cu[seq + 1] - start;
  if (len < 2) return;
  const int slot = record_of(p.q, seq);
  if (slot < 0) return;
  const bool cont = p.q.kv_lens[seq] > len;
  const int ch = tid / LPC, ln = tid % LPC, n0 = ln * NPT;
  const int c = blockIdx.x * CPB + ch;
  const bool live = c < p.C;
  float s0[NPT], a0[NPT], bias = 0.f, D = 0.f;
#pragma unroll
  for (int i = 0; i < NPT; ++i) s0[i] = a0[i] = 0.f;
  float* rec = p.state + (size_t(slot) * p.C + c) * p.N;
  if (live) {
    load_states<NPT>(p.A + size_t(c) * p.N, n0, p.N, a0);
    if (cont) load_states<NPT>(rec, n0, p.N, s0);
    bias = p.dt_bias[c];
    D = p.D[c];
  }
  uint64_t S[NPT / 2], A[NPT / 2];                         // pairs of neighbouring states
#pragma unroll
  for (int i = 0; i < NPT / 2; ++i) {
    S[i] = pack2(s0[2 * i], s0[2 * i + 1]);
    A[i] = pack2(a0[2 * i] * scan_unit<T>(), a0[2 * i + 1] * scan_unit<T>());
  }
  float rdt[G];
  T rx[G], rz[G], rb[kAheadB ? NB : 1];
  const T zero = T(0.f);
  auto fetch = [&](int b) {
    const int m = min(kScanRows, len - b);
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const int row = g * LPC + ln;
      rdt[g] = 0.f;
      rx[g] = rz[g] = zero;
      if (row < m && live) {
        const size_t t = size_t(start + b + row);
        rdt[g] = p.dt[t * p.C + c];
        rx[g] = p.x[t * p.C + c];
        rz[g] = p.z[t * p.ldz + c];
      }
    }
    if (kAheadB) {
#pragma unroll
      for (int i = 0; i < NB; ++i) {
        const int e = i * kScanThreads + tid, row = e / (2 * NP), n = e % (2 * NP), nn = n < NP ? n : n - NP;
        rb[kAheadB ? i : 0] = zero;
        if (row < m && nn < p.N) rb[kAheadB ? i : 0] = (n < NP ? p.B : p.Cm)[size_t(start + b + row) * p.ldb + nn];
      }
    }
  };
  auto put = [&](int b) {
    if (kAheadB) {
#pragma unroll
      for (int i = 0; i < NB; ++i) (&sBC[0][0])[i * kScanThreads + tid] = to_f32(rb[kAheadB ? i : 0]);
    } else {
      const int m = min(kScanRows, len - b);
      for (int e = tid; e < kScanRows * 2 * NP; e += kScanThreads) {
        const int row = e / (2 * NP), n = e % (2 * NP), nn = n < NP ? n : n - NP;
        (&sBC[0][0])[e] = row < m && nn < p.N ? to_f32((n < NP ? p.B : p.Cm)[size_t(start + b + row) * p.ldb + nn]) : 0.f;
      }
    }
  };
  fetch(0);
  put(0);
  for (int b = 0; b < len; b += kScanRows) {
    const int m = min(kScanRows, len - b);
    float x[G], z[G];
#pragma unroll
    for (int g = 0; g < G; ++g) {                          // rows beyond m: a step of size 0 leaves the state as it is
      const float dt = g * LPC + ln < m ? softplus(rdt[g] + bias) : 0.f;
      x[g] = to_f32(rx[g]);
      z[g] = to_f32(rz[g]);
      sDt[g * LPC + ln][ch] = make_float2(dt, dt * x[g]);
    }
    __syncthreads();
    if (b + kScanRows < len) fetch(b + kScanRows);
    float y[kScanRows];
    constexpr int RG = NPT <= 4 ? 4 : NPT <= 8 ? 2 : 1;    // rows whose factors and inputs are prepared ahead of the recurrence
#pragma unroll
    for (int r0 = 0; r0 < kScanRows; r0 += RG) {
      uint64_t e[RG][NPT / 2], u[RG][NPT / 2];
#pragma unroll
      for (int r = 0; r < RG; ++r) {
        const float2 d = sDt[r0 + r][ch];
        const uint64_t dt2 = pack2(d.x, d.x), dx2 = pack2(d.y, d.y);
#pragma unroll
        for (int i = 0; i < NPT / 2; i += 2) {
          const ulonglong2 bb = *reinterpret_cast<const ulonglong2*>(&sBC[r0 + r][n0 + 2 * i]);
          const float2 f0 = unpack2(mul2(dt2, A[i])), f1 = unpack2(mul2(dt2, A[i + 1]));
          e[r][i] = pack2(scan_decay<T>(f0.x), scan_decay<T>(f0.y));
          e[r][i + 1] = pack2(scan_decay<T>(f1.x), scan_decay<T>(f1.y));
          u[r][i] = mul2(dx2, bb.x);
          u[r][i + 1] = mul2(dx2, bb.y);
        }
      }
#pragma unroll
      for (int r = 0; r < RG; ++r) {
        uint64_t acc[2] = {0, 0};
#pragma unroll
        for (int i = 0; i < NPT / 2; i += 2) {
          const ulonglong2 cm = *reinterpret_cast<const ulonglong2*>(&sBC[r0 + r][NP + n0 + 2 * i]);
          S[i] = fma2(e[r][i], S[i], u[r][i]);
          S[i + 1] = fma2(e[r][i + 1], S[i + 1], u[r][i + 1]);
          acc[0] = fma2(S[i], cm.x, acc[0]);
          acc[1] = fma2(S[i + 1], cm.y, acc[1]);
        }
        const float2 f0 = unpack2(acc[0]), f1 = unpack2(acc[1]);
        y[r0 + r] = (f0.x + f0.y) + (f1.x + f1.y);
      }
    }
#pragma unroll
    for (int g = 0; g < G; ++g) {
      float part[LPC];
#pragma unroll
      for (int l = 0; l < LPC; ++l) part[l] = y[g * LPC + l];
      const float sum = sum_to_lanes<LPC>(part, ln);
      const int row = g * LPC + ln;
      if (row < m && live) from_f32(p.out + size_t(start + b + row) * p.C + c, fmaf(D, x[g], sum) * act_silu(z[g]));
    }
    __syncthreads();                                       // the tile's rows are read: both arrays may be written again
    if (b + kScanRows < len) put(b + kScanRows);
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < NPT / 2; ++i) {
      const float2 f = unpack2(S[i]);
      s0[2 * i] = f.x;
      s0[2 * i + 1] = f.y;
    }
    store_states<NPT>(rec, n0, p.N, s0);
  }
}

// Single rows: LPC lanes per channel, NPT states each, and several sequences per thread, so that A is read once for them and
// the states of all of them are under way before any is worked on.  Lane k prepares and finishes sequence k.  bc4: B and C can
// be read four at a time.
template <int NPT, int LPC> struct SingleCfg { static constexpr int NS = NPT > 4 ? 1 : LPC < 8 ? LPC : 8; };
template <typename T>
__device__ __forceinline__ void load_bc4(const T* p, float* f) {
  if constexpr (sizeof(T) == 2) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
    *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(p);
  }
}
template <typename T, int NPT, int LPC>
__global__ void __launch_bounds__(kScanThreads) scan_single_kernel(const ScanParams<T> p, int bc4) {
  constexpr int CPB = kScanThreads / LPC, NS = SingleCfg<NPT, LPC>::NS;
  const int tid = threadIdx.x, ch = tid / LPC, ln = tid % LPC, n0 = ln * NPT;
  const int c = blockIdx.x * CPB + ch;
  const bool live = c < p.C;
  // this lane's sequence
  const int own = ln % NS, my_seq = blockIdx.y * NS + own;
  int my_t = 0, my_slot = -1;
  bool my_cont = false;
  if (my_seq < p.q.n) {
    my_t = p.q.q_cu[my_seq];
    if (p.q.q_cu[my_seq + 1] - my_t == 1) {
      my_slot = p.q.slots[my_seq];
      my_cont = p.q.kv_lens[my_seq] > 1;
      if (my_slot < 0 || my_slot >= p.q.n_slots) {
        if (tid < NS) atomicExch(p.q.status, XL_ERR_BOUNDS);
        my_slot = -1;
      }
    }
  }
  if (!__any_sync(0xffffffffu, my_slot >= 0)) return;
  const bool mine = live && my_slot >= 0;
  float dt = 0.f, x = 0.f, z = 0.f, bias = 0.f, D = 0.f;
  if (mine) {
    dt = p.dt[size_t(my_t) * p.C + c];
    x = to_f32(p.x[size_t(my_t) * p.C + c]);
    z = to_f32(p.z[size_t(my_t) * p.ldz + c]);
  }
  float S[NS][NPT], A[NPT];
  int t[NS], slot[NS];
#pragma unroll
  for (int k = 0; k < NS; ++k) {
    t[k] = __shfl_sync(0xffffffffu, my_t, k, LPC);
    slot[k] = __shfl_sync(0xffffffffu, my_slot, k, LPC);
    const bool cont = __shfl_sync(0xffffffffu, int(my_cont), k, LPC);
#pragma unroll
    for (int i = 0; i < NPT; ++i) S[k][i] = 0.f;
    if (live && slot[k] >= 0 && cont) load_states<NPT>(p.state + (size_t(slot[k]) * p.C + c) * p.N, n0, p.N, S[k]);
  }
#pragma unroll
  for (int i = 0; i < NPT; ++i) A[i] = 0.f;
  if (live) {
    load_states<NPT>(p.A + size_t(c) * p.N, n0, p.N, A);
    bias = p.dt_bias[c];
    D = p.D[c];
#pragma unroll
    for (int i = 0; i < NPT; ++i) A[i] *= scan_unit<T>();
  }
  const float step = softplus(dt + bias), dx = step * x;
  float y[NS];
#pragma unroll
  for (int k = 0; k < NS; ++k) {
    y[k] = 0.f;
    const float step_k = __shfl_sync(0xffffffffu, step, k, LPC), dx_k = __shfl_sync(0xffffffffu, dx, k, LPC);
    if (slot[k] < 0) continue;                             // the same in every lane
    float B[NPT], Cm[NPT];
    const T *bp = p.B + size_t(t[k]) * p.ldb + n0, *cp = p.Cm + size_t(t[k]) * p.ldb + n0;
#pragma unroll
    for (int i = 0; i < NPT; i += 4) {
#pragma unroll
      for (int e = 0; e < 4; ++e) B[i + e] = Cm[i + e] = 0.f;
      if (bc4) {
        if (n0 + i < p.N) {
          load_bc4(bp + i, B + i);
          load_bc4(cp + i, Cm + i);
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (n0 + i + e < p.N) {
            B[i + e] = to_f32(bp[i + e]);
            Cm[i + e] = to_f32(cp[i + e]);
          }
      }
    }
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
      S[k][i] = fmaf(scan_decay<T>(step_k * A[i]), S[k][i], dx_k * B[i]);
      y[k] = fmaf(S[k][i], Cm[i], y[k]);
    }
    if (live) store_states<NPT>(p.state + (size_t(slot[k]) * p.C + c) * p.N, n0, p.N, S[k]);
  }
  float sum = sum_to_lanes<NS>(y, ln);
#pragma unroll
  for (int o = NS; o < LPC; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  if (mine && ln < NS) from_f32(p.out + size_t(my_t) * p.C + c, fmaf(D, x, sum) * act_silu(z));
}

template <typename T, int NPT, int LPC>
static int launch_rows(const ScanParams<T>& p, cudaStream_t st) {
  constexpr int CPB = kScanThreads / LPC;
  scan_rows_kernel<T, NPT, LPC><<<dim3((p.C + CPB - 1) / CPB, p.q.n), kScanThreads, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}
template <typename T, int NPT, int LPC>
static int launch_single(const ScanParams<T>& p, cudaStream_t st) {
  constexpr int CPB = kScanThreads / LPC;
  constexpr int NS = SingleCfg<NPT, LPC>::NS;
  const int bytes = 4 * int(sizeof(T));
  const bool bc4 = p.N % 4 == 0 && (p.ldb * sizeof(T)) % bytes == 0 && reinterpret_cast<uintptr_t>(p.B) % bytes == 0 &&
                   reinterpret_cast<uintptr_t>(p.Cm) % bytes == 0;
  scan_single_kernel<T, NPT, LPC><<<dim3((p.C + CPB - 1) / CPB, (p.q.n + NS - 1) / NS), kScanThreads, 0, st>>>(p, bc4);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}
template <typename T>
static int launch_scan(const ScanParams<T>& p, int has_long, int has_single, cudaStream_t st) {
  const int n = p.N;
  if (n > 256) return -2;
  int rc = 0;
  if (has_single) {
    if (n <= 4) rc = launch_single<T, 4, 1>(p, st);
    else if (n <= 8) rc = launch_single<T, 4, 2>(p, st);
    else if (n <= 16) rc = launch_single<T, 4, 4>(p, st);
    else if (n <= 32) rc = launch_single<T, 4, 8>(p, st);
    else if (n <= 64) rc = launch_single<T, 4, 16>(p, st);
    else if (n <= 128) rc = launch_single<T, 4, 32>(p, st);
    else rc = launch_single<T, 8, 32>(p, st);
  }
  if (rc || !has_long) return rc;
  if (n <= 4) return launch_rows<T, 4, 1>(p, st);
  if (n <= 8) return launch_rows<T, 8, 1>(p, st);
  // few channels x sequences: more lanes per channel, so that every scheduler has more than one warp
  if (n <= 16) return long(p.C) * p.q.n <= 4096 * 3 ? launch_rows<T, 4, 4>(p, st) : launch_rows<T, 8, 2>(p, st);
  if (n <= 32) return launch_rows<T, 8, 4>(p, st);
  if (n <= 64) return launch_rows<T, 8, 8>(p, st);
  if (n <= 128) return launch_rows<T, 16, 8>(p, st);
  return launch_rows<T, 32, 8>(p, st);
}

template <typename F>
static int by_type(int f32, F&& f) {
  return f32 ? f(static_cast<float*>(nullptr)) : f(static_cast<__nv_bfloat16*>(nullptr));
}
static Seqs make_seqs(const void* q_cu, const void* kv_lens, const void* slots, int n, int n_slots) {
  return Seqs{static_cast<const int*>(q_cu), static_cast<const int*>(kv_lens), static_cast<const int*>(slots), n, n_slots,
              xl_host::status_word()};
}
static bool aligned16(const void* a, const void* b, const void* c, const void* d) {
  return !((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c) |
            reinterpret_cast<uintptr_t>(d)) & 15);
}

}  // namespace xl_rc

using namespace xl_rc;

// `f32` below: 1 when the model's tensors are fp32, 0 for bf16.  q_cu [n_seqs + 1], kv_lens and slots [n_seqs].
// `has_long` / `has_single`: whether any sequence of the step may have several rows / a single one.

// out [n_mix, rows, W] = h + (previous row of the sequence - h) * mu[j]; last [n_slots, W]
XL_API int xl_token_shift(const void* h, const void* mu, void* last, void* out, const void* token_seq, const void* q_cu,
                          const void* kv_lens, const void* slots, int n_seqs, int n_slots, int rows, int W, int n_mix, int f32,
                          void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const Seqs q = make_seqs(q_cu, kv_lens, slots, n_seqs, n_slots);
  return by_type(f32, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const T *hh = static_cast<const T*>(h), *m = static_cast<const T*>(mu);
    T *l = static_cast<T*>(last), *o = static_cast<T*>(out);
    const int* ts = static_cast<const int*>(token_seq);
    if (W % 8 == 0 && aligned16(h, mu, last, out)) token_shift_kernel<T, 8><<<rows, 256, 0, st>>>(hh, m, l, o, ts, q, rows, W, n_mix);
    else token_shift_kernel<T, 1><<<rows, 256, 0, st>>>(hh, m, l, o, ts, q, rows, W, n_mix);
    return cudaGetLastError() == cudaSuccess ? 0 : -1;
  });
}

// out [rows, C] = act(bias + causal convolution of x (row pitch ldx) with w [taps, C]) (+ x); bias may be null; act: silu or none;
// state [n_slots, taps - 1, C]
XL_API int xl_causal_conv(const void* x, const void* w, const void* bias, void* state, void* out, const void* token_seq, const void* q_cu,
                          const void* kv_lens, const void* slots, int n_seqs, int n_slots, int rows, int C, int taps, long ldx,
                          int has_long, int silu, int residual, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (taps < 1) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const Seqs q = make_seqs(q_cu, kv_lens, slots, n_seqs, n_slots);
  const ConvOut act{silu, residual};
  return by_type(f32, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    const T *xx = static_cast<const T*>(x), *ww = static_cast<const T*>(w), *b = static_cast<const T*>(bias);
    T *s = static_cast<T*>(state), *o = static_cast<T*>(out);
    const int* ts = static_cast<const int*>(token_seq);
    const bool vec = C % 8 == 0 && ldx % 8 == 0 && aligned16(x, bias, state, out) && aligned16(w, w, w, w);
    const int per = vec ? 8 : 1, cols = (C + per * 128 - 1) / (per * 128);
    const int tile = has_long ? kConvRows : kConvRowsSingle;
    const dim3 grid((rows + tile - 1) / tile, cols);
#define XL_CONV(V, TAPS)                                                                                              \
  if (has_long) causal_conv_kernel<T, V, TAPS, kConvRows><<<grid, 128, 0, st>>>(xx, ww, b, s, o, ts, q, rows, C, taps, ldx, act); \
  else causal_conv_kernel<T, V, TAPS, kConvRowsSingle><<<grid, 128, 0, st>>>(xx, ww, b, s, o, ts, q, rows, C, taps, ldx, act)
    if (vec) {
      if (taps == 4) { XL_CONV(8, 4); } else if (taps == 3) { XL_CONV(8, 3); } else if (taps == 2) { XL_CONV(8, 2); } else { XL_CONV(8, 0); }
    } else {
      XL_CONV(1, 0);
    }
#undef XL_CONV
    if (has_long && taps > 1) {
      if (vec) conv_record_kernel<T, 8><<<dim3(n_seqs, cols), 128, 0, st>>>(xx, s, q, C, taps, ldx);
      else conv_record_kernel<T, 1><<<dim3(n_seqs, cols), 128, 0, st>>>(xx, s, q, C, taps, ldx);
    }
    return cudaGetLastError() == cudaSuccess ? 0 : -1;
  });
}

// What the matrix-state entry points share: r (queries) and k [rows, H * dk], v [rows, H * dv] with row pitch ld, gate with ldg; out with
// row pitch ldo.  Longer portions in segments of L rows, at most seg_cap of them; ws_s / ws_p (null when no portion has more
// than L rows) hold seg_cap * H records and seg_cap * H * dk floats.
struct MatrixArgs {
  const void *r, *k, *v, *z, *w0, *u, *gate, *norm_w;
  float scale, eps;
  void *state, *out;
  const void *q_cu, *kv_lens, *slots;
  int n_seqs, n_slots, H, dk, dv, norm_step;
  long ld, ldg, ldo;
  int L, seg_cap;
  void *ws_s, *ws_p;
  int has_long, has_single, f32;
  void* stream;
  float inv_tau, cap;
  void *top, *fi;
  int rows;
};
template <int KIND>
static int run_matrix(const MatrixArgs& a) {
  if (a.n_seqs <= 0) return 0;
  if (a.H < 1 || a.H > 65535 || a.dk < 1 || a.dk > 2048 || a.dv < 1 || a.dv > 2048 || a.L < 2) return -2;
  return by_type(a.f32, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    MixParams<T> p = {};
    p.r = static_cast<const T*>(a.r); p.k = static_cast<const T*>(a.k); p.v = static_cast<const T*>(a.v);
    p.gate = static_cast<const T*>(a.gate);
    p.z = static_cast<const float*>(a.z); p.w0 = static_cast<const float*>(a.w0); p.u = static_cast<const float*>(a.u);
    p.norm_w = static_cast<const T*>(a.norm_w); p.norm_step = a.norm_step;
    p.state = static_cast<float*>(a.state); p.out = static_cast<T*>(a.out);
    p.ld = a.ld; p.ldg = a.ldg; p.ldo = a.ldo; p.H = a.H; p.dk = a.dk; p.dv = a.dv; p.scale = a.scale; p.eps = a.eps;
    p.q_scale = 1.f / sqrtf(float(a.dk)); p.inv_tau = a.inv_tau; p.cap = a.cap;
    p.top = static_cast<float*>(a.top); p.fi = static_cast<float*>(a.fi); p.rows = a.rows;
    p.q = make_seqs(a.q_cu, a.kv_lens, a.slots, a.n_seqs, a.n_slots);
    p.L = a.L; p.ws_s = static_cast<float*>(a.ws_s); p.ws_p = static_cast<float*>(a.ws_p);
    return launch_matrix<T, KIND>(p, a.seg_cap, a.has_long, a.has_single, static_cast<cudaStream_t>(a.stream));
  });
}

// Time mixing: z [rows, H * d] fp32 dense; state [n_slots, H, d, d] fp32.
XL_API int xl_time_mix(const void* r, const void* k, const void* v, const void* z, const void* w0, const void* u, const void* gate,
                       const void* norm_w, float scale, float eps, void* state, void* out, const void* q_cu, const void* kv_lens,
                       const void* slots, int n_seqs, int n_slots, int H, int d, long ld, long ldg, long ldo, int L, int seg_cap,
                       void* ws_s, void* ws_p, int has_long, int has_single, int f32, void* stream) {
  return run_matrix<MIX_BONUS>(MatrixArgs{r, k, v, z, w0, u, gate, norm_w, scale, eps, state, out, q_cu, kv_lens, slots, n_seqs, n_slots, H, d,
                                          d, d, ld, ldg, ldo, L, seg_cap, ws_s, ws_p, has_long, has_single, f32, stream, 0.f, 0.f, nullptr,
                                          nullptr, 0});
}

// Gated linear attention: z [rows, H * dk] fp32 dense, decay sigmoid(z + bias)^inv_tau; state [n_slots, H, dk, dv] fp32; norm_w [dv].
XL_API int xl_gated_memory(const void* q, const void* k, const void* v, const void* z, const void* bias, float inv_tau, const void* gate,
                           const void* norm_w, float eps, void* state, void* out, const void* q_cu, const void* kv_lens, const void* slots,
                           int n_seqs, int n_slots, int H, int dk, int dv, long ld, long ldg, long ldo, int L, int seg_cap, void* ws_s,
                           void* ws_p, int has_long, int has_single, int f32, void* stream) {
  return run_matrix<MIX_GATED>(MatrixArgs{q, k, v, z, bias, nullptr, gate, norm_w, 1.f, eps, state, out, q_cu, kv_lens, slots, n_seqs, n_slots,
                                          H, dk, dv, 0, ld, ldg, ldo, L, seg_cap, ws_s, ws_p, has_long, has_single, f32, stream, inv_tau,
                                          0.f, nullptr, nullptr, 0});
}

// Matrix memory: gates [rows, 2 H] fp32 dense ahead of bias [2 H] and the bound `cap`; state [n_slots, H, dk * dv + dk] fp32, top
// [n_slots, H] fp32; norm_w [H * dv]; fi: 3 * H * rows floats of workspace.
XL_API int xl_matrix_memory(const void* q, const void* k, const void* v, const void* gates, const void* bias, float cap, const void* gate,
                            const void* norm_w, float eps, void* state, void* top, void* out, const void* q_cu, const void* kv_lens,
                            const void* slots, int n_seqs, int n_slots, int H, int dk, int dv, long ld, long ldg, long ldo, int L, int seg_cap,
                            void* ws_s, void* ws_p, void* fi, int rows, int has_long, int has_single, int f32, void* stream) {
  if (!fi || cap <= 0.f) return -2;
  return run_matrix<MIX_MEMORY>(MatrixArgs{q, k, v, gates, bias, nullptr, gate, norm_w, 1.f, eps, state, out, q_cu, kv_lens, slots, n_seqs,
                                           n_slots, H, dk, dv, dv, ld, ldg, ldo, L, seg_cap, ws_s, ws_p, has_long, has_single, f32, stream, 0.f,
                                           cap, top, fi, rows});
}

// out [rows, C] = (scan + D x) silu(z); B, Cm with row pitch ldb, z with ldz; state [n_slots, C, N] fp32
XL_API int xl_selective_scan(const void* x, const void* dt, const void* dt_bias, const void* A, const void* B, const void* Cm,
                             const void* D, const void* z, void* state, void* out, const void* q_cu, const void* kv_lens,
                             const void* slots, int n_seqs, int n_slots, int C, int N, long ldb, long ldz, int has_long, int has_single,
                             int f32, void* stream) {
  if (n_seqs <= 0) return 0;
  if (C < 1 || N < 1 || n_seqs > 65535) return -2;
  return by_type(f32, [&](auto* tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    ScanParams<T> p;
    p.x = static_cast<const T*>(x); p.dt = static_cast<const float*>(dt); p.dt_bias = static_cast<const float*>(dt_bias);
    p.A = static_cast<const float*>(A); p.D = static_cast<const float*>(D);
    p.B = static_cast<const T*>(B); p.Cm = static_cast<const T*>(Cm); p.z = static_cast<const T*>(z);
    p.state = static_cast<float*>(state); p.out = static_cast<T*>(out);
    p.ldb = ldb; p.ldz = ldz; p.C = C; p.N = N;
    p.q = make_seqs(q_cu, kv_lens, slots, n_seqs, n_slots);
    return launch_scan<T>(p, has_long, has_single, static_cast<cudaStream_t>(stream));
  });
}
