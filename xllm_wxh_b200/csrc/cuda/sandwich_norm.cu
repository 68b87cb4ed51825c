// Fused steps around an fp32 residual stream, of decoders whose sublayers are normed before and after:
//
//   x += rms(y) * w_post;  h = rms(x) * w_next                      (one kernel between a sublayer and the next one)
//
// with three sources of the first line:
//   SRC_ROWS   y is a tensor (the output of o_proj / down_proj);
//   SRC_MOE    y is assembled here: weighted sum of the chosen experts' rows, identity experts (whose output is the
//              sublayer's input itself, times the weight) and a shared expert, so that it never exists in memory;
//   SRC_PAIR   y is put together here from two branches, each normed with a weight of its own;
//   SRC_EMBED  there is no y: x = table[token] * scale (normed itself if w_post is given) starts the residual stream;
// and of decoders whose sublayers are normed before only:
//   SRC_ADD    x += scale * y                                    (no norm behind the sublayer)
//   SRC_SET    x = y + vec, y in fp32                            (the residual is replaced by a product of itself)
//   SRC_MOE with `add_only`  as SRC_ADD, y assembled as in SRC_MOE
// SRC_ADD and SRC_MOE may scale y by a vector (layer scale) and add embedding rows to x (`lead`, at the head of a pass through a
// loop); embedding rows may have a position vector; the norm's weight may be stored as its distance from `w_off`.
// Also the kernel that follows the qkv projection where positions do not rotate anything: per-head q / k RMSNorm and the
// write of k and v into the paged cache (q is normed in place), with norms per head (and a rotation behind them) or over the whole
// projection; the norms, rotation and cache write of latent attention's down projection, and the rotation of its queries; the gated
// activation of an unfused feed-forward; a sigmoid gate on attention's output; and the rows [x, x0] of a product that takes
// in the residual stream.
//
// All arithmetic is fp32; tensors are bf16, or fp32 when the model runs in 32-bit.
#include <type_traits>

#include "vec8.cuh"

namespace xl_sn {
using namespace xl;

enum { SRC_ROWS = 0, SRC_MOE = 1, SRC_EMBED = 2, SRC_ADD = 3, SRC_SET = 4, SRC_PAIR = 5 };

template <typename T>
struct NormParams {
  float* x;                  // [rows, H] fp32 residual stream, updated in place (SRC_EMBED: written)
  const T* w_post;           // [H] weight of the norm behind the sublayer
  const T* w_next;           // [H] weight of the norm ahead of the next sublayer
  T* h;                      // [rows, H] its output
  int H;
  float eps;
  const T* y;                // SRC_ROWS, SRC_PAIR: [rows, H]
  const T *y2, *w_y, *w_y2;  // SRC_PAIR: y = scale * (rms(y) w_y + rms(y2) w_y2)
  // SRC_MOE
  const T* y_exp;            // [*, H] expert outputs, row dst_of[t * k + j] belongs to choice j of token t (-1: none)
  const int* dst_of;
  const int* ids;            // [rows, k] chosen experts; ids >= first_identity are identity experts
  const float* weights;      // [rows, k]
  const T* h_in;             // [rows, H] the sublayer's input (identity experts)
  const T* shared;           // [rows, H] or null
  int k, first_identity;
  // SRC_EMBED
  const int* tokens;
  const T* table;            // [V, H]
  int V;
  float scale;               // also SRC_ADD, SRC_PAIR
  // SRC_SET
  const float* y32;          // [rows, H]
  const float* vec;          // [H]
  float w_off;               // joins w_next
  const T* ls;               // SRC_ADD, SRC_MOE with add_only: [H] factor of y (null: `scale`)
  int add_only;              // SRC_MOE: no norm behind the sublayer
  // rows of an embedding: SRC_EMBED (tokens, table, V, scale above), and `lead` of the others
  const int* positions;
  const T* pos_table;        // [pos_rows, H] or null
  int pos_rows;
  int lead;                  // add table[token] * lead_scale + pos_table[position] to x
  float lead_scale;
  int keep_x;                // SRC_EMBED: x is added to instead of written
};

// sum over the block of one value per thread; `red` holds one float per warp
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  const int warps = (blockDim.x + 31) >> 5;
  for (int i = 0; i < warps; ++i) t += red[i];
  return t;
}

// the same for two values; `red` holds two floats per warp
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  a = warp_sum(a);
  b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) {
    red[threadIdx.x >> 5] = a;
    red[8 + (threadIdx.x >> 5)] = b;
  }
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
  const int warps = (blockDim.x + 31) >> 5;
  for (int i = 0; i < warps; ++i) {
    t.x += red[i];
    t.y += red[8 + i];
  }
  return t;
}

__device__ __forceinline__ int clamp_id(int id, int V) { return id < 0 ? 0 : (id >= V ? V - 1 : id); }

// Embedding row (8 elements from column c), times s, plus its position vector.
template <typename T>
__device__ __forceinline__ void embed8(const NormParams<T>& p, int row, int c, float s, float (&y)[8]) {
  load8(p.table + size_t(clamp_id(p.tokens[row], p.V)) * p.H + c, y);
#pragma unroll
  for (int e = 0; e < 8; ++e) y[e] *= s;
  if (p.pos_table) {
    float f[8];
    load8(p.pos_table + size_t(clamp_id(p.positions[row], p.pos_rows)) * p.H + c, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) y[e] += f[e];
  }
}
template <typename T>
__device__ __forceinline__ float embed1(const NormParams<T>& p, int row, int c, float s) {
  const float y = to_f32(p.table[size_t(clamp_id(p.tokens[row], p.V)) * p.H + c]) * s;
  return p.pos_table ? y + to_f32(p.pos_table[size_t(clamp_id(p.positions[row], p.pos_rows)) * p.H + c]) : y;
}

// Register-resident rows: thread i owns the 8-element vectors i, i + blockDim, ... (VPT of them).
template <typename T, int VPT, int SRC>
__global__ void __launch_bounds__(256) sandwich_norm_kernel(const NormParams<T> p) {
  __shared__ float red_a[8], red_b[8], red_c[SRC == SRC_PAIR ? 16 : 1];
  const int row = blockIdx.x, H = p.H, nvec = H / 8;
  float y[VPT][8];
  float ss = 0.f;
  float w_id = 0.f;          // summed weight of this token's identity choices
  if (SRC == SRC_MOE) {
    for (int j = 0; j < p.k; ++j)
      if (p.ids[row * p.k + j] >= p.first_identity) w_id += p.weights[row * p.k + j];
  }
  if constexpr (SRC == SRC_PAIR) {
    float b[VPT][8], sa = 0.f, sb = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nvec) {
        load8(p.y + size_t(row) * H + v * 8, y[i]);
        load8(p.y2 + size_t(row) * H + v * 8, b[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          sa += y[i][e] * y[i][e];
          sb += b[i][e] * b[i][e];
        }
      }
    }
    const float2 s = block_sum2(sa, sb, red_c);
    const float ra = rsqrtf(s.x / float(H) + p.eps) * p.scale, rb = rsqrtf(s.y / float(H) + p.eps) * p.scale;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nvec) {
        float wa[8], wb[8];
        load8(p.w_y + v * 8, wa);
        load8(p.w_y2 + v * 8, wb);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[i][e] = fmaf(y[i][e] * ra, wa[e], b[i][e] * rb * wb[e]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nvec) {
      if (SRC == SRC_PAIR) {                               // put together above
      } else if (SRC == SRC_ROWS) {
        load8(p.y + size_t(row) * H + v * 8, y[i]);
      } else if (SRC == SRC_ADD) {
        float x[8], s[8];
        load8(p.y + size_t(row) * H + v * 8, y[i]);
        load8(p.x + size_t(row) * H + v * 8, x);
        if (p.ls) {
          load8(p.ls + v * 8, s);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) s[e] = p.scale;
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) y[i][e] = fmaf(s[e], y[i][e], x[e]);
        if (p.lead) {
          embed8(p, row, v * 8, p.lead_scale, x);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[i][e] += x[e];
        }
      } else if (SRC == SRC_SET) {
        float x[8];
        load8(p.y32 + size_t(row) * H + v * 8, y[i]);
        load8(p.vec + v * 8, x);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[i][e] += x[e];
      } else if (SRC == SRC_EMBED) {
        embed8(p, row, v * 8, p.scale, y[i]);
        if (p.keep_x) {
          float x[8];
          load8(p.x + size_t(row) * H + v * 8, x);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[i][e] += x[e];
        }
      } else {
        float f[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) y[i][e] = 0.f;
        if (p.shared) load8(p.shared + size_t(row) * H + v * 8, y[i]);
        if (w_id != 0.f) {
          load8(p.h_in + size_t(row) * H + v * 8, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[i][e] += w_id * f[e];
        }
        for (int j = 0; j < p.k; ++j) {
          const int r = p.dst_of[row * p.k + j];
          if (r < 0) continue;
          const float wj = p.weights[row * p.k + j];
          load8(p.y_exp + size_t(r) * H + v * 8, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[i][e] += wj * f[e];
        }
        if (p.add_only) {
          float x[8];
          load8(p.x + size_t(row) * H + v * 8, x);
          load8(p.ls + v * 8, f);
#pragma unroll
          for (int e = 0; e < 8; ++e) y[i][e] = fmaf(f[e], y[i][e], x[e]);
          if (p.lead) {
            embed8(p, row, v * 8, p.lead_scale, x);
#pragma unroll
            for (int e = 0; e < 8; ++e) y[i][e] += x[e];
          }
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += y[i][e] * y[i][e];
    }
  }
  const bool post = SRC == SRC_ROWS || SRC == SRC_PAIR || (SRC == SRC_MOE && !p.add_only) || (SRC == SRC_EMBED && p.w_post);
  if (post) {
    const float r_post = rsqrtf(block_sum(ss, red_a) / float(H) + p.eps);
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nvec) {
        float w[8], x[8] = {};
        load8(p.w_post + v * 8, w);
        if (SRC != SRC_EMBED) load8(p.x + size_t(row) * H + v * 8, x);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          y[i][e] = x[e] + y[i][e] * r_post * w[e];
          ss += y[i][e] * y[i][e];
        }
      }
    }
  }
  const float r_next = rsqrtf(block_sum(ss, red_b) / float(H) + p.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nvec) {
      float w[8];
      load8(p.w_next + v * 8, w);
      store8(p.x + size_t(row) * H + v * 8, y[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e] = y[i][e] * r_next * (w[e] + p.w_off);
      store8(p.h + size_t(row) * H + v * 8, w);
    }
  }
}

// Any width: one element at a time, the row kept in shared memory.
template <typename T, int SRC>
__global__ void __launch_bounds__(256) sandwich_norm_any_kernel(const NormParams<T> p) {
  extern __shared__ float row_cache[];
  __shared__ float red_a[8], red_b[8], red_c[SRC == SRC_PAIR ? 16 : 1];
  const int row = blockIdx.x, H = p.H;
  float ss = 0.f, w_id = 0.f, ra = 0.f, rb = 0.f;
  if constexpr (SRC == SRC_PAIR) {
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float a = to_f32(p.y[size_t(row) * H + i]), b = to_f32(p.y2[size_t(row) * H + i]);
      ra += a * a;
      rb += b * b;
    }
    const float2 s = block_sum2(ra, rb, red_c);
    ra = rsqrtf(s.x / float(H) + p.eps) * p.scale;
    rb = rsqrtf(s.y / float(H) + p.eps) * p.scale;
  }
  if (SRC == SRC_MOE) {
    for (int j = 0; j < p.k; ++j)
      if (p.ids[row * p.k + j] >= p.first_identity) w_id += p.weights[row * p.k + j];
  }
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float y = 0.f;
    if (SRC == SRC_PAIR) {
      const size_t at = size_t(row) * H + i;
      y = fmaf(to_f32(p.y[at]) * ra, to_f32(p.w_y[i]), to_f32(p.y2[at]) * rb * to_f32(p.w_y2[i]));
    } else if (SRC == SRC_ROWS) {
      y = to_f32(p.y[size_t(row) * H + i]);
    } else if (SRC == SRC_ADD) {
      y = fmaf(p.ls ? to_f32(p.ls[i]) : p.scale, to_f32(p.y[size_t(row) * H + i]), p.x[size_t(row) * H + i]);
      if (p.lead) y += embed1(p, row, i, p.lead_scale);
    } else if (SRC == SRC_SET) {
      y = p.y32[size_t(row) * H + i] + p.vec[i];
    } else if (SRC == SRC_EMBED) {
      y = embed1(p, row, i, p.scale);
      if (p.keep_x) y += p.x[size_t(row) * H + i];
    } else {
      if (p.shared) y = to_f32(p.shared[size_t(row) * H + i]);
      if (w_id != 0.f) y += w_id * to_f32(p.h_in[size_t(row) * H + i]);
      for (int j = 0; j < p.k; ++j) {
        const int r = p.dst_of[row * p.k + j];
        if (r >= 0) y += p.weights[row * p.k + j] * to_f32(p.y_exp[size_t(r) * H + i]);
      }
      if (p.add_only) {
        y = fmaf(to_f32(p.ls[i]), y, p.x[size_t(row) * H + i]);
        if (p.lead) y += embed1(p, row, i, p.lead_scale);
      }
    }
    row_cache[i] = y;
    ss += y * y;
  }
  if (SRC == SRC_ROWS || SRC == SRC_PAIR || (SRC == SRC_MOE && !p.add_only) || (SRC == SRC_EMBED && p.w_post)) {
    const float r_post = rsqrtf(block_sum(ss, red_a) / float(H) + p.eps);
    ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
      const float x = (SRC == SRC_EMBED ? 0.f : p.x[size_t(row) * H + i]) + row_cache[i] * r_post * to_f32(p.w_post[i]);
      row_cache[i] = x;
      ss += x * x;
    }
  }
  const float r_next = rsqrtf(block_sum(ss, red_b) / float(H) + p.eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    p.x[size_t(row) * H + i] = row_cache[i];
    from_f32(p.h + size_t(row) * H + i, row_cache[i] * r_next * (to_f32(p.w_next[i]) + p.w_off));
  }
}

template <typename T, int SRC>
static int launch_norm(const NormParams<T>& p, int rows, bool aligned, cudaStream_t st) {
  if (rows <= 0) return 0;
  const int nvec = p.H / 8;
  if (aligned && p.H % 8 == 0 && nvec <= 1024) {
    const int vpt = nvec <= 256 ? 1 : nvec <= 512 ? 2 : 4;
    const int threads = ((nvec + vpt - 1) / vpt + 31) / 32 * 32;
    if (vpt == 1) sandwich_norm_kernel<T, 1, SRC><<<rows, threads, 0, st>>>(p);
    else if (vpt == 2) sandwich_norm_kernel<T, 2, SRC><<<rows, threads, 0, st>>>(p);
    else sandwich_norm_kernel<T, 4, SRC><<<rows, threads, 0, st>>>(p);
  } else {
    const size_t smem = size_t(p.H) * sizeof(float);
    if (smem > 200 * 1024) return -2;
    static bool set = false;
    if (!set) {
      cudaFuncSetAttribute(sandwich_norm_any_kernel<T, SRC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      set = true;
    }
    sandwich_norm_any_kernel<T, SRC><<<rows, 256, smem, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

static bool al16(const void* a, const void* b = nullptr, const void* c = nullptr, const void* d = nullptr) {
  return !((reinterpret_cast<uintptr_t>(a) | reinterpret_cast<uintptr_t>(b) | reinterpret_cast<uintptr_t>(c) |
            reinterpret_cast<uintptr_t>(d)) & 15);
}

template <typename T>
static NormParams<T> base_params(void* x, const void* w_post, const void* w_next, void* h, int H, float eps) {
  NormParams<T> p = {};
  p.x = static_cast<float*>(x);
  p.w_post = static_cast<const T*>(w_post);
  p.w_next = static_cast<const T*>(w_next);
  p.h = static_cast<T*>(h);
  p.H = H;
  p.eps = eps;
  return p;
}

// ---------------------------------------------------------------- q / k norm + cache write
// LPH lanes per (token, head), 8 elements per lane; heads as laid out by the fused qkv projection:
// n_q query heads of dk, n_k key heads of dk, n_v value heads of dv.
struct Rotation {
  const float* table;        // [rows, dims] cosines of the dims / 2 pairs, then their sines (null: no rotation)
  const int* positions;
  int dims, rows, interleaved;
};
// Element i of a rotated head (v: its value, `other`: its pair's other one).
__device__ __forceinline__ int rot_pair(const Rotation& r, int i) {
  const int half = r.dims / 2;
  return r.interleaved ? i ^ 1 : (i < half ? i + half : i - half);
}
__device__ __forceinline__ float rot_one(const Rotation& r, const float* cs, int i, float v, float other) {
  const int half = r.dims / 2, j = r.interleaved ? i >> 1 : (i < half ? i : i - half);
  const bool first = r.interleaved ? !(i & 1) : i < half;
  return first ? v * cs[j] - other * cs[half + j] : v * cs[j] + other * cs[half + j];
}

// Eight elements as they lie in memory.
template <typename T> struct Raw8 { uint4 v[sizeof(T) / 2]; };
template <typename T>
__device__ __forceinline__ Raw8<T> load_raw8(const T* p) {
  Raw8<T> r;
#pragma unroll
  for (int i = 0; i < int(sizeof(T) / 2); ++i) r.v[i] = reinterpret_cast<const uint4*>(p)[i];
  return r;
}

// One token per CTA.  A q or k head takes 2^lph lanes of 8 elements each; a thread keeps its place in the head over all the heads it
// serves, and with it the angles, and fetches several heads ahead.  Values are copied as one run of nv elements.
template <typename T>
__global__ void __launch_bounds__(256, sizeof(T) == 2 ? 4 : 2) qknorm_kvwrite_vec_kernel(T* __restrict__ qkv, const int* __restrict__ slots,
                                                                 const T* __restrict__ q_w, const T* __restrict__ k_w,
                                                                 T* __restrict__ k_cache, T* __restrict__ v_cache, int n_q, int n_k, int nv,
                                                                 int dk, int lph, float eps, long cache_slots, const Rotation rot) {
  __shared__ __align__(16) float s_rot[256 * 8];
  const int t = blockIdx.x, heads = n_q + n_k, step = blockDim.x >> lph;
  const int sub = threadIdx.x & ((1 << lph) - 1), c0 = sub * 8;
  T* row = qkv + size_t(t) * (size_t(heads) * dk + nv);
  const int slot = slots[t];
  const bool in = slot >= 0 && slot < cache_slots, mine = c0 < dk;
  // 0: no rotation here, 1: both elements of every pair in this lane, 2: the others' lane is half / 8 away, 3: through shared memory
  const int half = rot.dims / 2;
  const int turn = !rot.table ? 0 : rot.interleaved ? 1 : half % 8 == 0 ? 2 : 3;
  const bool first = c0 < half;
  constexpr int kAhead = 4;
  const int h_own = threadIdx.x >> lph;
  Raw8<T> raw[kAhead];
  auto fetch = [&](int h0) {
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      const int h = h0 + u * step + h_own;
      if (mine && h < heads) raw[u] = load_raw8(row + size_t(h) * dk + c0);
    }
  };
  fetch(0);
  float cs[8], sn[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) cs[e] = 1.f, sn[e] = 0.f;
  if (turn && mine && c0 < rot.dims) {
    const float* tab = rot.table + size_t(clamp_id(rot.positions[t], rot.rows)) * rot.dims;
    if (turn == 2) {
      load8(tab + (first ? c0 : c0 - half), cs);
      load8(tab + half + (first ? c0 : c0 - half), sn);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int i = c0 + e, j = rot.interleaved ? i >> 1 : (i < half ? i : i - half);
        if (i < rot.dims) cs[e] = tab[j], sn[e] = tab[half + j];
      }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e)                   // the element of a pair that comes first takes the other's sine off
      if (rot.interleaved ? !(e & 1) : c0 + e < half) sn[e] = -sn[e];
  }
  for (int c = threadIdx.x * 8; c < nv; c += blockDim.x * 8) {
    float f[8];
    load8(row + size_t(heads) * dk + c, f);
    if (in) store8(v_cache + size_t(slot) * nv + c, f);
  }
  for (int h0 = 0; h0 < heads; h0 += kAhead * step) {
    if (h0 > 0) fetch(h0);
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
    if (h0 + u * step >= heads) break;            // whole warps stay in step
    const int h = h0 + u * step + h_own;
    const bool active = mine && h < heads;
    float f[8] = {0, 0, 0, 0, 0, 0, 0, 0};
    if (active) load8(reinterpret_cast<const T*>(&raw[u]), f);
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
    for (int o = 1 << lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const T* w = h >= n_q ? k_w : q_w;
    if (w && active) {
      const float r = rsqrtf(ss / float(dk) + eps);
      float wf[8];
      load8(w + c0, wf);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = f[e] * r * wf[e];
    }
    if (turn) {
      float o[8];
      if (turn == 1) {
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = f[e ^ 1];
      } else if (turn == 2) {
        const int lane = threadIdx.x & 31, other = c0 >= rot.dims ? lane : first ? lane + half / 8 : lane - half / 8;
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = __shfl_sync(0xffffffffu, f[e], other);
      } else {
        float* mem = s_rot + (threadIdx.x - sub) * 8;
        __syncwarp();
        store8(mem + c0, f);
        __syncwarp();
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] = c0 + e < rot.dims ? mem[rot_pair(rot, c0 + e)] : 0.f;
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = fmaf(o[e], sn[e], f[e] * cs[e]);
    }
    if (!active) continue;
    if (h < n_q) store8(row + size_t(h) * dk + c0, f);
    else if (in) store8(k_cache + (size_t(slot) * n_k + (h - n_q)) * dk + c0, f);
    }
  }
}

// Any head dimension: one warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256) qknorm_kvwrite_any_kernel(T* __restrict__ qkv, const int* __restrict__ slots,
                                                                 const T* __restrict__ q_w, const T* __restrict__ k_w,
                                                                 T* __restrict__ k_cache, T* __restrict__ v_cache, int T_rows,
                                                                 int n_q, int n_k, int n_v, int dk, int dv, float eps, long cache_slots,
                                                                 const Rotation rot) {
  const int heads = n_q + n_k + n_v, lane = threadIdx.x & 31;
  const long item = (blockIdx.x * long(blockDim.x) + threadIdx.x) >> 5;
  if (item >= long(T_rows) * heads) return;
  const int t = int(item / heads), h = int(item % heads);
  const size_t row = size_t(t) * (size_t(n_q + n_k) * dk + size_t(n_v) * dv);
  const bool is_v = h >= n_q + n_k;
  const int dim = is_v ? dv : dk;
  T* src = qkv + row + (is_v ? size_t(n_q + n_k) * dk + size_t(h - n_q - n_k) * dv : size_t(h) * dk);
  const T* w = is_v ? nullptr : (h >= n_q ? k_w : q_w);
  float r = 1.f;
  if (w) {
    float ss = 0.f;
    for (int i = lane; i < dim; i += 32) ss += to_f32(src[i]) * to_f32(src[i]);
    r = rsqrtf(warp_sum(ss) / float(dim) + eps);
  }
  const int slot = slots[t];
  T* dst = src;
  if (h >= n_q) {
    if (slot < 0 || slot >= cache_slots) return;
    dst = is_v ? v_cache + (size_t(slot) * n_v + (h - n_q - n_k)) * dv : k_cache + (size_t(slot) * n_k + (h - n_q)) * dk;
  }
  auto value = [&](int i) { return w ? to_f32(src[i]) * r * to_f32(w[i]) : to_f32(src[i]); };
  const int turned = rot.table && !is_v ? rot.dims : 0;
  if (turned) {                                   // one lane per pair, so that q may be turned in place
    const float* cs = rot.table + size_t(clamp_id(rot.positions[t], rot.rows)) * rot.dims;
    const int half = turned / 2;
    for (int j = lane; j < half; j += 32) {
      const int a = rot.interleaved ? 2 * j : j, b = rot_pair(rot, a);
      const float u = value(a), v = value(b);
      from_f32(dst + a, rot_one(rot, cs, a, u, v));
      from_f32(dst + b, rot_one(rot, cs, b, v, u));
    }
  }
  for (int i = turned + lane; i < dim; i += 32) from_f32(dst + i, value(i));
}

template <typename T>
static int launch_qknorm(void* qkv, const void* slots, const void* q_w, const void* k_w, void* k_cache, void* v_cache, int rows, int n_q,
                         int n_k, int n_v, int dk, int dv, float eps, long cache_slots, const Rotation& rot, cudaStream_t st) {
  const long items = long(rows) * (n_q + n_k + n_v);
  if (dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && al16(qkv, k_cache, v_cache, q_w) && al16(k_w) && (!rot.table || rot.dims % 8 == 0)) {
    int lph = 0;
    while (8 << lph < dk) ++lph;
    const int lanes = (n_q + n_k) << lph;
    qknorm_kvwrite_vec_kernel<T><<<rows, lanes > 128 ? 256 : 128, 0, st>>>(
        static_cast<T*>(qkv), static_cast<const int*>(slots), static_cast<const T*>(q_w), static_cast<const T*>(k_w),
        static_cast<T*>(k_cache), static_cast<T*>(v_cache), n_q, n_k, n_v * dv, dk, lph, eps, cache_slots, rot);
  } else {
    qknorm_kvwrite_any_kernel<T><<<int((items + 7) / 8), 256, 0, st>>>(
        static_cast<T*>(qkv), static_cast<const int*>(slots), static_cast<const T*>(q_w), static_cast<const T*>(k_w),
        static_cast<T*>(k_cache), static_cast<T*>(v_cache), rows, n_q, n_k, n_v, dk, dv, eps, cache_slots, rot);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

// ---------------------------------------------------------------- q / k norm over the whole projection + cache write
// One row per CTA; rows hold q, k and v (and possibly more behind them) with pitch ld.  With a rotation the first rot.dims columns of
// every head of dk are turned.  With `mix` [n_q, n_q] q leaves as n_q rows of n_k * dk columns: row h, key head j holds
// sum over the query heads g of j of mix[h, g] q_g.
struct AllNorm {
  int n_q, n_k, dk, nv;
  long ld;
  float eps;
  long cache_slots;
  const float* mix;
};

// q of one token in shared memory (fp32) -> its rows for every query head.  A thread keeps four columns of the query heads of one key
// head in registers as pairs (GROUP heads) and makes every n-th row, where threads are left over.  `twice`: the matrix in shared
// memory, every element twice.
template <typename T, int GROUP>
__device__ __forceinline__ void mix_rows4(const float* q, const float* twice, T* __restrict__ out, int n_q, int n_k, int dk) {
  const int width = n_k * dk, chunks = width / 4;
  const int parts = chunks < int(blockDim.x) ? int(blockDim.x) / chunks : 1;
  const int part = parts > 1 ? int(threadIdx.x) / chunks : 0;
  if (part >= parts) return;
  for (int i = parts > 1 ? threadIdx.x % chunks : threadIdx.x; i < chunks; i += blockDim.x) {
    const int c = i * 4, j = c / dk;
    const float* src = q + size_t(j) * GROUP * dk + c % dk;
    ulonglong2 qv[GROUP];
#pragma unroll
    for (int g = 0; g < GROUP; ++g) qv[g] = *reinterpret_cast<const ulonglong2*>(src + g * dk);
    const uint64_t* row = reinterpret_cast<const uint64_t*>(twice) + j * GROUP;
#pragma unroll 2
    for (int h = part; h < n_q; h += parts) {
      const uint64_t* m = row + size_t(h) * n_q;
      uint64_t a0 = 0, a1 = 0;
#pragma unroll
      for (int g = 0; g < GROUP; g += 2) {
        ulonglong2 mm;
        if (GROUP % 2 == 0) {
          mm = *reinterpret_cast<const ulonglong2*>(m + g);      // n_q and j * GROUP are even
        } else {
          mm.x = m[g];
          mm.y = 0;
        }
        a0 = fma2(mm.x, qv[g].x, a0);
        a1 = fma2(mm.x, qv[g].y, a1);
        if (GROUP % 2 == 0) {
          a0 = fma2(mm.y, qv[GROUP > 1 ? g + 1 : 0].x, a0);
          a1 = fma2(mm.y, qv[GROUP > 1 ? g + 1 : 0].y, a1);
        }
      }
      const float2 x = unpack2(a0), y = unpack2(a1);
      T* dst = out + size_t(h) * width + c;
      if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(x.x, x.y), pack_bf16x2(y.x, y.y));
      else *reinterpret_cast<float4*>(dst) = make_float4(x.x, x.y, y.x, y.y);
    }
  }
}
// The same for any sizes, an element at a time; element (h, g) of the matrix at mix[(h * n_q + g) * step].
template <typename T>
__device__ __forceinline__ void mix_rows_any(const float* q, const float* mix, int step, T* __restrict__ out, int n_q, int n_k, int dk) {
  const int width = n_k * dk, group = n_q / n_k;
  for (int i = threadIdx.x; i < n_q * width; i += blockDim.x) {
    const int h = i / width, c = i % width, j = c / dk;
    const float *src = q + size_t(j) * group * dk + c % dk, *m = mix + (size_t(h) * n_q + j * group) * step;
    float a = 0.f;
    for (int g = 0; g < group; ++g) a = fmaf(m[g * step], src[g * dk], a);
    from_f32(out + i, a);
  }
}

template <typename T, int V, bool MIX, bool TURN>
__global__ void __launch_bounds__(256, MIX ? 4 : 1) qknorm_all_kernel(T* __restrict__ qkv, const int* __restrict__ slots, const T* __restrict__ q_w,
                                                         const T* __restrict__ k_w, T* __restrict__ k_cache, T* __restrict__ v_cache,
                                                         T* __restrict__ wide, const AllNorm a, const Rotation rot, int mix_smem) {
  extern __shared__ __align__(16) float s_row[];       // MIX or rotation: normed q and k of the row; MIX: then the mixing matrix
  __shared__ float red_q[8], red_k[8];
  const int t = blockIdx.x, nq = a.n_q * a.dk, nk = a.n_k * a.dk, nv = a.nv;
  T* row = qkv + size_t(t) * a.ld;
  auto load = [](const T* p, float (&f)[V]) {
    if constexpr (V == 8) load8(p, f); else f[0] = to_f32(*p);
  };
  auto store = [](T* p, const float (&f)[V]) {
    if constexpr (V == 8) store8(p, f); else from_f32(p, f[0]);
  };
  float sq = 0.f, sk = 0.f, f[V], w[V];
  for (int c = threadIdx.x * V; c < nq + nk; c += blockDim.x * V) {
    load(row + c, f);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s += f[e] * f[e];
    if (c < nq) sq += s; else sk += s;
  }
  const float rq = rsqrtf(block_sum(sq, red_q) / float(nq) + a.eps), rk = rsqrtf(block_sum(sk, red_k) / float(nk) + a.eps);
  const int slot = slots[t];
  const bool in = slot >= 0 && slot < a.cache_slots;
  constexpr bool turned = TURN;
  const bool direct = V == 8 && turned && !rot.interleaved && rot.dims % 16 == 0 && a.dk % 8 == 0 && !(reinterpret_cast<uintptr_t>(rot.table) & 15);
  for (int c = threadIdx.x * V; c < nq + nk + nv; c += blockDim.x * V) {
    load(row + c, f);
    if (c < nq + nk) {
      const float r = c < nq ? rq : rk;
      load(c < nq ? q_w + c : k_w + (c - nq), w);
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] = f[e] * r * w[e];
      if constexpr (V == 8 && TURN) {
        const int at = c % a.dk;
        if (direct && at < rot.dims) {                     // turned here: the other elements of the eight pairs lie half away
          const int half = rot.dims / 2, away = at < half ? half : -half, j = at < half ? at : at - half;
          const float* tab = rot.table + size_t(clamp_id(rot.positions[t], rot.rows)) * rot.dims;
          float g[8], wg[8], cs[8], sn[8];
          load8(row + c + away, g);
          load8((c < nq ? q_w + c : k_w + (c - nq)) + away, wg);
          load8(tab + j, cs);
          load8(tab + half + j, sn);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = fmaf(at < half ? -sn[e] : sn[e], g[e] * r * wg[e], f[e] * cs[e]);
        }
      }
      if ((turned && !MIX) || (MIX && c < nq) || (turned && !direct)) {
        if constexpr (V == 8) store8(s_row + c, f); else s_row[c] = f[0];
      } else if (c < nq) {
        store(row + c, f);
      } else if (in) {
        store(k_cache + size_t(slot) * nk + (c - nq), f);
      }
    } else if (in) {
      store(v_cache + size_t(slot) * nv + (c - nq - nk), f);
    }
  }
  if (!turned && !MIX) return;
  float* s_mix = s_row + (nq + nk + 3) / 4 * 4;
  if (MIX && mix_smem)
    for (int i = threadIdx.x; i < a.n_q * a.n_q; i += blockDim.x) reinterpret_cast<float2*>(s_mix)[i] = make_float2(a.mix[i], a.mix[i]);
  __syncthreads();
  if (turned && !direct) {
    const float* cs = rot.table + size_t(clamp_id(rot.positions[t], rot.rows)) * rot.dims;
    const int half = rot.dims / 2;
    for (int i = threadIdx.x; i < (a.n_q + a.n_k) * half; i += blockDim.x) {
      const int j = i % half, x = rot.interleaved ? 2 * j : j, y = rot_pair(rot, x);
      float* head = s_row + i / half * a.dk;
      const float u = head[x], v = head[y];
      head[x] = rot_one(rot, cs, x, u, v);
      head[y] = rot_one(rot, cs, y, v, u);
    }
    __syncthreads();
  }
  if (turned && (!MIX || !direct)) {
    for (int c = (MIX ? nq : 0) + threadIdx.x * V; c < nq + nk; c += blockDim.x * V) {
#pragma unroll
      for (int e = 0; e < V; ++e) f[e] = s_row[c + e];
      if (c < nq) store(row + c, f);
      else if (in) store(k_cache + size_t(slot) * nk + (c - nq), f);
    }
  }
  if constexpr (MIX) {
    T* out = wide + size_t(t) * a.n_q * nk;
    if constexpr (V == 8) {
      if (mix_smem) {
        switch (a.n_q / a.n_k) {
          case 1: mix_rows4<T, 1>(s_row, s_mix, out, a.n_q, a.n_k, a.dk); return;
          case 2: mix_rows4<T, 2>(s_row, s_mix, out, a.n_q, a.n_k, a.dk); return;
          case 4: mix_rows4<T, 4>(s_row, s_mix, out, a.n_q, a.n_k, a.dk); return;
          case 8: mix_rows4<T, 8>(s_row, s_mix, out, a.n_q, a.n_k, a.dk); return;
        }
      }
    }
    mix_rows_any(s_row, mix_smem ? s_mix : a.mix, mix_smem ? 2 : 1, out, a.n_q, a.n_k, a.dk);
  }
}
template <typename T>
static int launch_qknorm_all(void* qkv, const void* slots, const void* q_w, const void* k_w, void* k_cache, void* v_cache, void* wide, int rows,
                             const AllNorm& a, const Rotation& rot, cudaStream_t st) {
  T *x = static_cast<T*>(qkv), *kc = static_cast<T*>(k_cache), *vc = static_cast<T*>(v_cache), *o = static_cast<T*>(wide);
  const T *qw = static_cast<const T*>(q_w), *kw = static_cast<const T*>(k_w);
  const int* s = static_cast<const int*>(slots);
  const int nq = a.n_q * a.dk, nk = a.n_k * a.dk;
  const bool vec = nq % 8 == 0 && nk % 8 == 0 && a.nv % 8 == 0 && a.ld % 8 == 0 && al16(qkv, q_w, k_w, k_cache) && al16(v_cache) &&
                   (!a.mix || (a.dk % 8 == 0 && al16(wide)));
  constexpr size_t kMost = 160 * 1024;
  size_t smem = a.mix || rot.table ? size_t(nq + nk + 3) / 4 * 16 : 0;
  const int mix_smem = a.mix && smem + size_t(a.n_q) * a.n_q * 8 <= kMost;
  if (mix_smem) smem += size_t(a.n_q) * a.n_q * 8;
  if (smem > kMost) return -2;
#define XL_ALL(V, MIX, TURN)                                                                                                           \
  do {                                                                                                                                 \
    static bool set = false;                                                                                                           \
    if (!set) { cudaFuncSetAttribute(qknorm_all_kernel<T, V, MIX, TURN>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(kMost)); set = true; } \
    qknorm_all_kernel<T, V, MIX, TURN><<<rows, 256, smem, st>>>(x, s, qw, kw, kc, vc, o, a, rot, mix_smem);                            \
  } while (0)
#define XL_ALL_TURN(V, MIX) do { if (rot.table) XL_ALL(V, MIX, true); else XL_ALL(V, MIX, false); } while (0)
  if (a.mix) { if (vec) XL_ALL_TURN(8, true); else XL_ALL_TURN(1, true); }
  else { if (vec) XL_ALL_TURN(8, false); else XL_ALL_TURN(1, false); }
#undef XL_ALL_TURN
#undef XL_ALL
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

// ---------------------------------------------------------------- latent attention: norms, rotation and cache write of one row per CTA
template <typename T, int V>
__global__ void __launch_bounds__(256) latent_down_kernel(const T* __restrict__ low, const T* __restrict__ q_w, const T* __restrict__ kv_w,
                                                          T* __restrict__ c_q, T* __restrict__ cache, const int* __restrict__ slots, int nq,
                                                          int nc, long ld, float eps, long cache_slots, const Rotation rot) {
  __shared__ float red_q[8], red_k[8];
  const int t = blockIdx.x;
  const T* row = low + size_t(t) * ld;
  auto load = [](const T* p, float (&f)[V]) {
    if constexpr (V == 8) load8(p, f); else f[0] = to_f32(*p);
  };
  auto store = [](T* p, const float (&f)[V]) {
    if constexpr (V == 8) store8(p, f); else from_f32(p, f[0]);
  };
  float sq = 0.f, sk = 0.f, f[V], w[V];
  for (int c = threadIdx.x * V; c < nq + nc; c += blockDim.x * V) {
    load(row + c, f);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s += f[e] * f[e];
    if (c < nq) sq += s; else sk += s;
  }
  const float rq = rsqrtf(block_sum(sq, red_q) / float(nq) + eps), rk = rsqrtf(block_sum(sk, red_k) / float(nc) + eps);
  const int slot = slots[t];
  const bool in = slot >= 0 && slot < cache_slots;
  T* dst = cache + (in ? size_t(slot) : 0) * (nc + rot.dims);
  for (int c = threadIdx.x * V; c < nq + nc; c += blockDim.x * V) {
    load(row + c, f);
    load(c < nq ? q_w + c : kv_w + (c - nq), w);
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] = f[e] * (c < nq ? rq : rk) * w[e];
    if (c < nq) store(c_q + size_t(t) * nq + c, f);
    else if (in) store(dst + (c - nq), f);
  }
  const float* cs = rot.table + size_t(clamp_id(rot.positions[t], rot.rows)) * rot.dims;
  const T* key = row + nq + nc;
  if (in)
    for (int i = threadIdx.x; i < rot.dims; i += blockDim.x)
      from_f32(dst + nc + i, rot_one(rot, cs, i, to_f32(key[i]), to_f32(key[rot_pair(rot, i)])));
}

// One pair per thread; x and out may be one and the same.
template <typename T>
__global__ void __launch_bounds__(256) rotate_kernel(const T* __restrict__ x, T* __restrict__ out, long total, int heads, long x_row,
                                                     long x_head, long out_row, long out_head, const Rotation rot) {
  const int half = rot.dims / 2;
  for (long idx = blockIdx.x * long(blockDim.x) + threadIdx.x; idx < total; idx += long(gridDim.x) * blockDim.x) {
    const long item = idx / half, t = item / heads, h = item % heads;
    const int j = int(idx % half), a = rot.interleaved ? 2 * j : j, b = rot_pair(rot, a);
    const T* src = x + t * x_row + h * x_head;
    T* dst = out + t * out_row + h * out_head;
    const float* cs = rot.table + size_t(clamp_id(rot.positions[t], rot.rows)) * rot.dims;
    const float u = to_f32(src[a]), v = to_f32(src[b]);
    from_f32(dst + a, rot_one(rot, cs, a, u, v));
    from_f32(dst + b, rot_one(rot, cs, b, v, u));
  }
}

// ---------------------------------------------------------------- out = o * sigmoid(gate) * scale, strided rows
template <typename T, int V>
__global__ void __launch_bounds__(256) sigmoid_gate_kernel(const T* __restrict__ o, const T* __restrict__ gate, T* __restrict__ out,
                                                           long total, int n, long ldg, long ldo, float scale) {
  const int per = n / V;
  for (long idx = blockIdx.x * long(blockDim.x) + threadIdx.x; idx < total; idx += long(gridDim.x) * blockDim.x) {
    const long t = idx / per;
    const int c = int(idx % per) * V;
    if constexpr (V == 8) {
      float a[8], g[8];
      load8(o + t * n + c, a);
      load8(gate + t * ldg + c, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) a[e] = a[e] * scale / (1.f + __expf(-g[e]));
      store8(out + t * ldo + c, a);
    } else {
      from_f32(out + t * ldo + c, to_f32(o[t * n + c]) * scale / (1.f + __expf(-to_f32(gate[t * ldg + c]))));
    }
  }
}

// ---------------------------------------------------------------- rows [x, x0], x0 = table[token] * scale; in bf16 the fp32 x
// as its rounded value and the rest
template <typename T>
__global__ void __launch_bounds__(256) split_rows_kernel(const float* __restrict__ x, const int* __restrict__ tokens,
                                                         const T* __restrict__ table, float scale, T* __restrict__ out, int W, int V) {
  const size_t t = blockIdx.x;
  constexpr int parts = sizeof(T) == 2 ? 2 : 1;
  T* dst = out + t * (parts + 1) * W;
  const T* x0 = table + size_t(clamp_id(tokens[t], V)) * W;
  for (int c = threadIdx.x; c < W; c += blockDim.x) {
    const float v = x[t * W + c];
    from_f32(dst + c, v);
    if constexpr (parts == 2) from_f32(dst + W + c, v - to_f32(dst[c]));
    from_f32(dst + parts * W + c, to_f32(x0[c]) * scale);
  }
}

// ---------------------------------------------------------------- gated activation: out[t, i] = act(x[t, i]) * x[t, I + i]
template <typename T>
__global__ void gated_act_kernel(const T* __restrict__ x, T* __restrict__ out, long total, int I, int act, float limit) {
  for (long idx = blockIdx.x * long(blockDim.x) + threadIdx.x; idx < total; idx += long(gridDim.x) * blockDim.x) {
    const long t = idx / I;
    const int i = int(idx % I);
    const T* row = x + t * 2 * I;
    from_f32(out + idx, gated(to_f32(row[i]), to_f32(row[I + i]), act, limit));
  }
}
template <typename T>
__global__ void gated_act_vec_kernel(const T* __restrict__ x, T* __restrict__ out, long total, int nvec, int act, float limit) {
  for (long idx = blockIdx.x * long(blockDim.x) + threadIdx.x; idx < total; idx += long(gridDim.x) * blockDim.x) {
    const long t = idx / nvec;
    const int v = int(idx % nvec);
    const T* row = x + t * 16 * nvec;
    float g[8], u[8];
    load8(row + v * 8, g);
    load8(row + (nvec + v) * 8, u);
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = gated(g[e], u[e], act, limit);
    store8(out + idx * 8, g);
  }
}
template <typename T>
static int launch_gated_act(const void* x, void* out, int rows, int I, int act, float limit, cudaStream_t st) {
  const bool vec = I % 8 == 0 && al16(x, out);
  const long total = long(rows) * (vec ? I / 8 : I);
  long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (vec) gated_act_vec_kernel<T><<<int(blocks), 256, 0, st>>>(static_cast<const T*>(x), static_cast<T*>(out), total, I / 8, act, limit);
  else gated_act_kernel<T><<<int(blocks), 256, 0, st>>>(static_cast<const T*>(x), static_cast<T*>(out), total, I, act, limit);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

}  // namespace xl_sn

using namespace xl_sn;

// `f32` in the entry points below: 1 when the model's tensors are fp32, 0 for bf16 (the residual x is fp32 either way).

// Rows of an embedding: table[tokens[t]] * scale + pos_table[positions[t]] (pos_table null: none).
struct LeadRows {
  const void *tokens, *table, *positions, *pos_table;
  int V, pos_rows;
  float scale;
};
template <typename T>
static void set_lead(NormParams<T>& p, const LeadRows& l) {
  p.tokens = static_cast<const int*>(l.tokens);
  p.table = static_cast<const T*>(l.table);
  p.positions = static_cast<const int*>(l.positions);
  p.pos_table = static_cast<const T*>(l.pos_table);
  p.V = l.V;
  p.pos_rows = l.pos_rows;
  p.scale = p.lead_scale = l.scale;
}

// x[t] = table[tokens[t]] * scale (+ pos_table[positions[t]]), with w_rows its rms times w_rows, or with keep_x: x[t] += it;
// h = rms(x) * (w_next + w_off)
XL_API int xl_embed_rms_norm(const void* tokens, const void* table, float scale, const void* positions, const void* pos_table, int pos_rows,
                             const void* w_rows, int keep_x, void* x, const void* w_next, float w_off, void* h, int rows, int H, int V, float eps, int f32,
                             void* stream) {
  if (w_rows && keep_x) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool al = al16(table, x, w_next, h) && al16(pos_table, w_rows);
  const LeadRows l{tokens, table, positions, pos_table, V, pos_rows, scale};
  auto go = [&](auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    auto p = base_params<E>(x, w_rows, w_next, h, H, eps);
    set_lead(p, l);
    p.w_off = w_off;
    p.keep_x = keep_x;
    return launch_norm<E, SRC_EMBED>(p, rows, al, st);
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// x += rms(y) * w_post;  h = rms(x) * w_next
XL_API int xl_post_norm_add_norm(const void* y, void* x, const void* w_post, const void* w_next, void* h, int rows, int H, float eps,
                                 int f32, void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool al = al16(y, x, w_post, w_next) && al16(h);
  if (f32) {
    auto p = base_params<float>(x, w_post, w_next, h, H, eps);
    p.y = static_cast<const float*>(y);
    return launch_norm<float, SRC_ROWS>(p, rows, al, st);
  }
  auto p = base_params<__nv_bfloat16>(x, w_post, w_next, h, H, eps);
  p.y = static_cast<const __nv_bfloat16*>(y);
  return launch_norm<__nv_bfloat16, SRC_ROWS>(p, rows, al, st);
}

// y = scale * (rms(ya) * w_a + rms(yb) * w_b);  x += rms(y) * w_post;  h = rms(x) * w_next
XL_API int xl_branches_post_norm_add_norm(const void* ya, const void* yb, const void* w_a, const void* w_b, float scale, void* x,
                                          const void* w_post, const void* w_next, void* h, int rows, int H, float eps, int f32, void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool al = al16(ya, yb, w_a, w_b) && al16(x, w_post, w_next, h);
  auto go = [&](auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    auto p = base_params<E>(x, w_post, w_next, h, H, eps);
    p.y = static_cast<const E*>(ya);
    p.y2 = static_cast<const E*>(yb);
    p.w_y = static_cast<const E*>(w_a);
    p.w_y2 = static_cast<const E*>(w_b);
    p.scale = scale;
    return launch_norm<E, SRC_PAIR>(p, rows, al, st);
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// x += mult * y, or ls * y element by element (ls [H], null: mult);  with `table`: x += table[tokens[t]] * lead_scale
// (+ pos_table[positions[t]]);  h = rms(x) * (w_next + w_off)
XL_API int xl_add_norm(const void* y, void* x, float mult, const void* ls, const void* w_next, float w_off, void* h, int rows, int H, float eps,
                       const void* tokens, const void* table, int V, float lead_scale, const void* positions, const void* pos_table,
                       int pos_rows, int f32, void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool al = al16(y, x, w_next, h) && al16(ls, table, pos_table);
  auto go = [&](auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    auto p = base_params<E>(x, nullptr, w_next, h, H, eps);
    if (table) set_lead(p, LeadRows{tokens, table, positions, pos_table, V, pos_rows, lead_scale});
    p.lead = table != nullptr;
    p.y = static_cast<const E*>(y);
    p.scale = mult;
    p.ls = static_cast<const E*>(ls);
    p.w_off = w_off;
    return launch_norm<E, SRC_ADD>(p, rows, al, st);
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// The same with y[t] = sum_j weights[t, j] * y_exp[dst_of[t, j]] (k choices, dst_of < 0: none); ls is required.
XL_API int xl_moe_combine_add_norm(const void* y_exp, const void* dst_of, const void* weights, int k, void* x, const void* ls,
                                   const void* w_next, float w_off, void* h, int rows, int H, float eps, const void* tokens, const void* table,
                                   int V, float lead_scale, const void* positions, const void* pos_table, int pos_rows, int f32, void* stream) {
  if (!ls) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool al = al16(y_exp, x, w_next, h) && al16(ls, table, pos_table);
  auto go = [&](auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    auto p = base_params<E>(x, nullptr, w_next, h, H, eps);
    if (table) set_lead(p, LeadRows{tokens, table, positions, pos_table, V, pos_rows, lead_scale});
    p.lead = table != nullptr;
    p.y_exp = static_cast<const E*>(y_exp);
    p.dst_of = static_cast<const int*>(dst_of);
    p.ids = p.dst_of;                        // any array of k entries: nothing reaches first_identity
    p.first_identity = 0x7fffffff;
    p.weights = static_cast<const float*>(weights);
    p.k = k;
    p.ls = static_cast<const E*>(ls);
    p.w_off = w_off;
    p.add_only = 1;
    return launch_norm<E, SRC_MOE>(p, rows, al, st);
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// x = y + vec (y [rows, H], vec [H] fp32);  h = rms(x) * w_next
XL_API int xl_replace_norm(const void* y, const void* vec, void* x, const void* w_next, void* h, int rows, int H, float eps, int f32,
                           void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool al = al16(y, x, w_next, h) && al16(vec);
  if (f32) {
    auto p = base_params<float>(x, nullptr, w_next, h, H, eps);
    p.y32 = static_cast<const float*>(y); p.vec = static_cast<const float*>(vec);
    return launch_norm<float, SRC_SET>(p, rows, al, st);
  }
  auto p = base_params<__nv_bfloat16>(x, nullptr, w_next, h, H, eps);
  p.y32 = static_cast<const float*>(y); p.vec = static_cast<const float*>(vec);
  return launch_norm<__nv_bfloat16, SRC_SET>(p, rows, al, st);
}

// out [rows, 2 W] = [x, x0] (fp32), or [rows, 3 W] = [bf16(x), bf16(x - bf16(x)), x0], x0 = table[token] * scale
XL_API int xl_split_rows(const void* x, const void* tokens, const void* table, float scale, void* out, int rows, int W, int V, int f32,
                         void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const float* xx = static_cast<const float*>(x);
  const int* tk = static_cast<const int*>(tokens);
  if (f32)
    split_rows_kernel<float><<<rows, 256, 0, st>>>(xx, tk, static_cast<const float*>(table), scale, static_cast<float*>(out), W, V);
  else
    split_rows_kernel<__nv_bfloat16><<<rows, 256, 0, st>>>(xx, tk, static_cast<const __nv_bfloat16*>(table), scale,
                                                          static_cast<__nv_bfloat16*>(out), W, V);
  return cudaGetLastError() == cudaSuccess ? 0 : -1;
}

// RMSNorm over the n_q * dk query and over the n_k * dk key columns of rows with pitch ld, then the rotation (null table: none); q in
// place, or with `mix` to wide [rows, n_q, n_k * dk] (see qknorm_all_kernel); k and v to the cache slots [cache_slots, nk | nv].
XL_API int xl_qknorm_all_kvwrite(void* qkv, const void* slots, const void* q_w, const void* k_w, void* k_cache, void* v_cache, int rows,
                                 int n_q, int n_k, int dk, int nv, long ld, float eps, long cache_slots, const void* rot_table,
                                 const void* positions, int rot_dims, int rot_rows, int interleaved, const void* mix, void* wide, int f32,
                                 void* stream) {
  if (rows <= 0) return 0;
  if (rot_table && (rot_dims > dk || rot_dims % 2 || rot_rows < 1)) return -2;
  if (mix && (!wide || n_q % n_k)) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const Rotation rot{static_cast<const float*>(rot_table), static_cast<const int*>(positions), rot_dims, rot_rows, interleaved};
  const AllNorm a{n_q, n_k, dk, nv, ld, eps, cache_slots, static_cast<const float*>(mix)};
  if (f32) return launch_qknorm_all<float>(qkv, slots, q_w, k_w, k_cache, v_cache, wide, rows, a, rot, st);
  return launch_qknorm_all<__nv_bfloat16>(qkv, slots, q_w, k_w, k_cache, v_cache, wide, rows, a, rot, st);
}

// out [rows, n] (pitch ldo) = o (dense) * sigmoid(gate, pitch ldg) * scale
XL_API int xl_sigmoid_gate(const void* o, const void* gate, void* out, int rows, int n, long ldg, long ldo, float scale, int f32,
                           void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = n % 8 == 0 && ldg % 8 == 0 && ldo % 8 == 0 && al16(o, gate, out);
  const long total = long(rows) * (vec ? n / 8 : n);
  long blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  auto go = [&](auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    const E *a = static_cast<const E*>(o), *g = static_cast<const E*>(gate);
    if (vec) sigmoid_gate_kernel<E, 8><<<int(blocks), 256, 0, st>>>(a, g, static_cast<E*>(out), total, n, ldg, ldo, scale);
    else sigmoid_gate_kernel<E, 1><<<int(blocks), 256, 0, st>>>(a, g, static_cast<E*>(out), total, n, ldg, ldo, scale);
    return cudaGetLastError() == cudaSuccess ? 0 : -1;
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// y[t] = sum_j weights[t, j] * expert output (an expert's row of y_exp, or h_in[t] for ids >= first_identity) + shared[t];
// then as above.
XL_API int xl_moe_combine_post_norm_add_norm(const void* y_exp, const void* dst_of, const void* ids, const void* weights,
                                             const void* h_in, const void* shared, int k, int first_identity, void* x,
                                             const void* w_post, const void* w_next, void* h, int rows, int H, float eps, int f32,
                                             void* stream) {
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool al = al16(y_exp, x, w_post, w_next) && al16(h, h_in, shared);
  auto fill = [&](auto& p, auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    p.y_exp = static_cast<const E*>(y_exp);
    p.dst_of = static_cast<const int*>(dst_of);
    p.ids = static_cast<const int*>(ids);
    p.weights = static_cast<const float*>(weights);
    p.h_in = static_cast<const E*>(h_in);
    p.shared = static_cast<const E*>(shared);
    p.k = k;
    p.first_identity = first_identity;
  };
  if (f32) {
    auto p = base_params<float>(x, w_post, w_next, h, H, eps);
    fill(p, static_cast<float*>(nullptr));
    return launch_norm<float, SRC_MOE>(p, rows, al, st);
  }
  auto p = base_params<__nv_bfloat16>(x, w_post, w_next, h, H, eps);
  fill(p, static_cast<__nv_bfloat16*>(nullptr));
  return launch_norm<__nv_bfloat16, SRC_MOE>(p, rows, al, st);
}

// Per-head RMSNorm of q (in place) and k (null weight: none), then their first `rot_dims` dimensions turned by the angles of
// rot_table [rot_rows, rot_dims] (null: not) at `positions`; k and v to the cache slots [cache_slots, n_k, dk] and [.., n_v, dv].
XL_API int xl_qknorm_kvwrite(void* qkv, const void* slots, const void* q_w, const void* k_w, void* k_cache, void* v_cache, int rows,
                             int n_q, int n_k, int n_v, int dk, int dv, float eps, long cache_slots, const void* rot_table,
                             const void* positions, int rot_dims, int rot_rows, int interleaved, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (rot_table && (rot_dims > dk || rot_dims % 2 || rot_rows < 1)) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const Rotation rot{static_cast<const float*>(rot_table), static_cast<const int*>(positions), rot_dims, rot_rows, interleaved};
  if (f32) return launch_qknorm<float>(qkv, slots, q_w, k_w, k_cache, v_cache, rows, n_q, n_k, n_v, dk, dv, eps, cache_slots, rot, st);
  return launch_qknorm<__nv_bfloat16>(qkv, slots, q_w, k_w, k_cache, v_cache, rows, n_q, n_k, n_v, dk, dv, eps, cache_slots, rot, st);
}

// Latent attention behind its down projection: rows (pitch ld) of nq query-latent, nc key/value-latent and rot.dims key columns.
// Both latents are normed; the query latent goes to c_q [rows, nq], [latent | turned key part] to the cache.
XL_API int xl_latent_down(const void* low, const void* q_w, const void* kv_w, void* c_q, void* cache, const void* slots, int rows, int nq,
                          int nc, long ld, float eps, long cache_slots, const void* rot_table, const void* positions, int rot_dims,
                          int rot_rows, int interleaved, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (!rot_table || rot_dims < 2 || rot_dims % 2 || rot_rows < 1) return -2;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const Rotation rot{static_cast<const float*>(rot_table), static_cast<const int*>(positions), rot_dims, rot_rows, interleaved};
  const bool vec = nq % 8 == 0 && nc % 8 == 0 && rot_dims % 8 == 0 && ld % 8 == 0 && al16(low, q_w, kv_w, c_q) && al16(cache);
  auto go = [&](auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    const E *x = static_cast<const E*>(low), *qw = static_cast<const E*>(q_w), *kw = static_cast<const E*>(kv_w);
    const int* s = static_cast<const int*>(slots);
    const int threads = (nq + nc) / 8 > 128 ? 256 : 128;
    if (vec) latent_down_kernel<E, 8><<<rows, threads, 0, st>>>(x, qw, kw, static_cast<E*>(c_q), static_cast<E*>(cache), s, nq, nc, ld, eps, cache_slots, rot);
    else latent_down_kernel<E, 1><<<rows, 256, 0, st>>>(x, qw, kw, static_cast<E*>(c_q), static_cast<E*>(cache), s, nq, nc, ld, eps, cache_slots, rot);
    return cudaGetLastError() == cudaSuccess ? 0 : -1;
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// out[t, h] = x[t, h] turned (rot_dims columns each; element strides of rows and heads given).
XL_API int xl_rotate(const void* x, void* out, int rows, int heads, long x_row, long x_head, long out_row, long out_head,
                     const void* rot_table, const void* positions, int rot_dims, int rot_rows, int interleaved, int f32, void* stream) {
  if (rows <= 0 || heads <= 0) return 0;
  if (!rot_table || rot_dims < 2 || rot_dims % 2 || rot_rows < 1) return -2;
  const Rotation rot{static_cast<const float*>(rot_table), static_cast<const int*>(positions), rot_dims, rot_rows, interleaved};
  const long total = long(rows) * heads * (rot_dims / 2);
  long blocks = (total + 255) / 256;
  if (blocks > 148 * 32) blocks = 148 * 32;
  auto go = [&](auto* tag) {
    using E = std::remove_pointer_t<decltype(tag)>;
    rotate_kernel<E><<<int(blocks), 256, 0, static_cast<cudaStream_t>(stream)>>>(static_cast<const E*>(x), static_cast<E*>(out), total, heads,
                                                                                x_row, x_head, out_row, out_head, rot);
    return cudaGetLastError() == cudaSuccess ? 0 : -1;
  };
  return f32 ? go(static_cast<float*>(nullptr)) : go(static_cast<__nv_bfloat16*>(nullptr));
}

// x [rows, 2 I] = [gate | up] -> act(gate) * up; act: 0 silu, 1 tanh-gelu, 2 clamped gate with `limit`
XL_API int xl_gated_act(const void* x, void* out, int rows, int I, int act, float limit, int f32, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return f32 ? launch_gated_act<float>(x, out, rows, I, act, limit, st) : launch_gated_act<__nv_bfloat16>(x, out, rows, I, act, limit, st);
}
