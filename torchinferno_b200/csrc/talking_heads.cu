// Attention inside a sliding window whose softmax weights are mixed across the heads before they meet the values.
//
//   row_norm_append   q, k, v columns of the fused projection (+ bias): q and k divided by the root mean square of the whole
//                     projected row (all heads at once) and multiplied by a weight per element; q goes to q_out, k and v
//                     into their pages
//   attention         query i sees the tokens j with 0 <= i - j < window (j <= i);
//                       s_h(i, j)  = cap(q_h,i . k_(h / group),j * scale) + bias[h][min(i - j, span - 1)],
//                                    cap(s) = c tanh(s / c) (c = 0: none)
//                       w_h(i, .)  = softmax over the visible j
//                       m_h(i, j)  = sum_g talk[h][g] w_g(i, j)
//                       out_h(i)   = sigmoid(gate_h,i) * sum_j m_h(i, j) v_(h / group),j
//
// The mix needs every head's denominator before any weight can meet a value, so nothing streams through in one pass.
// Three forms, all with scores, softmax, mix and sums in fp32:
//
//   CUDA cores (32-bit, any head size and number of heads): a block owns a token with all its heads and walks the keys
//   twice, 32 at a time, aligned to absolute positions: first the maxima and denominators, then weights, mix and values.
//
//   Tensor cores, portions (bf16): three kernels over a scratch array of one 32-bit word per (token, head, visible key).
//   "scores" (per key head: 64 rows of tokens x query heads against tiles of 64 keys) leaves the capped and biased scores and
//   each row's log of the denominator; "mix" (per token) turns them into weights and multiplies by the heads' matrix,
//   leaving every mixed weight as two bf16 terms (high part and remainder: 16 bits) in the word the score lay in; "values"
//   (per key head) multiplies them with the values and applies the gate.  The caller runs the three over ranges of tokens
//   small enough for the scratch to stay in the L2.
//
//   Tensor cores, single tokens (bf16): two kernels over (part of the context, key head, request).  The first leaves scores
//   and each part's maxima and denominators; the second adds those up for all heads, mixes, multiplies with the part's
//   values in fp32 and, in the block that comes last for its request and key head, adds the parts in their order.
//
// Tiles of keys are aligned to absolute positions and walked in rising order, so a row's sums do not depend on how a prompt
// was cut, on what else the step holds or on the pages used (single tokens: the order of fp32 sums over parts only).
#include "mma.cuh"
#include <math_constants.h>

namespace tib {

struct ThCache {
  const void* keys; const void* values;      // first key / value of the layer's first page
  const int* block_table; int table_stride;
  int page_size; int64_t page_stride; int num_pages;
};

__device__ __forceinline__ int th_page(const ThCache& c, const int* table, int index, int* error_word, int code) {
  const int page = table[index / c.page_size];
  if (page >= 0 && page < c.num_pages) return page;
  if (error_word) atomicExch(error_word, code);
  return -1;
}

// ---------------------------------------------------------------------------------------------------- append
struct ThAppendArgs {
  int64_t ld; int q_off, k_off, v_off;
  const float* q_bias; const float* k_bias; const float* v_bias;     // or null
  const float* q_weight; const float* k_weight;                      // [heads * dim], [kv_heads * dim]; null: no norm
  float eps;
  const int* positions; const int* token_slot;
  int heads, kv_heads, dim, vdim;
  void* keys; void* values;
  ThCache cache;
  int* error_word;
};

template <typename T, int VEC> __device__ __forceinline__ void th_load(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = bf16x2_floats(b[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = to_f32(p[i]);
  }
}
template <typename T, int VEC> __device__ __forceinline__ void th_store(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    uint4 raw;
    __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) b[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = from_f32<T>(v[i]);
  }
}
template <int VEC> __device__ __forceinline__ void th_load_f32(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = p[i];
  }
}

constexpr int kThAppendThreads = 256;
constexpr int kThAppendKeep = 2;      // pieces of a row a thread holds between the two passes (the rest is read again)

// grid (tokens, 3): a block each for a token's q, k and v.  VEC 8: bf16, every width a multiple of 8 (a piece of eight never
// crosses a head's edge).
template <typename T, int VEC>
__global__ void __launch_bounds__(kThAppendThreads) th_append_kernel(const T* __restrict__ proj, T* __restrict__ q_out, ThAppendArgs a) {
  __shared__ float scratch[33];
  const int t = blockIdx.x, part = blockIdx.y;         // 0: q, 1: k, 2: v
  const float* bias = part == 0 ? a.q_bias : part == 1 ? a.k_bias : a.v_bias;
  const float* weight = part == 0 ? a.q_weight : part == 1 ? a.k_weight : nullptr;
  const int head_width = part == 2 ? a.vdim : a.dim, width = (part == 0 ? a.heads : a.kv_heads) * head_width;
  const T* src = proj + (size_t)t * a.ld + (part == 0 ? a.q_off : part == 1 ? a.k_off : a.v_off);
  pdl_wait();
  pdl_trigger();
  T* dst = q_out + (size_t)t * width;                  // (k and v: the token's row in the first head of its page)
  if (part > 0) {
    const int pos = a.positions[t];
    const int* table = a.cache.block_table + (size_t)a.token_slot[t] * a.cache.table_stride;
    const int page = th_page(a.cache, table, pos, threadIdx.x == 0 ? a.error_word : nullptr, 0x30000 + (t & 0xffff));
    if (page < 0) return;                              // (the whole block)
    dst = reinterpret_cast<T*>(part == 1 ? a.keys : a.values) + (size_t)page * a.cache.page_stride + (size_t)(pos % a.cache.page_size) * head_width;
  }
  float kept[kThAppendKeep][VEC], gain[kThAppendKeep][VEC];
  auto biased = [&](int e, float (&v)[VEC]) {
    th_load<T, VEC>(src + e, v);
    if (bias) {
      float b[VEC];
      th_load_f32<VEC>(bias + e, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] += b[i];
    }
  };
  auto leave = [&](int e, const float (&v)[VEC]) {
    if (part == 0) th_store<T, VEC>(dst + e, v);
    else {
      const int h = e / head_width;
      th_store<T, VEC>(dst + (size_t)h * a.cache.page_size * head_width + (e - h * head_width), v);
    }
  };
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < kThAppendKeep; ++n) {
    const int e = (n * kThAppendThreads + threadIdx.x) * VEC;
    if (e < width) {
      biased(e, kept[n]);
      if (weight) th_load_f32<VEC>(weight + e, gain[n]);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(kept[n][i], kept[n][i], ss);
    }
  }
  constexpr int FIRST = kThAppendKeep * kThAppendThreads * VEC;
  if (weight)
    for (int e = FIRST + threadIdx.x * VEC; e < width; e += kThAppendThreads * VEC) {
      float v[VEC];
      biased(e, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
    }
  const float inv = weight ? 1.f / sqrtf(block_sum(ss, scratch) / (float)width + a.eps) : 1.f;
#pragma unroll
  for (int n = 0; n < kThAppendKeep; ++n) {
    const int e = (n * kThAppendThreads + threadIdx.x) * VEC;
    if (e < width) {
      if (weight) {
#pragma unroll
        for (int i = 0; i < VEC; ++i) kept[n][i] = kept[n][i] * inv * gain[n][i];
      }
      leave(e, kept[n]);
    }
  }
  for (int e = FIRST + threadIdx.x * VEC; e < width; e += kThAppendThreads * VEC) {
    float v[VEC];
    biased(e, v);
    if (weight) {
      float g[VEC];
      th_load_f32<VEC>(weight + e, g);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * g[i];
    }
    leave(e, v);
  }
}

// ------------------------------------------------------------------------------------------------- attention
constexpr float kThLog2e = 1.4426950408889634f;

struct ThArgs {
  const int* q_start; const int* kv_start; const int* slots; const int* positions;
  int heads, kv_heads, dim, vdim, window;
  float scale, cap;
  const float* bias; int span;                            // [heads][span] or null
  const float* talk;                                      // [heads][heads]
  const __nv_bfloat16* talk_hi; const __nv_bfloat16* talk_lo;    // [padded][padded] (multiples of 16, zeros outside); lo may be null
  const void* gate; int gate_dtype; int64_t ld_gate;      // [tokens, heads * vdim] logits or null
  ThCache cache;
  int* error_word;
  int first_token, last_token;                            // portions: the step's tokens first .. last - 1 are done in this call
  float* scores; float* lse; int key_span;                // scratch: [token][head][key_span] words, [token][head]
  int group_chunk, q_tile;
  float* part_ml; float* part_o; int* counters; int tiles_per_part, n_parts;    // single tokens
};

__device__ __forceinline__ float th_gate(const ThArgs& a, size_t token, int col) {
  const float g = a.gate_dtype == TIB_F32 ? reinterpret_cast<const float*>(a.gate)[token * a.ld_gate + col]
                                          : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(a.gate)[token * a.ld_gate + col]);
  return 1.f / (1.f + expf(-g));
}

// first visible position, and the tile edge (a multiple of 64) a token's words are counted from
__device__ __forceinline__ int th_first(int pos, int window) { return max(0, pos - window + 1); }
__device__ __forceinline__ int th_base(int pos, int window) { return th_first(pos, window) & ~63; }

// ------------------------------------------------------------ CUDA cores
constexpr int kThSimtThreads = 128;

template <typename T>
__global__ void __launch_bounds__(kThSimtThreads) th_simt_kernel(const T* __restrict__ q, T* __restrict__ out, ThArgs a) {
  pdl_wait();
  pdl_trigger();
  extern __shared__ float sm[];
  const int H = a.heads, d = a.dim, dv = a.vdim, group = H / a.kv_heads;
  float* q_s = sm;                        // [H][d]
  float* acc = q_s + H * d;               // [H][dv]
  float* w_s = acc + H * dv;              // [H][33] weights of 32 keys
  float* m_s = w_s + H * 33;              // [H][33] mixed weights
  float* top_s = m_s + H * 33;            // [H] maxima
  float* inv_s = top_s + H;               // [H] 1 / denominators
  long long* at_s = reinterpret_cast<long long*>(inv_s + H + ((H * (d + dv + 68)) & 1));       // [32] page base of a key, or -1
  int* row_s = reinterpret_cast<int*>(at_s + 32);                                              // [32] row in its page
  const int entry = blockIdx.y;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  const int t = blockIdx.x;
  if (t >= len) return;
  const size_t token = (size_t)(row0 + t);
  const int pos = a.kv_start[entry] + t, lo = th_first(pos, a.window);
  const int* table = a.cache.block_table + (size_t)a.slots[entry] * a.cache.table_stride;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int WARPS = kThSimtThreads / 32;
  for (int e = threadIdx.x; e < H * d; e += kThSimtThreads) q_s[e] = to_f32(q[token * H * d + e]);
  for (int e = threadIdx.x; e < H * dv; e += kThSimtThreads) acc[e] = 0.f;
  const T* keys = reinterpret_cast<const T*>(a.cache.keys);
  const T* values = reinterpret_cast<const T*>(a.cache.values);

  auto locate = [&](int base) {           // where the 32 keys from `base` on live
    __syncthreads();                      // (what the block before read is no longer needed; q_s and acc are written)
    if (threadIdx.x < 32) {
      const int idx = base + threadIdx.x;
      long long at = -1;
      int row = 0;
      if (idx >= lo && idx <= pos) {
        const int page = th_page(a.cache, table, idx, a.error_word, 0x10000 + entry);
        if (page >= 0) {
          at = (long long)page * a.cache.page_stride;
          row = idx % a.cache.page_size;
        }
      }
      at_s[threadIdx.x] = at;
      row_s[threadIdx.x] = row;
    }
    __syncthreads();
  };
  auto score = [&](int h, int base) {     // of key base + lane; minus infinity where it is not seen
    if (at_s[lane] < 0) return -CUDART_INF_F;
    const T* kr = keys + at_s[lane] + ((size_t)(h / group) * a.cache.page_size + row_s[lane]) * d;
    const float* qr = q_s + h * d;
    float s = 0.f;
    for (int i = 0; i < d; ++i) s = fmaf(qr[i], to_f32(kr[i]), s);
    s *= a.scale;
    if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
    if (a.bias) s += a.bias[(size_t)h * a.span + min(pos - base - lane, a.span - 1)];
    return s;
  };

  const int block_lo = lo / 32, block_hi = pos / 32;
  for (int h = warp; h < H; h += WARPS)
    if (lane == 0) { top_s[h] = -CUDART_INF_F; inv_s[h] = 0.f; }
  for (int b = block_lo; b <= block_hi; ++b) {
    locate(b * 32);
    for (int h = warp; h < H; h += WARPS) {
      const float s = score(h, b * 32);
      const float top = top_s[h], high = fmaxf(top, warp_max(s));
      if (high == -CUDART_INF_F) continue;
      const float sum = warp_sum(s == -CUDART_INF_F ? 0.f : expf(s - high));
      __syncwarp();
      if (lane == 0) {
        inv_s[h] = (top == -CUDART_INF_F ? 0.f : inv_s[h] * expf(top - high)) + sum;
        top_s[h] = high;
      }
      __syncwarp();
    }
  }
  __syncthreads();
  for (int h = threadIdx.x; h < H; h += kThSimtThreads) inv_s[h] = 1.f / inv_s[h];
  for (int b = block_lo; b <= block_hi; ++b) {
    locate(b * 32);
    for (int h = warp; h < H; h += WARPS) {
      const float s = score(h, b * 32);
      w_s[h * 33 + lane] = s == -CUDART_INF_F ? 0.f : expf(s - top_s[h]) * inv_s[h];
    }
    __syncthreads();
    for (int e = threadIdx.x; e < H * 32; e += kThSimtThreads) {
      const int h = e >> 5, j = e & 31;
      float m = 0.f;
      for (int g = 0; g < H; ++g) m = fmaf(a.talk[(size_t)h * H + g], w_s[g * 33 + j], m);
      m_s[h * 33 + j] = m;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < H * dv; e += kThSimtThreads) {
      const int h = e / dv, c = e - h * dv;
      float o = acc[e];
      for (int j = 0; j < 32; ++j)
        if (at_s[j] >= 0)
          o = fmaf(m_s[h * 33 + j], to_f32(values[at_s[j] + ((size_t)(h / group) * a.cache.page_size + row_s[j]) * dv + c]), o);
      acc[e] = o;
    }
  }
  for (int e = threadIdx.x; e < H * dv; e += kThSimtThreads) {
    float o = acc[e];
    if (a.gate) o *= th_gate(a, token, e);
    out[token * H * dv + e] = from_f32<T>(o);
  }
}

// ------------------------------------------------------------ tensor cores
constexpr int kThRows = 64, kThKeys = 64, kThThreads = 128;

__device__ __forceinline__ void th_cp_async4(void* smem, const void* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(s), "l"(gmem));
}

// Turns N raw products into capped scores: c tanh(s / c) with s = product * scale.  A warp whose values all lie where the
// series is exact to fp32 takes it (no special functions); otherwise tanh(y) = 1 - 2 / (e^(2y) + 1).
template <int N>
__device__ __forceinline__ void th_cap(float (&s)[N][4], float scale, float cap) {
  if (!(cap > 0.f)) {
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) s[n][c] *= scale;
    return;
  }
  const float to_y = scale / cap;
  float high = 0.f;
#pragma unroll
  for (int n = 0; n < N; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      s[n][c] *= to_y;
      high = fmaxf(high, fabsf(s[n][c]));
    }
  if (__any_sync(0xffffffffu, !(high <= 0.25f))) {
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) s[n][c] = cap * (1.f - __fdividef(2.f, exp2f(s[n][c] * (2.f * kThLog2e)) + 1.f));
  } else {
    // y - y^3 / 3 + 2 y^5 / 15 - 17 y^7 / 315: the next term is below 4e-7 of y at 1/4
#pragma unroll
    for (int n = 0; n < N; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float y = s[n][c], z = y * y;
        s[n][c] = cap * fmaf(y * z, fmaf(z, fmaf(z, -17.f / 315.f, 2.f / 15.f), -1.f / 3.f), y);
      }
  }
}

template <int DK>
__global__ void __launch_bounds__(kThThreads) th_scores_kernel(const __nv_bfloat16* __restrict__ q, ThArgs a) {
  pdl_wait();
  pdl_trigger();
  constexpr int KP = DK + 8;                     // padded rows: ldmatrix rows fall in different banks
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(sm_raw);         // [64][KP]
  __nv_bfloat16* k_s = q_s + kThRows * KP;                                // [2][64][KP]
  float* bias_s = reinterpret_cast<float*>(k_s + 2 * kThKeys * KP);       // [2][group_chunk][q_tile + 63]
  __shared__ long long key_at[2][kThKeys];

  const int d = a.dim, H = a.heads;
  const int entry = blockIdx.y;
  const int group = H / a.kv_heads;
  const int chunks = (group + a.group_chunk - 1) / a.group_chunk;
  const int kvh = blockIdx.z / chunks;
  const int g0 = (blockIdx.z - kvh * chunks) * a.group_chunk;
  const int gc = min(a.group_chunk, group - g0);
  const int row0 = a.q_start[entry];
  const int q_hi = min(a.q_start[entry + 1], a.last_token) - row0;       // (the entry's tokens that belong to this call)
  const int t0 = max(0, a.first_token - row0) + blockIdx.x * a.q_tile;
  if (t0 >= q_hi) return;
  const int nt = min(a.q_tile, q_hi - t0);
  const int nrows = nt * gc;
  const int pos0 = a.kv_start[entry] + t0, last_pos = pos0 + nt - 1;
  const int* table = a.cache.block_table + (size_t)a.slots[entry] * a.cache.table_stride;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int first_key = th_first(pos0, a.window);
  const int s_lo = first_key / kThKeys, steps = last_pos / kThKeys - s_lo + 1;
  const int bw = a.q_tile + kThKeys - 1;                                  // distances a tile spans
  const __nv_bfloat16* k_pages = reinterpret_cast<const __nv_bfloat16*>(a.cache.keys);

  auto fetch = [&](int stage, int step) {
    const int base = (s_lo + step) * kThKeys;
    if (tid < kThKeys) {
      const int idx = base + tid;
      long long at = -1;
      if (idx <= last_pos && idx >= first_key) {
        const int page = th_page(a.cache, table, idx, a.error_word, 0x10000 + entry);
        if (page >= 0) at = (long long)page * a.cache.page_stride + ((long long)kvh * a.cache.page_size + idx % a.cache.page_size) * d;
      }
      key_at[stage][tid] = at;
    }
    if (a.bias) {
      const int lead = pos0 - base - (kThKeys - 1);                       // the distance of entry 0
      float* dst = bias_s + (size_t)stage * a.group_chunk * bw;
      for (int e = tid; e < gc * bw; e += kThThreads) {
        const int g = e / bw, i = e - g * bw;
        th_cp_async4(dst + e, a.bias + (size_t)(kvh * group + g0 + g) * a.span + min(max(lead + i, 0), a.span - 1));
      }
    }
    __syncthreads();
    constexpr int PIECES = DK / 8;
    for (int e = tid; e < kThKeys * PIECES; e += kThThreads) {
      const int j = e / PIECES, cc = (e - j * PIECES) * 8;
      const long long at = key_at[stage][j];
      const bool ok = at >= 0 && cc < d;
      cp_async16(k_s + ((size_t)stage * kThKeys + j) * KP + cc, k_pages + (ok ? at + cc : 0), ok);
    }
    cp_async_commit();
  };
  {
    constexpr int PIECES = DK / 8;
    for (int e = tid; e < kThRows * PIECES; e += kThThreads) {
      const int r = e / PIECES, cc = (e - r * PIECES) * 8;
      const bool ok = r < nrows && cc < d;
      const int t = ok ? r / gc : 0, g = ok ? r - t * gc : 0;
      cp_async16(q_s + (size_t)r * KP + cc, q + (size_t)(row0 + t0 + t) * H * d + (size_t)(kvh * group + g0 + g) * d + (ok ? cc : 0), ok);
    }
  }
  fetch(0, 0);

  // this thread's two rows: g8 and g8 + 8 of the warp's sixteen
  const int g8 = lane >> 2, t4 = lane & 3, row_base = warp * 16;
  int qpos[2], lo[2], base_of[2], bias_at[2];
  float m[2], l[2];
  bool live[2];
  float* words[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = row_base + g8 + 8 * h;
    live[h] = r < nrows;
    const int t = live[h] ? r / gc : 0, g = live[h] ? r - t * gc : 0;
    qpos[h] = pos0 + t;
    lo[h] = th_first(qpos[h], a.window);
    base_of[h] = lo[h] & ~(kThKeys - 1);
    bias_at[h] = g * bw + t + kThKeys - 1;
    words[h] = a.scores + ((size_t)(row0 + t0 + t - a.first_token) * H + (kvh * group + g0 + g)) * a.key_span;
    m[h] = -CUDART_INF_F;
    l[h] = 0.f;
  }
  const int warp_last = pos0 + min(nrows - 1, row_base + 15) / gc;
  const int warp_base = th_base(pos0 + row_base / gc, a.window);
  constexpr int NT = kThKeys / 8;

  for (int step = 0; step < steps; ++step) {
    const int stage = step & 1;
    if (step + 1 < steps) fetch(stage ^ 1, step + 1);
    else cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const int base = (s_lo + step) * kThKeys;
    if (row_base < nrows && base <= warp_last && base >= warp_base) {       // (else the warp's rows see nothing of this tile)
      const __nv_bfloat16* kt = k_s + (size_t)stage * kThKeys * KP;
      float s[NT][4];
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) s[n][c] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DK; kk += 16) {
        uint32_t af[4];
        ldmatrix_x4(af, q_s + (size_t)(row_base + (lane & 15)) * KP + kk + (lane >> 4) * 8);
#pragma unroll
        for (int j = 0; j < NT / 2; ++j) {
          uint32_t bf[4];
          ldmatrix_x4(bf, kt + (size_t)(j * 16 + ((lane >> 4) << 3) + (lane & 7)) * KP + kk + ((lane >> 3) & 1) * 8);
          mma_bf16(s[2 * j], af, bf[0], bf[1]);
          mma_bf16(s[2 * j + 1], af, bf[2], bf[3]);
        }
      }
      th_cap<NT>(s, a.scale, a.cap);
      const float* bias = bias_s + (size_t)stage * a.group_chunk * bw;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        float mx = -CUDART_INF_F;
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int b = 0; b < 2; ++b) {
            const int j = n * 8 + 2 * t4 + b, idx = base + j;
            float v = s[n][2 * h + b];
            if (a.bias) v += bias[bias_at[h] - j];
            v = idx <= qpos[h] && idx >= lo[h] && live[h] ? v * kThLog2e : -CUDART_INF_F;
            s[n][2 * h + b] = v;
            mx = fmaxf(mx, v);
          }
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m[h], mx), top = m_new == -CUDART_INF_F ? 0.f : m_new;
        float sum = 0.f;
#pragma unroll
        for (int n = 0; n < NT; ++n) sum += exp2f(s[n][2 * h] - top) + exp2f(s[n][2 * h + 1] - top);
        l[h] = l[h] * exp2f(m[h] - top) + sum;
        m[h] = m_new;
        if (live[h] && base >= base_of[h] && base <= qpos[h]) {
          float* dst = words[h] + (base - base_of[h]) + 2 * t4;
#pragma unroll
          for (int n = 0; n < NT; ++n) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(s[n][2 * h], s[n][2 * h + 1]);
        }
      }
    }
    __syncthreads();      // the stage is free for the fetch after next
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float sum = l[h];
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    if (live[h] && t4 == 0) {
      const int r = row_base + g8 + 8 * h, t = r / gc, g = r - t * gc;
      a.lse[(size_t)(row0 + t0 + t - a.first_token) * H + (kvh * group + g0 + g)] = m[h] + log2f(sum);
    }
  }
}

__device__ __forceinline__ uint32_t th_split(float v) {      // high bf16 part in the low half, the remainder's in the high half
  const __nv_bfloat16 hi = __float2bfloat16_rn(v);
  const __nv_bfloat162 both = __halves2bfloat162(hi, __float2bfloat16_rn(v - __bfloat162float(hi)));
  return *reinterpret_cast<const uint32_t*>(&both);
}

// One block per token; a warp takes eight keys of all heads at a time: mixed[h][key] = sum_g talk[h][g] w[g][key] as a product
// of 16 x 16 x 8 pieces whose second operand (weights of heads x keys) is made in registers from the words it replaces.
constexpr int kThMixThreads = 256;
template <int HT, bool LO>
__global__ void __launch_bounds__(kThMixThreads) th_mix_kernel(ThArgs a) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, q2 = (lane & 3) * 2, r = lane >> 2;
  const int H = a.heads, padded = HT * 16;
  uint32_t hi_f[HT][HT][4], lo_f[LO ? HT : 1][LO ? HT : 1][4];
#pragma unroll
  for (int mt = 0; mt < HT; ++mt)
#pragma unroll
    for (int kt = 0; kt < HT; ++kt)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const size_t at = (size_t)(mt * 16 + r + (i & 1) * 8) * padded + kt * 16 + q2 + (i >> 1) * 8;
        hi_f[mt][kt][i] = *reinterpret_cast<const uint32_t*>(a.talk_hi + at);
        if (LO) lo_f[LO ? mt : 0][LO ? kt : 0][i] = *reinterpret_cast<const uint32_t*>(a.talk_lo + at);
      }
  pdl_wait();
  pdl_trigger();
  const int pos = a.positions[a.first_token + blockIdx.x];
  const int groups = (pos - th_base(pos, a.window)) / 8 + 1;
  float* words = a.scores + (size_t)blockIdx.x * H * a.key_span;
  float lse[HT][4];
#pragma unroll
  for (int kt = 0; kt < HT; ++kt)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int g = kt * 16 + q2 + (i & 1) + (i >> 1) * 8;
      lse[kt][i] = g < H ? a.lse[(size_t)blockIdx.x * H + g] : 0.f;
    }
  constexpr int WARPS = kThMixThreads / 32;
  constexpr int AHEAD = HT <= 2 ? 2 : 1;          // groups of keys a warp has in flight
  for (int n0 = warp * AHEAD; n0 < groups; n0 += WARPS * AHEAD) {
    float w[AHEAD][HT][4];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
#pragma unroll
      for (int kt = 0; kt < HT; ++kt)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int g = kt * 16 + q2 + (i & 1) + (i >> 1) * 8;
          w[u][kt][i] = g < H && n0 + u < groups ? words[(size_t)g * a.key_span + (n0 + u) * 8 + r] : -CUDART_INF_F;
        }
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      if (n0 + u >= groups) continue;             // (uniform in the warp)
      uint32_t bh[HT][2], bl[HT][2];
#pragma unroll
      for (int kt = 0; kt < HT; ++kt) {
        float e[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) e[i] = exp2f(w[u][kt][i] - lse[kt][i]);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const __nv_bfloat162 pair = __floats2bfloat162_rn(e[2 * half], e[2 * half + 1]);
          const float2 back = bf16x2_floats(pair);
          bh[kt][half] = *reinterpret_cast<const uint32_t*>(&pair);
          bl[kt][half] = pack_bf16(e[2 * half] - back.x, e[2 * half + 1] - back.y);
        }
      }
#pragma unroll
      for (int mt = 0; mt < HT; ++mt) {
        float c[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int kt = 0; kt < HT; ++kt) {
          mma_bf16(c, hi_f[mt][kt], bh[kt][0], bh[kt][1]);
          mma_bf16(c, hi_f[mt][kt], bl[kt][0], bl[kt][1]);
          if (LO) mma_bf16(c, lo_f[LO ? mt : 0][LO ? kt : 0], bh[kt][0], bh[kt][1]);
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int h = mt * 16 + r + half * 8;
          if (h < H)
            *reinterpret_cast<uint2*>(words + (size_t)h * a.key_span + (n0 + u) * 8 + q2) = make_uint2(th_split(c[2 * half]), th_split(c[2 * half + 1]));
        }
      }
    }
  }
}

// (four blocks an SM: the words of sixteen keys are asked for one piece ahead, and other blocks' warps cover the rest)
template <int DV>
__global__ void __launch_bounds__(kThThreads, 4) th_values_kernel(__nv_bfloat16* __restrict__ out, ThArgs a) {
  pdl_wait();
  pdl_trigger();
  constexpr int VP = DV + 8;
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(sm_raw);         // [2][64][VP]
  __shared__ long long val_at[2][kThKeys];
  const int vd = a.vdim, H = a.heads;
  const int entry = blockIdx.y;
  const int group = H / a.kv_heads;
  const int chunks = (group + a.group_chunk - 1) / a.group_chunk;
  const int kvh = blockIdx.z / chunks;
  const int g0 = (blockIdx.z - kvh * chunks) * a.group_chunk;
  const int gc = min(a.group_chunk, group - g0);
  const int row0 = a.q_start[entry];
  const int q_hi = min(a.q_start[entry + 1], a.last_token) - row0;
  const int t0 = max(0, a.first_token - row0) + blockIdx.x * a.q_tile;
  if (t0 >= q_hi) return;
  const int nt = min(a.q_tile, q_hi - t0);
  const int nrows = nt * gc;
  const int pos0 = a.kv_start[entry] + t0, last_pos = pos0 + nt - 1;
  const int* table = a.cache.block_table + (size_t)a.slots[entry] * a.cache.table_stride;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int first_key = th_first(pos0, a.window);
  const int s_lo = first_key / kThKeys, steps = last_pos / kThKeys - s_lo + 1;
  const __nv_bfloat16* v_pages = reinterpret_cast<const __nv_bfloat16*>(a.cache.values);

  auto fetch = [&](int stage, int step) {
    const int base = (s_lo + step) * kThKeys;
    if (tid < kThKeys) {
      const int idx = base + tid;
      long long at = -1;
      if (idx <= last_pos && idx >= first_key) {
        const int page = th_page(a.cache, table, idx, a.error_word, 0x10000 + entry);
        if (page >= 0) at = (long long)page * a.cache.page_stride + ((long long)kvh * a.cache.page_size + idx % a.cache.page_size) * vd;
      }
      val_at[stage][tid] = at;
    }
    __syncthreads();
    constexpr int PIECES = DV / 8;
    for (int e = tid; e < kThKeys * PIECES; e += kThThreads) {
      const int j = e / PIECES, cc = (e - j * PIECES) * 8;
      const long long at = val_at[stage][j];
      const bool ok = at >= 0 && cc < vd;
      cp_async16(v_s + ((size_t)stage * kThKeys + j) * VP + cc, v_pages + (ok ? at + cc : 0), ok);
    }
    cp_async_commit();
  };

  const int g8 = lane >> 2, t4 = lane & 3, row_base = warp * 16;
  int base_of[2], left[2];          // the tile edge the row's words are counted from, and the query's own place (-1: no row)
  bool live[2];
  const float* words[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = row_base + g8 + 8 * h;
    live[h] = r < nrows;
    const int t = live[h] ? r / gc : 0, g = live[h] ? r - t * gc : 0;
    base_of[h] = th_base(pos0 + t, a.window);
    left[h] = live[h] ? pos0 + t - base_of[h] : -1;
    words[h] = a.scores + ((size_t)(row0 + t0 + t - a.first_token) * H + (kvh * group + g0 + g)) * a.key_span;
  }
  // the mixed weights of sixteen keys, as the words lie: [row, row + 8 | keys, keys + 8]; words outside what the row sees of
  // its tiles are zeros
  auto take = [&](int key, uint2 (&f)[4]) {
#pragma unroll
    for (int h = 0; h < 2; ++h)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int at = key + half * 8 + 2 * t4 - base_of[h];
        f[h + 2 * half] = at >= 0 && at <= left[h] ? *reinterpret_cast<const uint2*>(words[h] + at) : make_uint2(0u, 0u);
      }
  };
  float o[DV / 8][4];
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[n][c] = 0.f;
  uint2 now[4], next[4];
  fetch(0, 0);
  take(s_lo * kThKeys, now);
  for (int step = 0; step < steps; ++step) {
    const int stage = step & 1;
    if (step + 1 < steps) fetch(stage ^ 1, step + 1);
    else cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    if (row_base < nrows) {
      const __nv_bfloat16* vt = v_s + (size_t)stage * kThKeys * VP;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        take((s_lo + step) * kThKeys + (kk + 1) * 16, next);
        uint32_t p_hi[4], p_lo[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          p_hi[i] = __byte_perm(now[i].x, now[i].y, 0x5410);
          p_lo[i] = __byte_perm(now[i].x, now[i].y, 0x7632);
        }
#pragma unroll
        for (int dn = 0; dn < DV / 16; ++dn) {
          uint32_t bv[4];
          ldmatrix_x4_trans(bv, vt + (size_t)(kk * 16 + (lane & 15)) * VP + dn * 16 + ((lane >> 4) << 3));
          mma_bf16(o[2 * dn], p_hi, bv[0], bv[1]);
          mma_bf16(o[2 * dn + 1], p_hi, bv[2], bv[3]);
          mma_bf16(o[2 * dn], p_lo, bv[0], bv[1]);
          mma_bf16(o[2 * dn + 1], p_lo, bv[2], bv[3]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) now[i] = next[i];
      }
    }
    __syncthreads();      // the stage is free for the fetch after next
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    if (!live[h]) continue;
    const int r = row_base + g8 + 8 * h, t = r / gc, g = r - t * gc;
    const size_t token = (size_t)(row0 + t0 + t);
    const int head = kvh * group + g0 + g;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) {
      const int c = n * 8 + 2 * t4;
      if (c >= vd) continue;
      float u = o[n][2 * h], v = o[n][2 * h + 1];
      if (a.gate) {
        u *= th_gate(a, token, head * vd + c);
        v *= th_gate(a, token, head * vd + c + 1);
      }
      *reinterpret_cast<uint32_t*>(out + token * H * vd + (size_t)head * vd + c) = pack_bf16(u, v);
    }
  }
}

// ---------------------------------------------------- tensor cores, single tokens
// grid (parts, key heads, requests): this part's tiles of 64 keys against the (up to sixteen) query heads of the key head.
template <int DK>
__global__ void __launch_bounds__(kThThreads) th_step_scores_kernel(const __nv_bfloat16* __restrict__ q, ThArgs a) {
  constexpr int KP = DK + 8, PIECES = DK / 8;
  __shared__ __align__(16) __nv_bfloat16 q_s[16 * KP];
  __shared__ __align__(16) __nv_bfloat16 k_s[kThKeys * KP];
  __shared__ long long key_at[kThKeys];
  __shared__ float m_s[4][16], l_s[4][16];
  const int part = blockIdx.x, kvh = blockIdx.y, entry = blockIdx.z;
  const int d = a.dim, H = a.heads, group = H / a.kv_heads;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos = a.kv_start[entry], lo = th_first(pos, a.window), base0 = th_base(pos, a.window);
  const int tiles = (pos - base0) / kThKeys + 1;
  const int tile_lo = part * a.tiles_per_part, tile_hi = min(tiles, tile_lo + a.tiles_per_part);
  const int* table = a.cache.block_table + (size_t)a.slots[entry] * a.cache.table_stride;
  const __nv_bfloat16* k_pages = reinterpret_cast<const __nv_bfloat16*>(a.cache.keys);
  const int row0 = a.q_start[entry];
  auto locate = [&](int tile) {
    if (tid < kThKeys) {
      const int idx = base0 + tile * kThKeys + tid;
      long long at = -1;
      if (idx <= pos && idx >= lo) {
        const int page = th_page(a.cache, table, idx, a.error_word, 0x10000 + entry);
        if (page >= 0) at = (long long)page * a.cache.page_stride + ((long long)kvh * a.cache.page_size + idx % a.cache.page_size) * d;
      }
      key_at[tid] = at;
    }
    __syncthreads();
  };
  // (the tile's keys but the newest one, which the kernel before this one writes, or that one alone)
  auto copy = [&](int tile, bool newest) {
    const int fresh = pos - (base0 + tile * kThKeys);
    for (int e = tid; e < kThKeys * PIECES; e += kThThreads) {
      const int j = e / PIECES, cc = (e - j * PIECES) * 8;
      if ((j == fresh) != newest) continue;
      const long long at = key_at[j];
      const bool ok = at >= 0 && cc < d;
      cp_async16(k_s + (size_t)j * KP + cc, k_pages + (ok ? at + cc : 0), ok);
    }
  };
  if (tile_lo < tile_hi) {      // what no kernel still running writes is on its way before the wait
    locate(tile_lo);
    copy(tile_lo, false);
  }
  pdl_wait();
  pdl_trigger();
  if (tile_lo >= tile_hi) return;
  copy(tile_lo, true);
  for (int e = tid; e < 16 * PIECES; e += kThThreads) {
    const int g = e / PIECES, cc = (e - g * PIECES) * 8;
    const bool ok = g < group && cc < d;
    cp_async16(q_s + (size_t)g * KP + cc, q + (size_t)row0 * H * d + (size_t)(kvh * group + (ok ? g : 0)) * d + (ok ? cc : 0), ok);
  }
  const int g8 = lane >> 2, t4 = lane & 3;
  float m[2] = {-CUDART_INF_F, -CUDART_INF_F}, l[2] = {0.f, 0.f};
  for (int tile = tile_lo; tile < tile_hi; ++tile) {
    if (tile > tile_lo) {
      __syncthreads();          // (the tile before is no longer read)
      locate(tile);
      copy(tile, false);
      copy(tile, true);
    }
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
    float s[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t af[4], bf[4];
      ldmatrix_x4(af, q_s + (size_t)(lane & 15) * KP + kk + (lane >> 4) * 8);
      ldmatrix_x4(bf, k_s + (size_t)(warp * 16 + ((lane >> 4) << 3) + (lane & 7)) * KP + kk + ((lane >> 3) & 1) * 8);
      mma_bf16(s[0], af, bf[0], bf[1]);
      mma_bf16(s[1], af, bf[2], bf[3]);
    }
    th_cap<2>(s, a.scale, a.cap);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int g = g8 + 8 * h;
      float mx = -CUDART_INF_F;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          const int idx = base0 + tile * kThKeys + warp * 16 + n * 8 + 2 * t4 + b;
          float v = s[n][2 * h + b];
          const bool seen = idx <= pos && idx >= lo && g < group;
          if (a.bias && seen) v += a.bias[(size_t)(kvh * group + g) * a.span + min(pos - idx, a.span - 1)];
          v = seen ? v * kThLog2e : -CUDART_INF_F;
          s[n][2 * h + b] = v;
          mx = fmaxf(mx, v);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m[h], mx), top = m_new == -CUDART_INF_F ? 0.f : m_new;
      float sum = 0.f;
#pragma unroll
      for (int n = 0; n < 2; ++n) sum += exp2f(s[n][2 * h] - top) + exp2f(s[n][2 * h + 1] - top);
      l[h] = l[h] * exp2f(m[h] - top) + sum;
      m[h] = m_new;
      if (g < group) {
        float* dst = a.scores + ((size_t)row0 * H + kvh * group + g) * a.key_span + tile * kThKeys + warp * 16 + 2 * t4;
#pragma unroll
        for (int n = 0; n < 2; ++n) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(s[n][2 * h], s[n][2 * h + 1]);
      }
    }
  }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    if (t4 == 0) { m_s[warp][g8 + 8 * h] = m[h]; l_s[warp][g8 + 8 * h] = l[h]; }
  }
  __syncthreads();
  if (tid < group) {
    float top = fmaxf(fmaxf(m_s[0][tid], m_s[1][tid]), fmaxf(m_s[2][tid], m_s[3][tid]));
    float sum = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) sum += m_s[w][tid] == -CUDART_INF_F ? 0.f : l_s[w][tid] * exp2f(m_s[w][tid] - top);
    float* dst = a.part_ml + (((size_t)row0 * a.n_parts + part) * H + kvh * group + tid) * 2;
    dst[0] = top;
    dst[1] = sum;
  }
}

// The same grid.  GC: query heads of a key head (at most), values up to 128 wide.
template <int GC>
__global__ void __launch_bounds__(kThThreads) th_step_values_kernel(__nv_bfloat16* __restrict__ out, ThArgs a) {
  constexpr int DV = 128, VP = DV + 8, PIECES = DV / 8;
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(sm_raw);          // [64][VP]
  float* mix_s = reinterpret_cast<float*>(v_s + kThKeys * VP);            // [2][GC][64]
  float* sum_s = mix_s + 2 * GC * kThKeys;                                // [GC][128]
  float* lse_s = sum_s + GC * DV;                                         // [heads]
  float* talk_s = lse_s + a.heads;                                        // [GC][heads]
  __shared__ long long val_at[kThKeys];
  __shared__ int is_last;
  const int part = blockIdx.x, kvh = blockIdx.y, entry = blockIdx.z;
  const int vd = a.vdim, H = a.heads, group = H / a.kv_heads;
  const int tid = threadIdx.x;
  const int pos = a.kv_start[entry], lo = th_first(pos, a.window), base0 = th_base(pos, a.window);
  const int tiles = (pos - base0) / kThKeys + 1;
  const int parts = (tiles + a.tiles_per_part - 1) / a.tiles_per_part;    // that have work
  const int tile_lo = part * a.tiles_per_part, tile_hi = min(tiles, tile_lo + a.tiles_per_part);
  const int* table = a.cache.block_table + (size_t)a.slots[entry] * a.cache.table_stride;
  const __nv_bfloat16* v_pages = reinterpret_cast<const __nv_bfloat16*>(a.cache.values);
  const int row0 = a.q_start[entry];
  auto fetch = [&](int tile) {
    if (tid < kThKeys) {
      const int idx = base0 + tile * kThKeys + tid;
      long long at = -1;
      if (idx <= pos && idx >= lo) {
        const int page = th_page(a.cache, table, idx, a.error_word, 0x10000 + entry);
        if (page >= 0) at = (long long)page * a.cache.page_stride + ((long long)kvh * a.cache.page_size + idx % a.cache.page_size) * vd;
      }
      val_at[tid] = at;
    }
    __syncthreads();
    for (int e = tid; e < kThKeys * PIECES; e += kThThreads) {
      const int j = e / PIECES, cc = (e - j * PIECES) * 8;
      const long long at = val_at[j];
      const bool ok = at >= 0 && cc < vd;
      cp_async16(v_s + (size_t)j * VP + cc, v_pages + (ok ? at + cc : 0), ok);
    }
    cp_async_commit();
  };
  if (tile_lo < tile_hi) {
    // The values were stored by the kernel before the one this kernel waits for, which had waited for it to end: the first
    // tile is on its way before the wait.
    fetch(tile_lo);
    for (int e = tid; e < group * H; e += kThThreads) talk_s[e] = a.talk[(size_t)kvh * group * H + e];
  }
  pdl_wait();
  pdl_trigger();
  if (tile_lo >= tile_hi) return;
  const int pair = tid & 63, half = tid >> 6;          // mix: key and half of the heads; values: two columns and half of the keys
  const float* words = a.scores + (size_t)row0 * H * a.key_span + pair;
  // the first scores are on their way while the parts' denominators are added up
  constexpr int AHEAD = 8;
  float ahead[AHEAD];
  auto ask = [&](int tile, int i0) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int h = half + 2 * (i0 + i);
      if (h < H) ahead[i] = words[(size_t)h * a.key_span + tile * kThKeys];
    }
  };
  ask(tile_lo, 0);
  // a warp per head, a lane per part (parts beyond 32 in rounds), four heads in flight
  for (int h0 = (tid >> 5) * 4; h0 < H; h0 += 16) {
    const int lane = tid & 31;
    float top[4], sum[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) { top[i] = -CUDART_INF_F; sum[i] = 0.f; }
    for (int p0 = 0; p0 < parts; p0 += 32) {
      float2 ml[4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        ml[i] = p0 + lane < parts && h0 + i < H
            ? *reinterpret_cast<const float2*>(a.part_ml + (((size_t)row0 * a.n_parts + p0 + lane) * H + h0 + i) * 2)
            : make_float2(-CUDART_INF_F, 0.f);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float high = fmaxf(top[i], warp_max(ml[i].x)), base = high == -CUDART_INF_F ? 0.f : high;
        sum[i] = sum[i] * exp2f(top[i] - base) + warp_sum(ml[i].y * exp2f(ml[i].x - base));
        top[i] = high;
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (lane == 0 && h0 + i < H) lse_s[h0 + i] = top[i] + log2f(sum[i]);
  }
  __syncthreads();
  float o[GC][2];
#pragma unroll
  for (int g = 0; g < GC; ++g) o[g][0] = o[g][1] = 0.f;
  for (int tile = tile_lo; tile < tile_hi; ++tile) {
    if (tile > tile_lo) {
      __syncthreads();
      fetch(tile);
    }
    {
      float mixed[GC];
#pragma unroll
      for (int g = 0; g < GC; ++g) mixed[g] = 0.f;
      for (int i0 = 0; half + 2 * i0 < H; i0 += AHEAD) {
        if (tile > tile_lo || i0 > 0) ask(tile, i0);
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
          const int h = half + 2 * (i0 + i);
          if (h >= H) continue;
          const float w = exp2f(ahead[i] - lse_s[h]);
#pragma unroll
          for (int g = 0; g < GC; ++g)
            if (g < group) mixed[g] = fmaf(talk_s[g * H + h], w, mixed[g]);
        }
      }
#pragma unroll
      for (int g = 0; g < GC; ++g) mix_s[(half * GC + g) * kThKeys + pair] = mixed[g];
    }
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll 4
    for (int jj = 0; jj < kThKeys / 2; ++jj) {
      const int j = half * (kThKeys / 2) + jj;
      const float2 v = bf16x2_floats(*reinterpret_cast<const __nv_bfloat162*>(v_s + (size_t)j * VP + 2 * pair));
#pragma unroll
      for (int g = 0; g < GC; ++g) {
        const float w = mix_s[g * kThKeys + j] + mix_s[(GC + g) * kThKeys + j];
        o[g][0] = fmaf(w, v.x, o[g][0]);
        o[g][1] = fmaf(w, v.y, o[g][1]);
      }
    }
  }
  if (half == 1) {
#pragma unroll
    for (int g = 0; g < GC; ++g) *reinterpret_cast<float2*>(sum_s + g * DV + 2 * pair) = make_float2(o[g][0], o[g][1]);
  }
  __syncthreads();
  const bool mine = half == 0 && 2 * pair < vd;
  if (half == 0) {
#pragma unroll
    for (int g = 0; g < GC; ++g) {
      const float2 f = *reinterpret_cast<const float2*>(sum_s + g * DV + 2 * pair);
      o[g][0] += f.x;
      o[g][1] += f.y;
    }
  }
  if (parts > 1) {
    const size_t stride = (size_t)H * DV;              // floats of one part
    float* dst = a.part_o + ((size_t)row0 * a.n_parts * H + kvh * group) * DV + 2 * pair;
    if (mine) {
#pragma unroll
      for (int g = 0; g < GC; ++g)
        if (g < group) *reinterpret_cast<float2*>(dst + part * stride + (size_t)g * DV) = make_float2(o[g][0], o[g][1]);
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      int* counter = a.counters + entry * a.kv_heads + kvh;
      is_last = atomicAdd(counter, 1) == parts - 1;
      if (is_last) *counter = 0;                        // (every part has counted itself in: ready for the next step)
    }
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    if (mine) {
#pragma unroll
      for (int g = 0; g < GC; ++g) {
        o[g][0] = o[g][1] = 0.f;
        if (g >= group) continue;
        for (int p = 0; p < parts; ++p) {
          const float2 f = __ldcg(reinterpret_cast<const float2*>(dst + p * stride + (size_t)g * DV));
          o[g][0] += f.x;
          o[g][1] += f.y;
        }
      }
    }
  }
  if (mine) {
#pragma unroll
    for (int g = 0; g < GC; ++g) {
      if (g >= group) continue;
      const int col = (kvh * group + g) * vd + 2 * pair;
      float u = o[g][0], v = o[g][1];
      if (a.gate) {
        u *= th_gate(a, (size_t)row0, col);
        v *= th_gate(a, (size_t)row0, col + 1);
      }
      *reinterpret_cast<uint32_t*>(out + (size_t)row0 * H * vd + col) = pack_bf16(u, v);
    }
  }
}

// ------------------------------------------------------------------ launches
template <typename K>
static int th_room(K kern, size_t smem) {
  if (smem > 227 * 1024) return TIB_E_SMEM;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return TIB_OK;
}

template <int DK>
static int th_launch_scores(const void* q, const ThArgs& a, dim3 grid, cudaStream_t stream) {
  const size_t smem = sizeof(__nv_bfloat16) * (size_t)(kThRows + 2 * kThKeys) * (DK + 8) +
                      (a.bias ? sizeof(float) * 2 * (size_t)a.group_chunk * (a.q_tile + kThKeys - 1) : 0);
  const int status = th_room(th_scores_kernel<DK>, smem);
  if (status != TIB_OK) return status;
  TIB_LAUNCH_DEPENDENT(th_scores_kernel<DK>, grid, kThThreads, smem, stream, (const __nv_bfloat16*)q, a);
  return TIB_OK;
}
template <int DV>
static int th_launch_values(void* out, const ThArgs& a, dim3 grid, cudaStream_t stream) {
  const size_t smem = sizeof(__nv_bfloat16) * 2 * (size_t)kThKeys * (DV + 8);
  const int status = th_room(th_values_kernel<DV>, smem);
  if (status != TIB_OK) return status;
  TIB_LAUNCH_DEPENDENT(th_values_kernel<DV>, grid, kThThreads, smem, stream, (__nv_bfloat16*)out, a);
  return TIB_OK;
}
template <int HT>
static int th_launch_mix(const ThArgs& a, int n_tokens, cudaStream_t stream) {
  if (a.talk_lo) TIB_LAUNCH_DEPENDENT((th_mix_kernel<HT, true>), n_tokens, kThMixThreads, 0, stream, a);
  else TIB_LAUNCH_DEPENDENT((th_mix_kernel<HT, false>), n_tokens, kThMixThreads, 0, stream, a);
  return TIB_OK;
}
template <int GC>
static int th_launch_step_values(void* out, const ThArgs& a, dim3 grid, cudaStream_t stream) {
  const size_t smem = sizeof(__nv_bfloat16) * (size_t)kThKeys * 136 +
                      sizeof(float) * (2 * (size_t)GC * kThKeys + (size_t)GC * 128 + a.heads + (size_t)GC * a.heads);
  const int status = th_room(th_step_values_kernel<GC>, smem);
  if (status != TIB_OK) return status;
  TIB_LAUNCH_DEPENDENT(th_step_values_kernel<GC>, grid, kThThreads, smem, stream, (__nv_bfloat16*)out, a);
  return TIB_OK;
}

static bool th_fits_mma(int heads, int dim, int vdim) { return dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 128 && heads <= 64; }

}  // namespace tib

using namespace tib;

// Whether the tensor-core kernels take these sizes (bf16), and whether those for single tokens do.
TIB_API int tib_talking_heads_takes_mma(int heads, int dim, int vdim) { return th_fits_mma(heads, dim, vdim) ? 1 : 0; }
TIB_API int tib_talking_heads_takes_step(int heads, int kv_heads, int dim, int vdim) {
  return kv_heads > 0 && th_fits_mma(heads, dim, vdim) && heads / kv_heads <= 16 ? 1 : 0;
}
// Words of scratch a (token, head) row takes when a query sees at most `window` keys of a context of at most max_kv_len.
TIB_API int tib_talking_heads_key_span(int window, int max_kv_len) {
  const int64_t seen = (int64_t)window + 63, all = max_kv_len;
  return (int)(((seen < all ? seen : all) + 63) / 64 * 64);
}
// Tiles of 64 keys a block of a step of `n_entries` single tokens takes, for rows of key_span words: about six blocks an SM.
TIB_API int tib_talking_heads_tiles_per_part(int n_entries, int kv_heads, int key_span) {
  const int tiles = key_span / 64, rows = n_entries * kv_heads;
  int parts = 6 * 148 / (rows < 1 ? 1 : rows);
  parts = parts < 1 ? 1 : parts > tiles ? tiles : parts;
  return ceil_div(tiles, parts < 1 ? 1 : parts);
}

// proj: [n_tokens, ld] rows with q at q_off, k at k_off, v at v_off; biases and weights fp32 (biases or weights may be null).
TIB_API int tib_row_norm_append(const void* proj, int64_t ld, int q_off, int k_off, int v_off, const float* q_bias,
                                const float* k_bias, const float* v_bias, const float* q_weight, const float* k_weight, float eps,
                                void* q_out, void* k_pages, void* v_pages, const int* positions, const int* token_slot,
                                const int* block_table, int table_stride, int n_tokens, int heads, int kv_heads, int dim, int vdim,
                                int page_size, int64_t page_stride, int num_pages, int* error_word, int dtype, cudaStream_t stream) {
  if (n_tokens == 0) return TIB_OK;
  if (!proj || !q_out || !k_pages || !v_pages || !positions || !token_slot || !block_table || n_tokens < 0) return TIB_E_ARG;
  if (heads < 1 || kv_heads < 1 || dim < 1 || vdim < 1 || page_size < 1) return TIB_E_SIZE;
  ThAppendArgs a;
  a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.q_bias = q_bias; a.k_bias = k_bias; a.v_bias = v_bias;
  a.q_weight = q_weight; a.k_weight = k_weight; a.eps = eps; a.positions = positions; a.token_slot = token_slot;
  a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.vdim = vdim; a.keys = k_pages; a.values = v_pages;
  a.cache.keys = k_pages; a.cache.values = v_pages; a.cache.block_table = block_table; a.cache.table_stride = table_stride;
  a.cache.page_size = page_size; a.cache.page_stride = page_stride; a.cache.num_pages = num_pages; a.error_word = error_word;
  const uintptr_t bits = (uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)q_bias |
                         (uintptr_t)k_bias | (uintptr_t)v_bias | (uintptr_t)q_weight | (uintptr_t)k_weight;
  const bool eights = dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 &&
                      page_stride % 8 == 0 && (bits & 15) == 0;
  if (dtype == TIB_F32)
    TIB_LAUNCH_DEPENDENT((th_append_kernel<float, 1>), dim3(n_tokens, 3), kThAppendThreads, 0, stream, (const float*)proj, (float*)q_out, a);
  else if (dtype == TIB_BF16 && eights)
    TIB_LAUNCH_DEPENDENT((th_append_kernel<__nv_bfloat16, 8>), dim3(n_tokens, 3), kThAppendThreads, 0, stream, (const __nv_bfloat16*)proj, (__nv_bfloat16*)q_out, a);
  else if (dtype == TIB_BF16)
    TIB_LAUNCH_DEPENDENT((th_append_kernel<__nv_bfloat16, 1>), dim3(n_tokens, 3), kThAppendThreads, 0, stream, (const __nv_bfloat16*)proj, (__nv_bfloat16*)q_out, a);
  else
    return TIB_E_DTYPE;
  return TIB_OK;
}

// q: [n_tokens, heads * dim]; out: [n_tokens, heads * vdim]; talk: [heads, heads] fp32; bias: [heads, span] fp32 or null; cap 0:
// none; gate: [n_tokens, heads * vdim] logits (row stride ld_gate, its own dtype) or null.
// form 0: CUDA cores.  form 1 (bf16): portions on the tensor cores, the step's tokens first_token .. last_token - 1; needs
// talk_hi (and talk_lo where talk is not exact in bf16), scores [last - first, heads, key_span] and lse [last - first, heads].
// form 2 (bf16): a step of single tokens; needs scores [n_tokens, heads, key_span], part_ml [n_tokens, n_parts, heads, 2],
// part_o [n_tokens, n_parts, heads, 128] and counters [n_entries * kv_heads] (zeros, and left so).
TIB_API int tib_talking_heads_attention(const void* q, void* out, const int* q_start, const int* kv_start, const int* slots,
                                        const int* positions, const void* k_pages, const void* v_pages, const int* block_table,
                                        int table_stride, int page_size, int64_t page_stride, int num_pages, int n_entries,
                                        int max_q_len, int heads, int kv_heads, int dim, int vdim, int window, float scale, float cap,
                                        const float* bias, int span, const float* talk, const void* talk_hi, const void* talk_lo,
                                        const void* gate, int gate_dtype, int64_t ld_gate, int form, int first_token, int last_token,
                                        float* scores, float* lse, int key_span, float* part_ml, float* part_o, int* counters,
                                        int tiles_per_part, int n_parts, int* error_word, int dtype, cudaStream_t stream) {
  if (n_entries == 0 || max_q_len == 0) return TIB_OK;
  if (!q || !out || !q_start || !kv_start || !slots || !positions || !k_pages || !v_pages || !block_table || !talk) return TIB_E_ARG;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || page_size < 1 || window < 1) return TIB_E_SIZE;
  if (n_entries > 65535 || (bias && span < 1) || !(cap >= 0.f)) return TIB_E_SIZE;
  if (gate && gate_dtype != TIB_F32 && gate_dtype != TIB_BF16) return TIB_E_DTYPE;
  ThArgs a = {};
  a.q_start = q_start; a.kv_start = kv_start; a.slots = slots; a.positions = positions; a.heads = heads; a.kv_heads = kv_heads;
  a.dim = dim; a.vdim = vdim; a.window = window; a.scale = scale; a.cap = cap; a.bias = bias; a.span = span; a.talk = talk;
  a.talk_hi = (const __nv_bfloat16*)talk_hi; a.talk_lo = (const __nv_bfloat16*)talk_lo; a.gate = gate; a.gate_dtype = gate_dtype;
  a.ld_gate = ld_gate; a.error_word = error_word; a.scores = scores; a.lse = lse; a.key_span = key_span;
  a.cache.keys = k_pages; a.cache.values = v_pages; a.cache.block_table = block_table; a.cache.table_stride = table_stride;
  a.cache.page_size = page_size; a.cache.page_stride = page_stride; a.cache.num_pages = num_pages;
  if (form == 0) {
    const size_t smem = sizeof(float) * ((size_t)heads * (dim + vdim + 68) + 1) + 32 * (sizeof(long long) + sizeof(int));
    const dim3 grid(max_q_len, n_entries);
    if (dtype == TIB_F32) {
      const int status = th_room(th_simt_kernel<float>, smem);
      if (status != TIB_OK) return status;
      TIB_LAUNCH_DEPENDENT(th_simt_kernel<float>, grid, kThSimtThreads, smem, stream, (const float*)q, (float*)out, a);
      return TIB_OK;
    }
    if (dtype != TIB_BF16) return TIB_E_DTYPE;
    const int status = th_room(th_simt_kernel<__nv_bfloat16>, smem);
    if (status != TIB_OK) return status;
    TIB_LAUNCH_DEPENDENT(th_simt_kernel<__nv_bfloat16>, grid, kThSimtThreads, smem, stream, (const __nv_bfloat16*)q, (__nv_bfloat16*)out, a);
    return TIB_OK;
  }
  if (dtype != TIB_BF16) return TIB_E_DTYPE;
  if (!th_fits_mma(heads, dim, vdim) || key_span < 64 || key_span % 64) return TIB_E_SIZE;
  if (page_stride % 8 || (((uintptr_t)q | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)scores) & 15) || ((uintptr_t)out & 3)) return TIB_E_ALIGN;
  const int group = heads / kv_heads;
  if (form == 2) {
    if (max_q_len != 1 || group > 16 || tiles_per_part < 1 || n_parts < 1 || (int64_t)tiles_per_part * n_parts * 64 < key_span) return TIB_E_SIZE;
    if (!scores || !part_ml || !part_o || !counters) return TIB_E_ARG;
    a.part_ml = part_ml; a.part_o = part_o; a.counters = counters; a.tiles_per_part = tiles_per_part; a.n_parts = n_parts;
    const dim3 grid(n_parts, kv_heads, n_entries);
    if (dim <= 64) TIB_LAUNCH_DEPENDENT(th_step_scores_kernel<64>, grid, kThThreads, 0, stream, (const __nv_bfloat16*)q, a);
    else TIB_LAUNCH_DEPENDENT(th_step_scores_kernel<128>, grid, kThThreads, 0, stream, (const __nv_bfloat16*)q, a);
    if (group <= 1) return th_launch_step_values<1>(out, a, grid, stream);
    if (group <= 2) return th_launch_step_values<2>(out, a, grid, stream);
    if (group <= 4) return th_launch_step_values<4>(out, a, grid, stream);
    if (group <= 8) return th_launch_step_values<8>(out, a, grid, stream);
    return th_launch_step_values<16>(out, a, grid, stream);
  }
  if (form != 1) return TIB_E_ARG;
  if (!scores || !lse || !talk_hi || first_token < 0 || last_token <= first_token) return TIB_E_ARG;
  a.first_token = first_token; a.last_token = last_token;
  a.group_chunk = group < kThRows ? group : kThRows;
  a.q_tile = kThRows / a.group_chunk;
  const int chunks = ceil_div(group, a.group_chunk), longest = max_q_len < last_token - first_token ? max_q_len : last_token - first_token;
  if ((int64_t)kv_heads * chunks > 65535) return TIB_E_SIZE;
  const dim3 grid(ceil_div(longest, a.q_tile), n_entries, kv_heads * chunks);
  int status = dim <= 64 ? th_launch_scores<64>(q, a, grid, stream) : th_launch_scores<128>(q, a, grid, stream);
  if (status != TIB_OK) return status;
  const int n = last_token - first_token;
  status = heads <= 16 ? th_launch_mix<1>(a, n, stream) : heads <= 32 ? th_launch_mix<2>(a, n, stream) : th_launch_mix<4>(a, n, stream);
  if (status != TIB_OK) return status;
  return vdim <= 64 ? th_launch_values<64>(out, a, grid, stream) : th_launch_values<128>(out, a, grid, stream);
}
