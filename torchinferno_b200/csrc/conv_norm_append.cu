// What an attention does between its projection and its scores when q and k pass a short convolution over time:
//
//     u'_t  = sum_j w[j] * u_(t - taps + 1 + j)          per channel of q and of k; rows before a sequence's start are zero
//     value = k'_t as it is (tied values)
//     q, k  = u' / rms of the whole row (all heads at once) * weight per element        (weights null: not normed)
//     pairs (2i, 2i + 1) of the first 2 * n_freq elements of every head turned by position * freq[i]
//
// q goes to q_out, k and the value into their pages.  All of it is fp32 between the projection's rows and what is stored.  The
// last taps - 1 projected rows of a request (its q channels, then its k channels, oldest row first) are carried in its state
// slot.  Every kernel reads the step's ragged batch through its device arrays.
#include "common.cuh"

namespace tib {

struct CnaArgs {
  int64_t ld; int q_off, k_off;
  const float* q_conv; const float* k_conv;            // [taps][heads * dim], [taps][kv_heads * dim]
  const float* q_weight; const float* k_weight;        // [heads * dim], [kv_heads * dim], or both null
  float eps;
  const float* freq; int n_freq;
  const int* positions;
  const int* q_start; const int* slots; int n_entries;
  float* state; int64_t state_stride, state_off;       // per slot: [taps - 1][heads * dim + kv_heads * dim] at state_off
  int heads, kv_heads, dim, taps;
  void* keys; void* values;                            // first key / value of the layer's first page
  const int* block_table; int table_stride;
  int page_size; int64_t page_stride; int num_pages;
  int* error_word;
};

template <typename T, int VEC> __device__ __forceinline__ void cna_load(const T* p, float (&v)[VEC]) {
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
    v[0] = to_f32(p[0]);
  }
}
template <int VEC> __device__ __forceinline__ void cna_load_f32(const float* p, float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  } else {
    v[0] = p[0];
  }
}
template <int VEC> __device__ __forceinline__ void cna_store_f32(float* p, const float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  } else {
    p[0] = v[0];
  }
}
template <typename T, int VEC> __device__ __forceinline__ void cna_store(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    uint4 raw;
    __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) b[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = raw;
  } else {
    p[0] = from_f32<T>(v[0]);
  }
}

constexpr int kCnaThreads = 256;
constexpr int kCnaTapsAhead = 4;       // rows of the convolution asked for together

// grid (tokens, 2): a block each for a token's q and k.  The first taps - 1 tokens of an entry read the carried rows, which the
// entry's last tokens replace: one block (the one of the entry's first token) works through all of them and then leaves the new
// rows, so that no block's read can meet another's write.  VEC 8: bf16, dim a multiple of 8 (a piece of eight never crosses a
// head's edge).
template <typename T, int VEC>
__global__ void __launch_bounds__(kCnaThreads) conv_norm_append_kernel(const T* __restrict__ proj, T* __restrict__ q_out, CnaArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float scratch[33];
  const bool is_q = blockIdx.y == 0;
  const int width = (is_q ? a.heads : a.kv_heads) * a.dim, carried = a.taps - 1;
  const int channels = (a.heads + a.kv_heads) * a.dim, chan0 = is_q ? 0 : a.heads * a.dim;
  float* row_s = sm;                     // [width] the convolved row
  float* cos_s = sm + (width + 3) / 4 * 4;       // [n_freq]
  float* sin_s = cos_s + a.n_freq;       // [n_freq]
  const float* conv = is_q ? a.q_conv : a.k_conv;
  const float* weight = is_q ? a.q_weight : a.k_weight;
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  // the entry this token belongs to: how many entries start at or before it (every warp for itself)
  int entry = -1;
  for (int base = 0; base < a.n_entries; base += 32) {
    const bool at_or_before = base + lane < a.n_entries && a.q_start[base + lane] <= t;
    entry += __popc(__ballot_sync(0xffffffffu, at_or_before));
  }
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0, r0 = t - row0;
  if (r0 > 0 && r0 < carried) return;
  const int r1 = r0 == 0 ? min(max(carried, 1), len) : r0 + 1;
  const int slot = a.slots[entry];
  float* state = a.state ? a.state + (size_t)slot * a.state_stride + a.state_off + chan0 : nullptr;
  const T* src = proj + (size_t)row0 * a.ld + (is_q ? a.q_off : a.k_off);
  const int* table = a.block_table + (size_t)slot * a.table_stride;
  for (int r = r0; r < r1; ++r) {
    const int pos = a.positions[row0 + r];
    for (int i = threadIdx.x; i < a.n_freq; i += kCnaThreads) {
      const float angle = (float)pos * a.freq[i];
      cos_s[i] = cosf(angle);
      sin_s[i] = sinf(angle);
    }
    T* key = nullptr;
    T* value = nullptr;
    if (!is_q) {
      const int page = table[pos / a.page_size];
      if (page >= 0 && page < a.num_pages) {
        const size_t at = (size_t)page * a.page_stride + (size_t)(pos % a.page_size) * a.dim;
        key = reinterpret_cast<T*>(a.keys) + at;
        value = reinterpret_cast<T*>(a.values) + at;
      } else if (a.error_word && threadIdx.x == 0) {
        atomicExch(a.error_word, 0x30000 + (t & 0xffff));
      }
    }
    float ss = 0.f;
    for (int e = threadIdx.x * VEC; e < width; e += kCnaThreads * VEC) {
      float acc[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) acc[i] = 0.f;
      for (int j0 = 0; j0 < a.taps; j0 += kCnaTapsAhead) {
        float u[kCnaTapsAhead][VEC], w[kCnaTapsAhead][VEC];
#pragma unroll
        for (int x = 0; x < kCnaTapsAhead; ++x) {
          const int j = j0 + x, from = r - carried + j;
#pragma unroll
          for (int i = 0; i < VEC; ++i) u[x][i] = w[x][i] = 0.f;
          if (j >= a.taps) continue;
          cna_load_f32<VEC>(conv + (size_t)j * width + e, w[x]);
          if (from >= 0) cna_load<T, VEC>(src + (size_t)from * a.ld + e, u[x]);
          else cna_load_f32<VEC>(state + (size_t)(carried + from) * channels + e, u[x]);
        }
#pragma unroll
        for (int x = 0; x < kCnaTapsAhead; ++x)
#pragma unroll
          for (int i = 0; i < VEC; ++i) acc[i] = fmaf(w[x][i], u[x][i], acc[i]);
      }
      cna_store_f32<VEC>(row_s + e, acc);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(acc[i], acc[i], ss);
      if (value) cna_store<T, VEC>(value + (size_t)(e / a.dim) * a.page_size * a.dim + e % a.dim, acc);
    }
    // (the sum's barriers also publish the row and the angles)
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + a.eps);
    for (int e = threadIdx.x * VEC; e < width; e += kCnaThreads * VEC) {
      const int head = e / a.dim, d = e - head * a.dim;
      float v[VEC];
      if constexpr (VEC == 8) {
        cna_load_f32<VEC>(row_s + e, v);
        if (weight) {
          float g[VEC];
          cna_load_f32<VEC>(weight + e, g);
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[i] = v[i] * inv * g[i];
        }
#pragma unroll
        for (int i = 0; i < VEC; i += 2) {
          const int pair = (d + i) >> 1;
          if (pair >= a.n_freq) continue;
          const float lo = v[i], hi = v[i + 1];
          v[i] = rope_lo(lo, hi, cos_s[pair], sin_s[pair]);
          v[i + 1] = rope_hi(lo, hi, cos_s[pair], sin_s[pair]);
        }
      } else {
        auto normed = [&](int at) { return weight ? row_s[at] * inv * weight[at] : row_s[at]; };
        v[0] = normed(e);
        const int pair = d >> 1;
        if (pair < a.n_freq) {
          const float other = normed(d & 1 ? e - 1 : e + 1);
          v[0] = d & 1 ? rope_hi(other, v[0], cos_s[pair], sin_s[pair]) : rope_lo(v[0], other, cos_s[pair], sin_s[pair]);
        }
      }
      if (is_q) cna_store<T, VEC>(q_out + (size_t)(row0 + r) * width + e, v);
      else if (key) cna_store<T, VEC>(key + (size_t)head * a.page_size * a.dim + d, v);
    }
    __syncthreads();      // the row and the angles are free for the next token
  }
  if (r0 == 0 && carried > 0) {
    // what the next step finds: the last taps - 1 projected rows (rows move up in place, a channel by one thread)
    for (int e = threadIdx.x * VEC; e < width; e += kCnaThreads * VEC)
      for (int k = 0; k < carried; ++k) {
        const int from = len - carried + k;
        float v[VEC];
        if (from >= 0) cna_load<T, VEC>(src + (size_t)from * a.ld + e, v);
        else cna_load_f32<VEC>(state + (size_t)(k + len) * channels + e, v);
        cna_store_f32<VEC>(state + (size_t)k * channels + e, v);
      }
  }
}

// The same for bf16 rows of at most 8 * 1024 columns and at most four taps: a thread owns eight channels, keeps their taps in
// registers and slides over kCnaSegment tokens, whose rows it asks for together; the segment's sums of squares are one reduction.
// grid (segments, entries, 2).  The block of an entry's first segment alone touches the carried rows (a segment is no shorter than
// what is carried): it reads them first and then leaves the new ones.
constexpr int kCnaSegment = 4, kCnaFewTaps = 4;

template <int THREADS>
__global__ void __launch_bounds__(THREADS) conv_norm_append_rows_kernel(const __nv_bfloat16* __restrict__ proj, __nv_bfloat16* __restrict__ q_out, CnaArgs a) {
  extern __shared__ __align__(16) float sm[];                // cos, then sin: [segment][n_freq] each
  __shared__ float sums_s[kCnaSegment][33];
  constexpr int SEG = kCnaSegment, BACK = kCnaFewTaps - 1;
  const bool is_q = blockIdx.z == 0;
  const int width = (is_q ? a.heads : a.kv_heads) * a.dim, carried = a.taps - 1;
  const int channels = (a.heads + a.kv_heads) * a.dim, chan0 = is_q ? 0 : a.heads * a.dim;
  const int e = threadIdx.x * 8, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const bool active = e < width;
  const float* conv = is_q ? a.q_conv : a.k_conv;
  const float* weight = is_q ? a.q_weight : a.k_weight;
  const int entry = blockIdx.y;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0, r0 = blockIdx.x * SEG;
  // taps and gains do not depend on the kernel before.  w[j] is the tap of the row BACK - j places back (zero where there is none)
  float w[kCnaFewTaps][8], gain[8];
#pragma unroll
  for (int j = 0; j < kCnaFewTaps; ++j) {
    const int tap = j - (BACK - carried);
#pragma unroll
    for (int i = 0; i < 8; ++i) w[j][i] = 0.f;
    if (active && tap >= 0) cna_load_f32<8>(conv + (size_t)tap * width + e, w[j]);
  }
  if (active && weight) cna_load_f32<8>(weight + e, gain);
  pdl_wait();
  pdl_trigger();
  if (r0 >= len) return;
  const int n = min(SEG, len - r0);
  const int slot = a.slots[entry];
  float* state = a.state ? a.state + (size_t)slot * a.state_stride + a.state_off + chan0 : nullptr;
  const __nv_bfloat16* src = proj + (size_t)row0 * a.ld + (is_q ? a.q_off : a.k_off);
  float v[SEG][8], ss[SEG];
#pragma unroll
  for (int t = 0; t < SEG; ++t) {
    ss[t] = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) v[t][i] = 0.f;
  }
  if (active) {
    uint4 raw[SEG + BACK];
#pragma unroll
    for (int x = 0; x < SEG + BACK; ++x) {
      const int r = r0 - BACK + x;
      raw[x] = r >= 0 && r < r0 + n ? *reinterpret_cast<const uint4*>(src + (size_t)r * a.ld + e) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int x = 0; x < SEG + BACK; ++x) {
      const int r = r0 - BACK + x;
      float u[8];
      const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&raw[x]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = bf16x2_floats(b[i]);
        u[2 * i] = f.x;
        u[2 * i + 1] = f.y;
      }
      if (r < 0 && r + carried >= 0) cna_load_f32<8>(state + (size_t)(r + carried) * channels + e, u);      // (r < 0 in the first segment only)
#pragma unroll
      for (int t = 0; t < SEG; ++t) {
        const int j = x - t;                               // this row's place among the taps of token t
        if (j < 0 || j > BACK) continue;
#pragma unroll
        for (int i = 0; i < 8; ++i) v[t][i] = fmaf(w[j][i], u[i], v[t][i]);
      }
    }
#pragma unroll
    for (int t = 0; t < SEG; ++t)
#pragma unroll
      for (int i = 0; i < 8; ++i) ss[t] = fmaf(v[t][i], v[t][i], ss[t]);
    if (r0 == 0 && carried > 0)       // what the next step finds: the last projected rows (rows move up in place, a channel by one thread)
      for (int k = 0; k < carried; ++k) {
        const int from = len - carried + k;
        float u[8];
        if (from >= 0) cna_load<__nv_bfloat16, 8>(src + (size_t)from * a.ld + e, u);
        else cna_load_f32<8>(state + (size_t)(k + len) * channels + e, u);
        cna_store_f32<8>(state + (size_t)k * channels + e, u);
      }
  }
  for (int i = threadIdx.x; i < n * a.n_freq; i += blockDim.x) {
    const int t = i / a.n_freq, f = i - t * a.n_freq;
    const float angle = (float)a.positions[row0 + r0 + t] * a.freq[f];
    sm[i] = cosf(angle);
    sm[SEG * a.n_freq + i] = sinf(angle);
  }
#pragma unroll
  for (int t = 0; t < SEG; ++t) {
    const float s = warp_sum(ss[t]);
    if (lane == 0) sums_s[t][warp] = s;
  }
  __syncthreads();
  if (!active) return;
  const int head = e / a.dim, d = e - head * a.dim;
  const int* table = a.block_table + (size_t)slot * a.table_stride;
#pragma unroll
  for (int t = 0; t < SEG; ++t) {
    if (t >= n) break;
    const size_t token = (size_t)row0 + r0 + t;
    __nv_bfloat16* dst = q_out + token * width + e;
    if (!is_q) {
      const int pos = a.positions[token], page = table[pos / a.page_size];
      if (page < 0 || page >= a.num_pages) {
        if (a.error_word && threadIdx.x == 0) atomicExch(a.error_word, 0x30000 + (int)(token & 0xffff));
        continue;
      }
      const size_t at = (size_t)page * a.page_stride + ((size_t)head * a.page_size + pos % a.page_size) * a.dim + d;
      cna_store<__nv_bfloat16, 8>(reinterpret_cast<__nv_bfloat16*>(a.values) + at, v[t]);
      dst = reinterpret_cast<__nv_bfloat16*>(a.keys) + at;
    }
    if (weight) {
      float total = 0.f;
      for (int x = 0; x < warps; ++x) total += sums_s[t][x];
      const float inv = 1.f / sqrtf(total / (float)width + a.eps);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[t][i] = v[t][i] * inv * gain[i];
    }
#pragma unroll
    for (int i = 0; i < 8; i += 2) {
      const int pair = (d + i) >> 1;
      if (pair >= a.n_freq) continue;
      const float lo = v[t][i], hi = v[t][i + 1], c = sm[t * a.n_freq + pair], sn = sm[(SEG + t) * a.n_freq + pair];
      v[t][i] = rope_lo(lo, hi, c, sn);
      v[t][i + 1] = rope_hi(lo, hi, c, sn);
    }
    cna_store<__nv_bfloat16, 8>(dst, v[t]);
  }
}

}  // namespace tib

using namespace tib;

// proj: [n_tokens, ld] rows with q at q_off and k at k_off; q_out: [n_tokens, heads * dim]; k_pages / v_pages: first key / value
// of this layer's first page (heads of `dim` elements in both); state (null when taps is 1): see CnaArgs.  max_q_len: the longest entry of the step.
TIB_API int tib_conv_norm_append(const void* proj, int64_t ld, int q_off, int k_off, const float* q_conv, const float* k_conv, int taps,
                                 const float* q_weight, const float* k_weight, float eps, const float* freq, int n_freq, void* q_out,
                                 void* k_pages, void* v_pages, const int* positions, const int* block_table,
                                 int table_stride, const int* q_start, const int* slots, int n_entries, float* state,
                                 int64_t state_stride, int64_t state_off, int n_tokens, int max_q_len, int heads, int kv_heads,
                                 int dim, int page_size, int64_t page_stride, int num_pages, int* error_word, int dtype, cudaStream_t stream) {
  if (n_tokens == 0 || n_entries == 0 || max_q_len == 0) return TIB_OK;
  if (!proj || !q_out || !k_pages || !v_pages || !q_conv || !k_conv || !positions || !block_table || !q_start || !slots) return TIB_E_ARG;
  if ((!q_weight) != (!k_weight) || (n_freq > 0 && !freq) || (taps > 1 && !state)) return TIB_E_ARG;
  if (heads < 1 || kv_heads < 1 || dim < 1 || taps < 1 || n_freq < 0 || 2 * n_freq > dim || page_size < 1) return TIB_E_SIZE;
  CnaArgs a;
  a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.q_conv = q_conv; a.k_conv = k_conv; a.q_weight = q_weight; a.k_weight = k_weight;
  a.eps = eps; a.freq = freq; a.n_freq = n_freq; a.positions = positions; a.q_start = q_start;
  a.slots = slots; a.n_entries = n_entries; a.state = taps > 1 ? state : nullptr; a.state_stride = state_stride; a.state_off = state_off;
  a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.taps = taps; a.keys = k_pages; a.values = v_pages;
  a.block_table = block_table; a.table_stride = table_stride; a.page_size = page_size; a.page_stride = page_stride;
  a.num_pages = num_pages; a.error_word = error_word;
  const size_t smem = sizeof(float) * ((size_t)(heads > kv_heads ? heads : kv_heads) * dim + 4 + 2 * (size_t)n_freq);
  if (smem > 227 * 1024) return TIB_E_SMEM;
  uintptr_t bits = (uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)q_conv | (uintptr_t)k_conv |
                   (uintptr_t)q_weight | (uintptr_t)k_weight | (uintptr_t)state;
  const bool pieces = dtype == TIB_BF16 && dim % 8 == 0 && ld % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && page_stride % 8 == 0 &&
                      state_stride % 4 == 0 && state_off % 4 == 0 && (bits & 15) == 0;
#define TIB_CNA(T, VEC)                                                                                              \
  do {                                                                                                               \
    auto kern = conv_norm_append_kernel<T, VEC>;                                                                     \
    if (smem > 48 * 1024) {                                                                                          \
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);            \
      if (e != cudaSuccess) return (int)e;                                                                           \
    }                                                                                                                \
    TIB_LAUNCH_DEPENDENT(kern, dim3(n_tokens, 2), kCnaThreads, smem, stream, (const T*)proj, (T*)q_out, a);          \
  } while (0)
  const int wide = (heads > kv_heads ? heads : kv_heads) * dim, segments = ceil_div(max_q_len, kCnaSegment);
  if (pieces && taps <= kCnaFewTaps && wide <= 8 * 1024 && n_entries <= 65535) {
    const int threads = ceil_div(wide / 8, 32) * 32;
    const size_t angles = sizeof(float) * 2 * kCnaSegment * (size_t)n_freq;
    if (angles <= 48 * 1024) {
      const dim3 grid(segments, n_entries, 2);
      if (threads <= 512)
        TIB_LAUNCH_DEPENDENT(conv_norm_append_rows_kernel<512>, grid, threads, angles, stream, (const __nv_bfloat16*)proj, (__nv_bfloat16*)q_out, a);
      else
        TIB_LAUNCH_DEPENDENT(conv_norm_append_rows_kernel<1024>, grid, threads, angles, stream, (const __nv_bfloat16*)proj, (__nv_bfloat16*)q_out, a);
      return TIB_OK;
    }
  }
  if (pieces) TIB_CNA(__nv_bfloat16, 8);
  else if (dtype == TIB_BF16) TIB_CNA(__nv_bfloat16, 1);
  else if (dtype == TIB_F32) TIB_CNA(float, 1);
  else return TIB_E_DTYPE;
#undef TIB_CNA
  return TIB_OK;
}
