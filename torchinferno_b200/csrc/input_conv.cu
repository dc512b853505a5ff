// A short causal convolution over time on each channel of a sublayer's normed input, added to that input:
//
//   out_t = h_t + sum_j w[j] * h_(t - taps + 1 + j)          (per channel; zeros before a request's first token)
//
//   input_conv        h is given (the norm's rows); the ragged batch, portions and single tokens in one launch
//   norm_conv_step    a step of single tokens: residual += delta, h = RMS norm of the new residual row, the convolution
//                     and the move of the carried rows on by one, in one launch
//
// The last taps - 1 rows h of a request are carried in its state slot (fp32, [taps - 1][width], oldest first, zeros for a
// new request).  Sums are fp32; h is rounded to the activation type before it enters the sum, in both kernels, so that a
// token's row does not depend on the kernel that made it.  The weights come as [taps][width].
#include "common.cuh"

namespace tib {

constexpr int kIcRegTaps = 8;          // taps held in registers; longer convolutions read their rows again
constexpr int kIcThreads = 128;
constexpr int kIcSegment = 16;         // tokens a thread walks (at least the kIcRegTaps - 1 rows that are carried)

struct InputConvArgs {
  const float* weight;                                     // [taps][width]
  float* state; int64_t state_stride; int64_t state_off;   // per slot: [taps - 1][width] at state_off
  const int* q_start; const int* slots;
  int width, taps, segment;
};

template <typename T, int VEC> struct IcRow;
template <typename T> struct IcRow<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f32(*p); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { *p = from_f32<T>(v[0]); }
};
template <> struct IcRow<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct IcRow<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = bf16x2_floats(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = bf16x2_floats(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    uint2 raw;
    *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v[0], v[1]);
    *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = raw;
  }
};

// grid (column tiles, segments, entries).  The block of segment 0 alone touches the request's carried rows: it reads them
// first and leaves the new ones last, so no other block's read can meet its write.  A segment is never shorter than what is
// carried (the host sees to it), so only segment 0 looks back beyond the portion's first row.
template <typename T, int VEC, int MAXT>
__global__ void __launch_bounds__(kIcThreads) input_conv_kernel(const T* __restrict__ x, T* __restrict__ out, InputConvArgs a) {
  pdl_wait();
  pdl_trigger();
  const int entry = blockIdx.z, seg = blockIdx.y;
  const int c = (blockIdx.x * kIcThreads + threadIdx.x) * VEC;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  const int t0 = seg * a.segment;
  if (c >= a.width || t0 >= len) return;
  const int carried = a.taps - 1;
  float* st = a.state + (size_t)a.slots[entry] * a.state_stride + a.state_off + c;
  const T* src = x + (size_t)row0 * a.width + c;
  T* dst = out + (size_t)row0 * a.width + c;
  const int t1 = min(len, t0 + a.segment);
  using Row = IcRow<T, VEC>;
  using State = IcRow<float, VEC>;
  auto row_before = [&](int r, float (&v)[VEC]) {         // row r of the portion, or what the slot carries from before it
    if (r >= 0) Row::load(src + (size_t)r * a.width, v);
    else State::load(st + (size_t)(carried + r) * a.width, v);
  };
  float w[MAXT][VEC], prev[MAXT][VEC];                     // prev[k]: the row carried - k tokens before the one at hand
#pragma unroll
  for (int k = 0; k < MAXT; ++k) {
    if (k < a.taps) State::load(a.weight + (size_t)k * a.width + c, w[k]);
    if (k < carried) row_before(t0 - carried + k, prev[k]);
  }
  float last[MAXT][VEC];                                   // (segment 0) what the next step finds
#pragma unroll
  for (int k = 0; k < MAXT; ++k)
    if (seg == 0 && k < carried) row_before(len - carried + k, last[k]);
  constexpr int AHEAD = 4;
  for (int t = t0; t < t1; t += AHEAD) {
    float h[AHEAD][VEC];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (t + i < t1) Row::load(src + (size_t)(t + i) * a.width, h[i]);
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (t + i >= t1) break;
      float sum[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) sum[e] = 0.f;
#pragma unroll
      for (int k = 0; k < MAXT; ++k)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          if (k < carried) sum[e] = fmaf(w[k][e], prev[k][e], sum[e]);
          else if (k == carried) sum[e] = fmaf(w[k][e], h[i][e], sum[e]);
        }
#pragma unroll
      for (int k = 0; k < MAXT; ++k)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          if (k + 1 < carried) prev[k][e] = prev[k + 1 < MAXT ? k + 1 : k][e];
          else if (k == carried - 1) prev[k][e] = h[i][e];
        }
#pragma unroll
      for (int e = 0; e < VEC; ++e) sum[e] += h[i][e];
      Row::store(dst + (size_t)(t + i) * a.width, sum);
    }
  }
  if (seg == 0) {
#pragma unroll
    for (int k = 0; k < MAXT; ++k)
      if (k < carried) State::store(st + (size_t)k * a.width, last[k]);
  }
}

// Any number of taps: the rows of the sum are read again for every token.  One block walks a portion (grid (column tiles, 1,
// entries)); the carried rows are moved on at the end, oldest first, from rows that are not yet overwritten.
template <typename T>
__global__ void __launch_bounds__(kIcThreads) input_conv_long_kernel(const T* __restrict__ x, T* __restrict__ out, InputConvArgs a) {
  pdl_wait();
  pdl_trigger();
  const int entry = blockIdx.z;
  const int c = blockIdx.x * kIcThreads + threadIdx.x;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  if (c >= a.width || len <= 0) return;
  const int carried = a.taps - 1;
  float* st = a.state + (size_t)a.slots[entry] * a.state_stride + a.state_off + c;
  const T* src = x + (size_t)row0 * a.width + c;
  for (int t = 0; t < len; ++t) {
    float sum = 0.f;
    for (int k = 0; k <= carried; ++k) {
      const int r = t - carried + k;
      const float h = r >= 0 ? to_f32(src[(size_t)r * a.width]) : st[(size_t)(carried + r) * a.width];
      sum = fmaf(a.weight[(size_t)k * a.width + c], h, sum);
    }
    out[(size_t)(row0 + t) * a.width + c] = from_f32<T>(to_f32(src[(size_t)t * a.width]) + sum);
  }
  for (int k = 0; k < carried; ++k) {                      // (row k takes row k + len, which lies behind it)
    const int r = len - carried + k;
    st[(size_t)k * a.width] = r >= 0 ? to_f32(src[(size_t)r * a.width]) : st[(size_t)(carried + r) * a.width];
  }
}

// ------------------------------------------------------------------------------- norm and convolution of single tokens
struct NormConvArgs {
  float* residual; const float* norm_weight; float eps;
  const float* weight;
  float* state; int64_t state_stride; int64_t state_off;
  const int* slots;
  int width, taps;
};

// One block per row; a thread owns eight columns (width a multiple of 8, at most 8 * THREADS): what it needs of the carried
// rows and of the weights is on its way while the row's sum of squares is made.
template <int MAXT, int THREADS>
__global__ void __launch_bounds__(THREADS)
norm_conv_step_x8_kernel(const __nv_bfloat16* __restrict__ delta, __nv_bfloat16* __restrict__ out, NormConvArgs a) {
  __shared__ float scratch[33];
  const int row = blockIdx.x, c = threadIdx.x * 8, carried = a.taps - 1;
  const bool active = c < a.width;
  float4 g0, g1, w[MAXT][2], p[MAXT][2];
  if (active) {        // (the weights are on their way while the kernel before this one drains)
    g0 = *reinterpret_cast<const float4*>(a.norm_weight + c);
    g1 = *reinterpret_cast<const float4*>(a.norm_weight + c + 4);
#pragma unroll
    for (int k = 0; k < MAXT; ++k) {
      if (k < a.taps) {
        w[k][0] = *reinterpret_cast<const float4*>(a.weight + (size_t)k * a.width + c);
        w[k][1] = *reinterpret_cast<const float4*>(a.weight + (size_t)k * a.width + c + 4);
      }
    }
  }
  pdl_wait();
  pdl_trigger();
  float* st = a.state + (size_t)a.slots[row] * a.state_stride + a.state_off + c;
  float h[8];
  float ss = 0.f;
  if (active) {
#pragma unroll
    for (int k = 0; k < MAXT; ++k)
      if (k < carried) {
        p[k][0] = *reinterpret_cast<const float4*>(st + (size_t)k * a.width);
        p[k][1] = *reinterpret_cast<const float4*>(st + (size_t)k * a.width + 4);
      }
    float* res = a.residual + (size_t)row * a.width + c;
    const float4 r0 = *reinterpret_cast<const float4*>(res), r1 = *reinterpret_cast<const float4*>(res + 4);
    uint4 raw = make_uint4(0, 0, 0, 0);
    if (delta) raw = *reinterpret_cast<const uint4*>(delta + (size_t)row * a.width + c);
    h[0] = r0.x; h[1] = r0.y; h[2] = r0.z; h[3] = r0.w; h[4] = r1.x; h[5] = r1.y; h[6] = r1.z; h[7] = r1.w;
    if (delta) {
      const __nv_bfloat162* d2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = bf16x2_floats(d2[i]);
        h[2 * i] += f.x;
        h[2 * i + 1] += f.y;
      }
      *reinterpret_cast<float4*>(res) = make_float4(h[0], h[1], h[2], h[3]);
      *reinterpret_cast<float4*>(res + 4) = make_float4(h[4], h[5], h[6], h[7]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += h[i] * h[i];
  }
  const float total = block_sum(ss, scratch);
  if (!active) return;
  const float inv = rsqrtf(total / (float)a.width + a.eps);
  const float g[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
  uint4 packed;
  __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&packed);
#pragma unroll
  for (int i = 0; i < 8; ++i) h[i] = __bfloat162float(__float2bfloat16_rn(h[i] * inv * g[i]));
  float sum[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) sum[i] = 0.f;
#pragma unroll
  for (int k = 0; k < MAXT; ++k) {
    if (k > carried) continue;
    const float wk[8] = {w[k][0].x, w[k][0].y, w[k][0].z, w[k][0].w, w[k][1].x, w[k][1].y, w[k][1].z, w[k][1].w};
    if (k < carried) {
      const float pk[8] = {p[k][0].x, p[k][0].y, p[k][0].z, p[k][0].w, p[k][1].x, p[k][1].y, p[k][1].z, p[k][1].w};
#pragma unroll
      for (int i = 0; i < 8; ++i) sum[i] = fmaf(wk[i], pk[i], sum[i]);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) sum[i] = fmaf(wk[i], h[i], sum[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) o2[i] = __floats2bfloat162_rn(sum[2 * i] + h[2 * i], sum[2 * i + 1] + h[2 * i + 1]);
  *reinterpret_cast<uint4*>(out + (size_t)row * a.width + c) = packed;
  // the carried rows move on by one
#pragma unroll
  for (int k = 0; k < MAXT; ++k) {
    if (k + 1 < carried) {
      *reinterpret_cast<float4*>(st + (size_t)k * a.width) = p[k + 1 < MAXT ? k + 1 : k][0];
      *reinterpret_cast<float4*>(st + (size_t)k * a.width + 4) = p[k + 1 < MAXT ? k + 1 : k][1];
    } else if (k + 1 == carried) {
      *reinterpret_cast<float4*>(st + (size_t)k * a.width) = make_float4(h[0], h[1], h[2], h[3]);
      *reinterpret_cast<float4*>(st + (size_t)k * a.width + 4) = make_float4(h[4], h[5], h[6], h[7]);
    }
  }
}

// Any width, any number of taps, both types.
template <typename T>
__global__ void norm_conv_step_kernel(const T* __restrict__ delta, T* __restrict__ out, NormConvArgs a) {
  pdl_wait();
  pdl_trigger();
  __shared__ float scratch[33];
  const int row = blockIdx.x, carried = a.taps - 1;
  float* res = a.residual + (size_t)row * a.width;
  float* st = a.state + (size_t)a.slots[row] * a.state_stride + a.state_off;
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
    float v = res[c];
    if (delta) {
      v += to_f32(delta[(size_t)row * a.width + c]);
      res[c] = v;
    }
    ss += v * v;
  }
  const float total = block_sum(ss, scratch);
  const float inv = rsqrtf(total / (float)a.width + a.eps);
  for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
    const float h = to_f32(from_f32<T>(res[c] * inv * a.norm_weight[c]));
    float sum = 0.f;
    for (int k = 0; k < carried; ++k) {
      const float p = st[(size_t)k * a.width + c];
      sum = fmaf(a.weight[(size_t)k * a.width + c], p, sum);
      if (k > 0) st[(size_t)(k - 1) * a.width + c] = p;
    }
    sum = fmaf(a.weight[(size_t)carried * a.width + c], h, sum);
    if (carried > 0) st[(size_t)(carried - 1) * a.width + c] = h;
    out[(size_t)row * a.width + c] = from_f32<T>(h + sum);
  }
}

template <typename T, int VEC>
static int launch_input_conv(const void* x, void* out, InputConvArgs a, int n_entries, int max_q_len, cudaStream_t stream) {
  if (a.taps > kIcRegTaps) {
    TIB_LAUNCH_DEPENDENT(input_conv_long_kernel<T>, dim3(ceil_div(a.width, kIcThreads), 1, n_entries), kIcThreads, 0, stream,
                         (const T*)x, (T*)out, a);
    return TIB_OK;
  }
  a.segment = kIcSegment;
  const dim3 grid(ceil_div(a.width, kIcThreads * VEC), ceil_div(max_q_len, a.segment), n_entries);
  if (grid.y > 65535) return TIB_E_SIZE;
  if (a.taps <= 4) TIB_LAUNCH_DEPENDENT((input_conv_kernel<T, VEC, 4>), grid, kIcThreads, 0, stream, (const T*)x, (T*)out, a);
  else TIB_LAUNCH_DEPENDENT((input_conv_kernel<T, VEC, kIcRegTaps>), grid, kIcThreads, 0, stream, (const T*)x, (T*)out, a);
  return TIB_OK;
}

}  // namespace tib

using namespace tib;

// x, out: [tokens, width] rows of `dtype` that do not overlap; weight: [taps, width] fp32; state: rows of state_stride floats per
// slot, the carried rows [taps - 1, width] at state_off.
TIB_API int tib_input_conv(const void* x, void* out, const float* weight, float* state, int64_t state_stride, int64_t state_off,
                           const int* q_start, const int* slots, int n_entries, int max_q_len, int width, int taps, int dtype,
                           cudaStream_t stream) {
  if (n_entries == 0 || max_q_len == 0) return TIB_OK;
  if (!x || !out || !weight || !q_start || !slots || (taps > 1 && !state) || n_entries < 0 || max_q_len < 0) return TIB_E_ARG;
  if (width < 1 || taps < 1 || n_entries > 65535) return TIB_E_SIZE;
  InputConvArgs a;
  a.weight = weight; a.state = state; a.state_stride = state_stride; a.state_off = state_off; a.q_start = q_start; a.slots = slots;
  a.width = width; a.taps = taps; a.segment = 0;
  const bool vec = width % 4 == 0 && state_stride % 4 == 0 && state_off % 4 == 0 &&
                   (((uintptr_t)x | (uintptr_t)out | (uintptr_t)weight | (uintptr_t)state) & 15) == 0;
  if (dtype == TIB_F32)
    return vec ? launch_input_conv<float, 4>(x, out, a, n_entries, max_q_len, stream)
               : launch_input_conv<float, 1>(x, out, a, n_entries, max_q_len, stream);
  if (dtype == TIB_BF16)
    return vec ? launch_input_conv<__nv_bfloat16, 4>(x, out, a, n_entries, max_q_len, stream)
               : launch_input_conv<__nv_bfloat16, 1>(x, out, a, n_entries, max_q_len, stream);
  return TIB_E_DTYPE;
}

// A step of single tokens: row i belongs to slot slots[i].  delta may be null.
TIB_API int tib_norm_conv_step(const void* delta, float* residual, const float* norm_weight, float eps, const float* weight,
                               float* state, int64_t state_stride, int64_t state_off, const int* slots, void* out, int n_rows,
                               int width, int taps, int dtype, cudaStream_t stream) {
  if (n_rows == 0) return TIB_OK;
  if (!residual || !norm_weight || !weight || !slots || !out || (taps > 1 && !state) || n_rows < 0) return TIB_E_ARG;
  if (width < 1 || taps < 1) return TIB_E_SIZE;
  NormConvArgs a;
  a.residual = residual; a.norm_weight = norm_weight; a.eps = eps; a.weight = weight; a.state = state; a.state_stride = state_stride;
  a.state_off = state_off; a.slots = slots; a.width = width; a.taps = taps;
  int threads = ((width + 3) / 4 + 31) / 32 * 32;
  threads = threads > 1024 ? 1024 : threads;
  if (dtype == TIB_F32) {
    TIB_LAUNCH_DEPENDENT(norm_conv_step_kernel<float>, n_rows, threads, 0, stream, (const float*)delta, (float*)out, a);
    return TIB_OK;
  }
  if (dtype != TIB_BF16) return TIB_E_DTYPE;
  const uintptr_t bits = (uintptr_t)delta | (uintptr_t)residual | (uintptr_t)norm_weight | (uintptr_t)weight | (uintptr_t)state | (uintptr_t)out;
  if (taps <= kIcRegTaps && width % 8 == 0 && width <= (taps <= 4 ? 4096 : 2048) && state_stride % 4 == 0 && state_off % 4 == 0 && (bits & 15) == 0) {
    const int vec_threads = (width / 8 + 31) / 32 * 32;
    if (taps <= 4)
      TIB_LAUNCH_DEPENDENT((norm_conv_step_x8_kernel<4, 512>), n_rows, vec_threads, 0, stream, (const __nv_bfloat16*)delta, (__nv_bfloat16*)out, a);
    else
      TIB_LAUNCH_DEPENDENT((norm_conv_step_x8_kernel<kIcRegTaps, 256>), n_rows, vec_threads, 0, stream, (const __nv_bfloat16*)delta, (__nv_bfloat16*)out, a);
    return TIB_OK;
  }
  TIB_LAUNCH_DEPENDENT(norm_conv_step_kernel<__nv_bfloat16>, n_rows, threads, 0, stream, (const __nv_bfloat16*)delta, (__nv_bfloat16*)out, a);
  return TIB_OK;
}
