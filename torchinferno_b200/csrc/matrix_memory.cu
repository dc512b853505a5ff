// A matrix memory with exponential gates (the mLSTM of xLSTM), after its projections.  Per head, with q and k of D elements, v of
// V, all of it in 32-bit:
//
//     i_t = cap tanh((raw_i + bias_i) / cap),   f_t = logsigmoid(cap tanh((raw_f + bias_f) / cap))
//     m_t = max(f_t + m_(t-1), i_t)                                                     (m starts at 0)
//     S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T;   n_t likewise with k_t alone
//     y_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6),   q_t = q_scale times the projected row
//     out_t = y_t / rms(y_t) * weight * sigmoid(gate_t)                                 (per head; optional, see below)
//
// for the tokens of a ragged batch, read through its device arrays only.  A request's state: S of every head [H][D][V], then
// for every head and every tile of kMemTile value columns a copy of n [D] and m (a block owns a tile of columns and keeps its
// own n and m, so no block waits for another), zero for a new request.
//
// Two ways to run a step:
//   walk     token after token, fp32 on the CUDA cores: single tokens, short portions, the 32-bit path, any head size up to 512.
//            A block owns (head, tile of columns, request) with its part of S in registers: four columns a thread, every
//            eighth row.  A step of single tokens may have the block work the two gate rows out itself (two dot products with
//            the layer's input), and where a head is one tile the norm and the gate end the kernel.
//   chunks   longer portions in bf16 (head sizes that are multiples of 8, D up to 256): chunks of 64 tokens side by side on the
//            tensor cores (mma.sync).  With F_t the sum of f up to t and everything relative to a chunk's start,
//                m_t = F_t + max(m_start, max over s <= t of (i_s - F_s))
//                S_end = exp(F_end + m_start - m_end) S_start + sum_s exp(F_end - F_s + i_s - m_end) k_s v_s^T
//                S_t^T q_t = exp(F_t + m_start - m_t) S_start^T q_t + sum_(s <= t) exp(F_t - F_s + i_s - m_t) (q_t . k_s) v_s
//            which is the recurrence written out.  Kernels: gates (F in double precision by a scan over the portion, and
//            m), local (every chunk's own sum), fold (the states at the chunks' starts, one after another; the last one goes to
//            the slot), out (the outputs of every chunk).  q, k and v are bf16 as the projection left them; everything
//            computed (weighted keys, weighted scores, S) enters a product as a high bf16 part plus the remainder, 16 bits, and
//            all sums are fp32.  Where a portion is cut changes the order of fp32 sums only.
#include "mma.cuh"

namespace tib {

constexpr int kMemTile = 128;          // value columns of a tile
constexpr int kMemChunk = 64;          // tokens of a chunk
constexpr int kMemMaxDim = 512;

struct MemArgs {
  const void* proj; int64_t ld; int q_off, k_off, v_off, g_off;     // rows of the fused projection (type T); g: the output gate
  float q_scale;
  const float* logits; int64_t ld_logits;                            // [tokens, >= 2 * heads] raw gate rows (i of every head, then f), or null:
  const void* x; int64_t ldx; const float* gate_w; int width;       //   the layer's input rows (type T) and the rows' weights [2 * heads, width]
  const float* gate_bias; float cap;                                 // [2 * heads]
  float* state; int64_t state_stride;
  const int* q_start; const int* slots;
  const float* norm_weight; float eps;                               // [heads * V], or null: `y` gets the heads' outputs as they are
  float* y;                                                          // [tokens, heads * V] fp32, or null
  void* out;                                                         // [tokens, heads * V] of type T (normed and gated), or null
  int heads, D, V, tiles, n_tokens;
  // chunks
  double* cum; float* log_in; float* top;                            // [heads][tokens]: F from the entry's start, i, m
  float* top0;                                                       // [heads][entries]: m ahead of the entry's first token
  float* run_state; float* run_n; float* run_keep;                   // [runs][heads][D * V], [runs][heads][D], [runs][heads]
  int n_entries;
};

__device__ __forceinline__ float* mem_norm_state(const MemArgs& a, float* slot, int h, int tile) {
  return slot + (size_t)a.heads * a.D * a.V + ((size_t)h * a.tiles + tile) * (a.D + 1);
}
__device__ __forceinline__ float mem_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float mem_capped(float z, float cap) { return cap * tanhf(z / cap); }

// ------------------------------------------------------------------------------------------------------- walk
constexpr int kWalkThreads = 256, kWalkWarps = 8;

// R: rows of S a thread holds (every eighth row of the head's D)
template <typename T, int R>
__global__ void __launch_bounds__(kWalkThreads) mem_walk_kernel(MemArgs a) {
  __shared__ float k_s[kMemMaxDim], q_s[kMemMaxDim], n_s[kMemMaxDim];
  __shared__ __align__(16) float v_s[kMemTile];
  __shared__ __align__(16) float part_s[kWalkWarps][kMemTile];
  __shared__ float sum_s[2][kWalkWarps];
  __shared__ float gate_s[2];
  __shared__ float scratch[33];
  const int D = a.D, V = a.V, H = a.heads;
  const int h = blockIdx.x / a.tiles, tile = blockIdx.x - h * a.tiles, entry = blockIdx.y;
  const int c0 = tile * kMemTile, cols = min(kMemTile, V - c0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  if (len <= 0) {
    pdl_wait();
    return;
  }
  float* slot = a.state + (size_t)a.slots[entry] * a.state_stride;
  float* S = slot + (size_t)h * D * V + c0;
  float* nm = mem_norm_state(a, slot, h, tile);
  const bool vec = V % 4 == 0 && (((uintptr_t)slot) & 15) == 0;
  const int c = lane * 4;
  // The state was left by an earlier step, long complete: it is asked for ahead of the wait for the projection.
  float4 s[R];
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int d = warp + kWalkWarps * j;
    s[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (d < D && c < cols) {
      const float* p = S + (size_t)d * V + c;
      if (vec) s[j] = *reinterpret_cast<const float4*>(p);
      else {
        s[j].x = p[0];
        if (c + 1 < cols) s[j].y = p[1];
        if (c + 2 < cols) s[j].z = p[2];
        if (c + 3 < cols) s[j].w = p[3];
      }
    }
  }
  for (int d = tid; d < D; d += kWalkThreads) n_s[d] = nm[d];
  float m = nm[D];
  const float bias_i = a.gate_bias[h], bias_f = a.gate_bias[H + h];
  pdl_wait();
  pdl_trigger();
  const T* proj = reinterpret_cast<const T*>(a.proj);
  for (int t = 0; t < len; ++t) {
    const size_t token = row0 + t;
    const T* row = proj + token * a.ld;
    for (int d = tid; d < D; d += kWalkThreads) {
      q_s[d] = to_f32(row[a.q_off + h * D + d]) * a.q_scale;
      k_s[d] = to_f32(row[a.k_off + h * D + d]);
    }
    if (tid < cols) v_s[tid] = to_f32(row[a.v_off + h * V + c0 + tid]);
    else if (tid < kMemTile) v_s[tid] = 0.f;
    if (a.logits) {
      if (tid < 2) gate_s[tid] = a.logits[token * a.ld_logits + tid * H + h];
    } else {
      // the two gate rows times this token's input
      const T* x = reinterpret_cast<const T*>(a.x) + token * a.ldx;
      const float* wi = a.gate_w + (size_t)h * a.width;
      const float* wf = a.gate_w + (size_t)(H + h) * a.width;
      float zi = 0.f, zf = 0.f;
#pragma unroll 4
      for (int e = tid; e < a.width; e += kWalkThreads) {
        const float xv = to_f32(x[e]);
        zi = fmaf(xv, wi[e], zi);
        zf = fmaf(xv, wf[e], zf);
      }
      zi = warp_sum(zi);
      zf = warp_sum(zf);
      if (lane == 0) { sum_s[0][warp] = zi; sum_s[1][warp] = zf; }
      __syncthreads();
      if (tid < 2) {
        float z = 0.f;
#pragma unroll
        for (int w = 0; w < kWalkWarps; ++w) z += sum_s[tid][w];
        gate_s[tid] = z;
      }
    }
    __syncthreads();
    const float log_in = mem_capped(gate_s[0] + bias_i, a.cap);
    const float log_keep = mem_log_sigmoid(mem_capped(gate_s[1] + bias_f, a.cap)) + m;
    const float m_new = fmaxf(log_keep, log_in);
    const float keep = expf(log_keep - m_new), take = expf(log_in - m_new);
    m = m_new;
    float nq = 0.f;
    for (int d = tid; d < D; d += kWalkThreads) {
      const float nv = fmaf(keep, n_s[d], take * k_s[d]);
      n_s[d] = nv;
      nq = fmaf(nv, q_s[d], nq);
    }
    const float4 v4 = *reinterpret_cast<const float4*>(v_s + c);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int d = warp + kWalkWarps * j;
      if (d >= D) break;
      const float kt = take * k_s[d], qd = q_s[d];
      s[j].x = fmaf(keep, s[j].x, kt * v4.x); s[j].y = fmaf(keep, s[j].y, kt * v4.y);
      s[j].z = fmaf(keep, s[j].z, kt * v4.z); s[j].w = fmaf(keep, s[j].w, kt * v4.w);
      acc.x = fmaf(qd, s[j].x, acc.x); acc.y = fmaf(qd, s[j].y, acc.y);
      acc.z = fmaf(qd, s[j].z, acc.z); acc.w = fmaf(qd, s[j].w, acc.w);
    }
    *reinterpret_cast<float4*>(&part_s[warp][c]) = acc;
    nq = block_sum(nq, scratch);            // (its barriers also publish part_s)
    float y = 0.f;
    if (tid < cols) {
#pragma unroll
      for (int w = 0; w < kWalkWarps; ++w) y += part_s[w][tid];
      y /= fmaxf(fabsf(nq), expf(-m)) + 1e-6f;
    }
    const size_t at = token * (size_t)H * V + (size_t)h * V + c0 + tid;
    if (a.norm_weight) {                    // (the head is one tile)
      const float inv = 1.f / sqrtf(block_sum(tid < cols ? y * y : 0.f, scratch) / (float)V + a.eps);
      if (tid < cols) {
        const float g = to_f32(row[a.g_off + h * V + tid]);
        reinterpret_cast<T*>(a.out)[at] = from_f32<T>(y * inv * a.norm_weight[h * V + tid] / (1.f + expf(-g)));
      }
    } else if (tid < cols) {
      a.y[at] = y;
    }
    __syncthreads();                        // q_s, k_s, v_s, gate_s, part_s are free for the next token
  }
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int d = warp + kWalkWarps * j;
    if (d < D && c < cols) {
      float* p = S + (size_t)d * V + c;
      if (vec) *reinterpret_cast<float4*>(p) = s[j];
      else {
        p[0] = s[j].x;
        if (c + 1 < cols) p[1] = s[j].y;
        if (c + 2 < cols) p[2] = s[j].z;
        if (c + 3 < cols) p[3] = s[j].w;
      }
    }
  }
  for (int d = tid; d < D; d += kWalkThreads) nm[d] = n_s[d];
  if (tid == 0) nm[D] = m;
}

// ------------------------------------------------------------------------------------------------------ chunks
// The first run of an entry in the run arrays (an entry of len tokens has at most len / kMemChunk + 1 chunks, and the next
// entry starts len rows and one entry later).
__device__ __forceinline__ size_t mem_first_run(int row0, int entry) { return (size_t)(row0 / kMemChunk) + entry; }

// Two steps after one another, (F1, a1) then (F2, a2), with m_after = F + max(m_before, a).
struct MemSpan { double F, a; };
__device__ __forceinline__ MemSpan mem_then(MemSpan x, MemSpan y) { return {x.F + y.F, fmax(x.a, y.a - x.F)}; }

constexpr int kGateThreads = 256;

// grid (heads, entries): i, the running sum of f and m of every token.
__global__ void __launch_bounds__(kGateThreads) mem_gates_kernel(MemArgs a) {
  __shared__ MemSpan warp_s[kGateThreads / 32];
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, entry = blockIdx.y, H = a.heads;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  if (len <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* slot = a.state + (size_t)a.slots[entry] * a.state_stride;
  const double m0 = (double)mem_norm_state(a, slot, h, 0)[a.D];
  if (tid == 0) a.top0[(size_t)h * a.n_entries + entry] = (float)m0;
  const float bias_i = a.gate_bias[h], bias_f = a.gate_bias[H + h];
  double* cum = a.cum + (size_t)h * a.n_tokens + row0;
  float* log_in = a.log_in + (size_t)h * a.n_tokens + row0;
  float* top = a.top + (size_t)h * a.n_tokens + row0;
  // pass by pass over the portion, a token a thread; what the passes before leave behind is (F, a) = `before`
  MemSpan before = {0.0, -1e300};
  for (int base = 0; base < len; base += kGateThreads) {
    const int t = base + tid;
    MemSpan mine = {0.0, -1e300};            // (a thread without a token changes nothing)
    float in = 0.f;
    if (t < len) {
      const float* z = a.logits + (size_t)(row0 + t) * a.ld_logits + h;
      in = mem_capped(z[0] + bias_i, a.cap);
      const double f = (double)mem_log_sigmoid(mem_capped(z[H] + bias_f, a.cap));
      mine = {f, (double)in - f};
    }
    // inclusive scan: within the warp, then over the warps
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const MemSpan left = {__shfl_up_sync(0xffffffffu, mine.F, o), __shfl_up_sync(0xffffffffu, mine.a, o)};
      if (lane >= o) mine = mem_then(left, mine);
    }
    if (lane == 31) warp_s[warp] = mine;
    __syncthreads();
    MemSpan ahead = before;
    for (int w = 0; w < warp; ++w) ahead = mem_then(ahead, warp_s[w]);
    mine = mem_then(ahead, mine);
    if (t < len) {
      cum[t] = mine.F;
      log_in[t] = in;
      top[t] = (float)(mine.F + fmax(m0, mine.a));
    }
    for (int w = 0; w < kGateThreads / 32; ++w) before = mem_then(before, warp_s[w]);
    __syncthreads();                         // warp_s is free for the next pass
  }
}

// What a block of the two kernels below needs of a chunk: F relative to the chunk's start as two floats (their differences are
// then exact to the last bit that matters), i, m, and m ahead of the chunk.
struct MemChunkGates {
  float hi[kMemChunk], lo[kMemChunk], in[kMemChunk], top[kMemChunk];
};
__device__ __forceinline__ float mem_load_gates(const MemArgs& a, MemChunkGates& g, int h, int entry, int row0, int t0, int n) {
  const size_t first = (size_t)h * a.n_tokens + row0 + t0;
  const double base = t0 > 0 ? a.cum[first - 1] : 0.0;
  for (int t = threadIdx.x; t < kMemChunk; t += blockDim.x) {
    double F = 0.0;
    if (t < n) F = a.cum[first + t] - base;
    const float hi = (float)F;
    g.hi[t] = hi;
    g.lo[t] = (float)(F - (double)hi);
    g.in[t] = t < n ? a.log_in[first + t] : 0.f;
    g.top[t] = t < n ? a.top[first + t] : 0.f;
  }
  return t0 > 0 ? a.top[first - 1] : a.top0[(size_t)h * a.n_entries + entry];
}

constexpr int kLocalThreads = 256;

static inline size_t mem_local_smem(int dp, int vt) {
  return sizeof(__nv_bfloat16) * ((size_t)2 * kMemChunk * (dp + 8) + (size_t)kMemChunk * (vt + 8));
}

// grid (chunks, heads * tiles, entries): run_state = sum_s w_s k_s v_s^T and run_n = sum_s w_s k_s over the chunk's tokens,
// w_s = exp(F_end - F_s + i_s - m_end); run_keep = what S_start is multiplied by on the way to the chunk's end.
template <int VT>
__global__ void __launch_bounds__(kLocalThreads) mem_local_kernel(MemArgs a) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ MemChunkGates gates;
  pdl_wait();
  pdl_trigger();
  const int D = a.D, V = a.V, DP = (D + 15) & ~15, KP = DP + 8;
  constexpr int VP = VT + 8;
  __nv_bfloat16* k_hi = reinterpret_cast<__nv_bfloat16*>(sm_raw);      // [64][KP]
  __nv_bfloat16* k_lo = k_hi + kMemChunk * KP;                          // [64][KP]
  __nv_bfloat16* v_s = k_lo + kMemChunk * KP;                           // [64][VP]
  const int entry = blockIdx.z, h = blockIdx.y / a.tiles, tile = blockIdx.y - h * a.tiles;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  const int t0 = blockIdx.x * kMemChunk;
  if (t0 >= len) return;
  const int n = min(kMemChunk, len - t0);
  const int c0 = tile * kMemTile, cols = min(VT, V - c0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj) + (size_t)(row0 + t0) * a.ld;
  for (int e = tid; e < kMemChunk * (VT / 8); e += kLocalThreads) {
    const int t = e / (VT / 8), cc = (e - t * (VT / 8)) * 8;
    const bool ok = t < n && cc < cols;
    cp_async16(v_s + t * VP + cc, ok ? proj + (size_t)t * a.ld + a.v_off + h * V + c0 + cc : proj, ok);
  }
  cp_async_commit();
  const float m_start = mem_load_gates(a, gates, h, entry, row0, t0, n);
  __syncthreads();
  const float hi_end = gates.hi[n - 1], lo_end = gates.lo[n - 1], m_end = gates.top[n - 1];
  const size_t run = mem_first_run(row0, entry) + blockIdx.x;
  if (tid == 0 && tile == 0) a.run_keep[run * a.heads + h] = expf(hi_end + (lo_end + (m_start - m_end)));
  for (int e = tid; e < kMemChunk * (DP / 8); e += kLocalThreads) {
    const int t = e / (DP / 8), d = (e - t * (DP / 8)) * 8;
    uint4 hi4 = make_uint4(0, 0, 0, 0), lo4 = hi4;
    if (t < n && d < D) {
      const float w = expf((hi_end - gates.hi[t]) + ((lo_end - gates.lo[t]) + (gates.in[t] - m_end)));
      const uint4 raw = *reinterpret_cast<const uint4*>(proj + (size_t)t * a.ld + a.k_off + h * D + d);
      const __nv_bfloat162* k2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
      __nv_bfloat162* ph = reinterpret_cast<__nv_bfloat162*>(&hi4);
      uint32_t* pl = reinterpret_cast<uint32_t*>(&lo4);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = bf16x2_floats(k2[i]);
        const float x = f.x * w, y = f.y * w;
        ph[i] = __floats2bfloat162_rn(x, y);
        const float2 r = bf16x2_floats(ph[i]);
        pl[i] = pack_bf16(x - r.x, y - r.y);
      }
    }
    *reinterpret_cast<uint4*>(k_hi + t * KP + d) = hi4;
    *reinterpret_cast<uint4*>(k_lo + t * KP + d) = lo4;
  }
  cp_async_wait<0>();
  __syncthreads();
  if (tile == 0) {
    for (int d = tid; d < D; d += kLocalThreads) {
      float sum = 0.f;
      for (int t = 0; t < n; ++t) sum += __bfloat162float(k_hi[t * KP + d]) + __bfloat162float(k_lo[t * KP + d]);
      a.run_n[(run * a.heads + h) * D + d] = sum;
    }
  }
  // 16 rows of S x 64 columns a job; the tokens past the portion's end are zero rows
  const int g8 = lane >> 2, t4 = lane & 3;
  float* out = a.run_state + (run * a.heads + h) * (size_t)D * V + c0;
  const int jobs = (DP / 16) * (VT / 64), k_steps = (n + 15) / 16;
  for (int job = warp; job < jobs; job += kLocalThreads / 32) {
    const int d0 = (job / (VT / 64)) * 16, cb = (job % (VT / 64)) * 64;
    if (cb >= cols) continue;
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[i][x] = 0.f;
    for (int kk = 0; kk < k_steps; ++kk) {
      const int s_row = kk * 16 + ((lane >> 4) & 1) * 8 + (lane & 7), d_col = d0 + ((lane >> 3) & 1) * 8;
      uint32_t ah[4], al[4];
      ldmatrix_x4_trans(ah, k_hi + s_row * KP + d_col);
      ldmatrix_x4_trans(al, k_lo + s_row * KP + d_col);
      uint32_t b[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        ldmatrix_x4_trans(b[i], v_s + (kk * 16 + (lane & 15)) * VP + cb + i * 16 + ((lane >> 4) << 3));
        mma_bf16(acc[2 * i], ah, b[i][0], b[i][1]);
        mma_bf16(acc[2 * i + 1], ah, b[i][2], b[i][3]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        mma_bf16(acc[2 * i], al, b[i][0], b[i][1]);
        mma_bf16(acc[2 * i + 1], al, b[i][2], b[i][3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int d = d0 + g8 + 8 * half, cc = cb + i * 8 + 2 * t4;
        if (d < D && cc < cols) *reinterpret_cast<float2*>(out + (size_t)d * V + cc) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
      }
  }
}

// grid (elements / 256, entries): S_(r+1) = keep_r S_r + L_r over the entry's chunks; run_state[r] turns from L_r into S_r (run_n
// alike), and the slot gets the last one, with m.
__global__ void __launch_bounds__(256) mem_fold_kernel(MemArgs a) {
  pdl_wait();
  pdl_trigger();
  const int entry = blockIdx.y, H = a.heads, D = a.D;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  const size_t per_head = (size_t)D * a.V / 4, width = per_head * H;            // (pieces of four columns)
  const size_t e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (len <= 0 || e >= width + (size_t)H * D) return;
  const int runs = (len + kMemChunk - 1) / kMemChunk;
  const size_t run0 = mem_first_run(row0, entry);
  float* slot = a.state + (size_t)a.slots[entry] * a.state_stride;
  constexpr int AHEAD = 4;
  if (e < width) {
    const int h = (int)(e / per_head);
    float4* mine = reinterpret_cast<float4*>(slot) + e;
    float4 st = *mine;
    for (int r = 0; r < runs; r += AHEAD) {
      float4 sum[AHEAD];
      float keep[AHEAD];
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        const bool in = r + u < runs;
        sum[u] = in ? reinterpret_cast<const float4*>(a.run_state)[(run0 + r + u) * width + e] : make_float4(0.f, 0.f, 0.f, 0.f);
        keep[u] = in ? a.run_keep[(run0 + r + u) * H + h] : 1.f;
      }
#pragma unroll
      for (int u = 0; u < AHEAD; ++u) {
        if (r + u >= runs) break;
        reinterpret_cast<float4*>(a.run_state)[(run0 + r + u) * width + e] = st;
        st.x = fmaf(keep[u], st.x, sum[u].x); st.y = fmaf(keep[u], st.y, sum[u].y);
        st.z = fmaf(keep[u], st.z, sum[u].z); st.w = fmaf(keep[u], st.w, sum[u].w);
      }
    }
    *mine = st;
    return;
  }
  const int i = (int)(e - width), h = i / D, d = i - h * D;
  float st = mem_norm_state(a, slot, h, 0)[d];
  for (int r = 0; r < runs; ++r) {
    float* at = a.run_n + ((run0 + r) * H + h) * D + d;
    const float sum = *at;
    *at = st;
    st = fmaf(a.run_keep[(run0 + r) * H + h], st, sum);
  }
  const float m_end = a.top[(size_t)h * a.n_tokens + row0 + len - 1];
  for (int tile = 0; tile < a.tiles; ++tile) {
    float* nm = mem_norm_state(a, slot, h, tile);
    nm[d] = st;
    if (d == 0) nm[D] = m_end;
  }
}

constexpr int kOutThreads = 128;
constexpr int kOutRows = 64;           // rows of S in shared memory at a time

static inline size_t mem_out_smem(int dp, int vt) {
  return sizeof(__nv_bfloat16) * ((size_t)2 * kMemChunk * (dp + 8) + (size_t)kMemChunk * (vt + 8) + (size_t)2 * kOutRows * (vt + 8)) +
         sizeof(float) * (size_t)dp;
}

// grid (chunks, heads * tiles, entries): a warp owns sixteen tokens of the chunk.
template <int VT>
__global__ void __launch_bounds__(kOutThreads) mem_out_kernel(MemArgs a) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ MemChunkGates gates;
  pdl_wait();
  pdl_trigger();
  const int D = a.D, V = a.V, H = a.heads, DP = (D + 15) & ~15, KP = DP + 8;
  constexpr int VP = VT + 8;
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(sm_raw);       // [64][KP]
  __nv_bfloat16* k_s = q_s + kMemChunk * KP;                            // [64][KP]
  __nv_bfloat16* v_s = k_s + kMemChunk * KP;                            // [64][VP]
  __nv_bfloat16* s_hi = v_s + kMemChunk * VP;                           // [64][VP]
  __nv_bfloat16* s_lo = s_hi + kOutRows * VP;                           // [64][VP]
  float* n_s = reinterpret_cast<float*>(s_lo + kOutRows * VP);          // [DP]
  const int entry = blockIdx.z, h = blockIdx.y / a.tiles, tile = blockIdx.y - h * a.tiles;
  const int row0 = a.q_start[entry], len = a.q_start[entry + 1] - row0;
  const int t0 = blockIdx.x * kMemChunk;
  if (t0 >= len) return;
  const int n = min(kMemChunk, len - t0);
  const int c0 = tile * kMemTile, cols = min(VT, V - c0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g8 = lane >> 2, t4 = lane & 3, row_base = warp * 16;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj) + (size_t)(row0 + t0) * a.ld;
  for (int e = tid; e < kMemChunk * (DP / 8); e += kOutThreads) {
    const int t = e / (DP / 8), d = (e - t * (DP / 8)) * 8;
    const bool ok = t < n && d < D;
    const __nv_bfloat16* src = ok ? proj + (size_t)t * a.ld + h * D + d : proj;
    cp_async16(q_s + t * KP + d, ok ? src + a.q_off : src, ok);
    cp_async16(k_s + t * KP + d, ok ? src + a.k_off : src, ok);
  }
  for (int e = tid; e < kMemChunk * (VT / 8); e += kOutThreads) {
    const int t = e / (VT / 8), cc = (e - t * (VT / 8)) * 8;
    const bool ok = t < n && cc < cols;
    cp_async16(v_s + t * VP + cc, ok ? proj + (size_t)t * a.ld + a.v_off + h * V + c0 + cc : proj, ok);
  }
  cp_async_commit();
  const size_t run = mem_first_run(row0, entry) + blockIdx.x;
  const float* S = a.run_state + (run * H + h) * (size_t)D * V + c0;
  for (int d = tid; d < DP; d += kOutThreads) n_s[d] = d < D ? a.run_n[(run * H + h) * D + d] : 0.f;
  const float m_start = mem_load_gates(a, gates, h, entry, row0, t0, n);

  // S^T q over the chunk's starting state, 64 rows of S at a time
  float o[VT / 8][4];
#pragma unroll
  for (int i = 0; i < VT / 8; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) o[i][x] = 0.f;
  for (int d0 = 0; d0 < DP; d0 += kOutRows) {
    const int rows = min(kOutRows, DP - d0);
    if (d0 > 0) __syncthreads();                          // the piece before is no longer read
    constexpr int PIECES = VT / 4;
    for (int e = tid; e < rows * PIECES; e += 4 * kOutThreads) {
      float4 got[4];                                       // (four loads of a thread in flight)
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int x = e + u * kOutThreads, d = x / PIECES, cc = (x - d * PIECES) * 4;
        got[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (x < rows * PIECES && d0 + d < D && cc < cols) got[u] = *reinterpret_cast<const float4*>(S + (size_t)(d0 + d) * V + cc);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int x = e + u * kOutThreads, d = x / PIECES, cc = (x - d * PIECES) * 4;
        if (x >= rows * PIECES) break;
        const __nv_bfloat162 h01 = __floats2bfloat162_rn(got[u].x, got[u].y), h23 = __floats2bfloat162_rn(got[u].z, got[u].w);
        const float2 f01 = bf16x2_floats(h01), f23 = bf16x2_floats(h23);
        uint2 hi, lo;
        hi.x = *reinterpret_cast<const uint32_t*>(&h01);
        hi.y = *reinterpret_cast<const uint32_t*>(&h23);
        lo.x = pack_bf16(got[u].x - f01.x, got[u].y - f01.y);
        lo.y = pack_bf16(got[u].z - f23.x, got[u].w - f23.y);
        *reinterpret_cast<uint2*>(s_hi + d * VP + cc) = hi;
        *reinterpret_cast<uint2*>(s_lo + d * VP + cc) = lo;
      }
    }
    cp_async_wait<0>();
    __syncthreads();
    if (row_base < n) {
      for (int kk = 0; kk < rows; kk += 16) {
        uint32_t qa[4];
        ldmatrix_x4(qa, q_s + (row_base + (lane & 15)) * KP + d0 + kk + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < VT / 16; ++i) {
          uint32_t b[4], bl[4];
          ldmatrix_x4_trans(b, s_hi + (kk + (lane & 15)) * VP + i * 16 + ((lane >> 4) << 3));
          ldmatrix_x4_trans(bl, s_lo + (kk + (lane & 15)) * VP + i * 16 + ((lane >> 4) << 3));
          mma_bf16(o[2 * i], qa, b[0], b[1]);
          mma_bf16(o[2 * i + 1], qa, b[2], b[3]);
          mma_bf16(o[2 * i], qa, bl[0], bl[1]);
          mma_bf16(o[2 * i + 1], qa, bl[2], bl[3]);
        }
      }
    }
  }
  if (row_base >= n) return;

  // scores of this warp's tokens against the chunk's keys up to the last of them, and their weights
  float s[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) s[i][x] = 0.f;
  for (int kk = 0; kk < DP; kk += 16) {
    uint32_t qa[4];
    ldmatrix_x4(qa, q_s + (row_base + (lane & 15)) * KP + kk + (lane >> 4) * 8);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j > warp) continue;
      uint32_t b[4];
      ldmatrix_x4(b, k_s + (j * 16 + ((lane >> 4) << 3) + (lane & 7)) * KP + kk + ((lane >> 3) & 1) * 8);
      mma_bf16(s[2 * j], qa, b[0], b[1]);
      mma_bf16(s[2 * j + 1], qa, b[2], b[3]);
    }
  }
  // n_start . q of the sixteen rows: two lanes a row
  float nq_start;
  {
    const int r = row_base + (lane & 15);
    const __nv_bfloat162* q2 = reinterpret_cast<const __nv_bfloat162*>(q_s + r * KP);
    float sum = 0.f;
    for (int d = (lane >> 4); d < DP / 2; d += 2) {
      const float2 f = bf16x2_floats(q2[d]);
      sum = fmaf(f.x, n_s[2 * d], sum);
      sum = fmaf(f.y, n_s[2 * d + 1], sum);
    }
    nq_start = sum + __shfl_xor_sync(0xffffffffu, sum, 16);      // (lane l holds row row_base + (l & 15))
  }
  float bottom[2], start_scale[2];
  uint32_t p_hi[4][4], p_lo[4][4];
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int r = row_base + g8 + 8 * hh;
    const float hi_r = gates.hi[r], lo_r = gates.lo[r], top_r = gates.top[r];
    start_scale[hh] = expf(hi_r + (lo_r + (m_start - top_r))) * a.q_scale;
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int key = i * 8 + 2 * t4 + x;
        float w = 0.f;
        if (key <= r && r < n) w = expf((hi_r - gates.hi[key]) + ((lo_r - gates.lo[key]) + (gates.in[key] - top_r))) * a.q_scale;
        s[i][2 * hh + x] *= w;
        sum += s[i][2 * hh + x];
      }
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    const float nq = fmaf(start_scale[hh], __shfl_sync(0xffffffffu, nq_start, g8 + 8 * hh), sum);
    bottom[hh] = fmaxf(fabsf(nq), expf(-top_r)) + 1e-6f;
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int kk = i >> 1, half = (i & 1) * 2;
    const __nv_bfloat162 h01 = __floats2bfloat162_rn(s[i][0], s[i][1]), h23 = __floats2bfloat162_rn(s[i][2], s[i][3]);
    const float2 f01 = bf16x2_floats(h01), f23 = bf16x2_floats(h23);
    p_hi[kk][half] = *reinterpret_cast<const uint32_t*>(&h01);
    p_hi[kk][half + 1] = *reinterpret_cast<const uint32_t*>(&h23);
    p_lo[kk][half] = pack_bf16(s[i][0] - f01.x, s[i][1] - f01.y);
    p_lo[kk][half + 1] = pack_bf16(s[i][2] - f23.x, s[i][3] - f23.y);
  }
#pragma unroll
  for (int i = 0; i < VT / 8; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) o[i][x] *= start_scale[x >> 1];
#pragma unroll
  for (int kk = 0; kk < 4; ++kk) {
    if (kk > warp) continue;
#pragma unroll
    for (int i = 0; i < VT / 16; ++i) {
      uint32_t b[4];
      ldmatrix_x4_trans(b, v_s + (kk * 16 + (lane & 15)) * VP + i * 16 + ((lane >> 4) << 3));
      mma_bf16(o[2 * i], p_hi[kk], b[0], b[1]);
      mma_bf16(o[2 * i + 1], p_hi[kk], b[2], b[3]);
      mma_bf16(o[2 * i], p_lo[kk], b[0], b[1]);
      mma_bf16(o[2 * i + 1], p_lo[kk], b[2], b[3]);
    }
  }
  // divide; then either leave the rows as they are, or norm the head and gate it
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int r = row_base + g8 + 8 * hh;
    const float by = 1.f / bottom[hh];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VT / 8; ++i)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        o[i][2 * hh + x] *= by;
        ss = fmaf(o[i][2 * hh + x], o[i][2 * hh + x], ss);      // (columns past the head's width are zero)
      }
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if (r >= n) continue;
    const size_t token = (size_t)row0 + t0 + r;
    const size_t at = token * (size_t)H * V + (size_t)h * V + c0;
    if (a.norm_weight) {                                    // (the head is one tile)
      const float inv = 1.f / sqrtf(ss / (float)V + a.eps);
      const __nv_bfloat16* g_row = reinterpret_cast<const __nv_bfloat16*>(a.proj) + token * a.ld + a.g_off + h * V;
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + at;
#pragma unroll
      for (int i = 0; i < VT / 8; ++i) {
        const int cc = i * 8 + 2 * t4;
        if (cc >= cols) continue;
        const float2 g = bf16x2_floats(*reinterpret_cast<const __nv_bfloat162*>(g_row + cc));
        const float2 w = *reinterpret_cast<const float2*>(a.norm_weight + h * V + cc);
        *reinterpret_cast<__nv_bfloat162*>(out + cc) =
            __floats2bfloat162_rn(o[i][2 * hh] * inv * w.x / (1.f + expf(-g.x)), o[i][2 * hh + 1] * inv * w.y / (1.f + expf(-g.y)));
      }
    } else {
      float* out = a.y + at;
#pragma unroll
      for (int i = 0; i < VT / 8; ++i) {
        const int cc = i * 8 + 2 * t4;
        if (cc < cols) *reinterpret_cast<float2*>(out + cc) = make_float2(o[i][2 * hh], o[i][2 * hh + 1]);
      }
    }
  }
}

template <int VT>
static int mem_chunks_launch(const MemArgs& a, int n_entries, int max_q_len, cudaStream_t stream) {
  const int dp = (a.D + 15) & ~15, chunks = ceil_div(max_q_len, kMemChunk);
  const size_t local = mem_local_smem(dp, VT), outs = mem_out_smem(dp, VT);
  if (local > 227 * 1024 || outs > 227 * 1024) return TIB_E_SMEM;
  cudaError_t e = cudaFuncSetAttribute(mem_local_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)local);
  if (e == cudaSuccess) e = cudaFuncSetAttribute(mem_out_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)outs);
  if (e != cudaSuccess) return (int)e;
  const dim3 grid(chunks, a.heads * a.tiles, n_entries);
  TIB_LAUNCH_DEPENDENT(mem_gates_kernel, dim3(a.heads, n_entries), kGateThreads, 0, stream, a);
  TIB_LAUNCH_DEPENDENT(mem_local_kernel<VT>, grid, kLocalThreads, local, stream, a);
  const int64_t pieces = (int64_t)a.heads * a.D * a.V / 4 + (int64_t)a.heads * a.D;
  TIB_LAUNCH_DEPENDENT(mem_fold_kernel, dim3((unsigned)ceil_div64(pieces, 256), n_entries), 256, 0, stream, a);
  TIB_LAUNCH_DEPENDENT(mem_out_kernel<VT>, grid, kOutThreads, outs, stream, a);
  return TIB_OK;
}

template <typename T>
static int mem_walk_launch(const MemArgs& a, int n_entries, cudaStream_t stream) {
  const dim3 grid(a.heads * a.tiles, n_entries);
  const int rows = ceil_div(a.D, kWalkWarps);
#define TIB_WALK(R) TIB_LAUNCH_DEPENDENT((mem_walk_kernel<T, R>), grid, kWalkThreads, 0, stream, a)
  if (rows <= 4) TIB_WALK(4);
  else if (rows <= 8) TIB_WALK(8);
  else if (rows <= 16) TIB_WALK(16);
  else if (rows <= 32) TIB_WALK(32);
  else TIB_WALK(64);
#undef TIB_WALK
  return TIB_OK;
}

}  // namespace tib

using namespace tib;

// Value columns of a tile, tokens of a chunk, the largest key width; whether the chunk form takes these head sizes.
TIB_API int tib_matrix_memory_tile() { return kMemTile; }
TIB_API int tib_matrix_memory_chunk() { return kMemChunk; }
TIB_API int tib_matrix_memory_max_dim() { return kMemMaxDim; }
TIB_API int tib_matrix_memory_takes_chunks(int dim, int vdim) { return dim % 8 == 0 && vdim % 8 == 0 && dim <= 256; }

// proj: rows of `dtype` with q, k, v and the output gate's logits at their offsets; logits [n_tokens, 2 * heads] fp32 (raw gate
// rows, ld_logits apart), or null and x / gate_w [2 * heads, width]; gate_bias [2 * heads]; state: per slot (stride state_stride floats, a
// multiple of 4) heads * D * V + heads * ceil(V / tile) * (D + 1) floats.  norm_weight [heads * V] (V at most a tile): out gets
// the normed and gated rows in `dtype`; null: y gets fp32 rows.  chunks != 0: the chunk form (bf16, logits given), with cum
// [heads, n_tokens] double, log_in and top [heads, n_tokens], top0 [heads, n_entries], run_state [run_capacity, heads, D, V],
// run_n [run_capacity, heads, D], run_keep [run_capacity, heads]; run_capacity >= n_tokens / chunk + n_entries.
TIB_API int tib_matrix_memory(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int g_off, float q_scale,
                              const float* logits, int64_t ld_logits, const void* x, int64_t ldx, const float* gate_w, int width,
                              const float* gate_bias, float cap, float* state, int64_t state_stride, const int* q_start,
                              const int* slots, const float* norm_weight, float eps, float* y, void* out, int heads, int D, int V,
                              int n_entries, int n_tokens, int max_q_len, int chunks, double* cum, float* log_in, float* top,
                              float* top0, float* run_state, float* run_n, float* run_keep, int64_t run_capacity, int dtype,
                              cudaStream_t stream) {
  if (n_entries == 0 || n_tokens == 0 || max_q_len == 0) return TIB_OK;
  if (!proj || !gate_bias || !state || !q_start || !slots || (!y && !out) || (norm_weight && !out) || (!norm_weight && !y)) return TIB_E_ARG;
  if (!logits && (!x || !gate_w || width < 1)) return TIB_E_ARG;
  if (logits && ld_logits < 2 * (int64_t)heads) return TIB_E_SIZE;
  if (heads < 1 || D < 1 || D > kMemMaxDim || V < 1 || !(cap > 0.f) || n_entries > 65535 || state_stride % 4) return TIB_E_SIZE;
  if (dtype != TIB_F32 && dtype != TIB_BF16) return TIB_E_DTYPE;
  MemArgs a = {};
  a.proj = proj; a.ld = ld; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off; a.q_scale = q_scale;
  a.logits = logits; a.ld_logits = ld_logits; a.x = x; a.ldx = ldx; a.gate_w = gate_w; a.width = width; a.gate_bias = gate_bias; a.cap = cap;
  a.state = state; a.state_stride = state_stride; a.q_start = q_start; a.slots = slots; a.norm_weight = norm_weight; a.eps = eps;
  a.y = y; a.out = out; a.heads = heads; a.D = D; a.V = V; a.tiles = ceil_div(V, kMemTile); a.n_tokens = n_tokens;
  a.cum = cum; a.log_in = log_in; a.top = top; a.top0 = top0; a.run_state = run_state; a.run_n = run_n; a.run_keep = run_keep;
  a.n_entries = n_entries;
  if (norm_weight && a.tiles > 1) return TIB_E_SIZE;
  if ((int64_t)heads * a.tiles > 65535) return TIB_E_SIZE;
  if (chunks) {
    if (dtype != TIB_BF16 || !tib_matrix_memory_takes_chunks(D, V)) return TIB_E_SIZE;
    if (!logits || !cum || !log_in || !top || !top0 || !run_state || !run_n || !run_keep) return TIB_E_ARG;
    if (run_capacity < n_tokens / kMemChunk + n_entries) return TIB_E_SIZE;
    if (ld % 8 || q_off % 8 || k_off % 8 || v_off % 8 || g_off % 2 || (((uintptr_t)proj | (uintptr_t)state | (uintptr_t)run_state) & 15) ||
        (norm_weight && ((uintptr_t)norm_weight & 7)))
      return TIB_E_ALIGN;
    return V <= 64 ? mem_chunks_launch<64>(a, n_entries, max_q_len, stream) : mem_chunks_launch<128>(a, n_entries, max_q_len, stream);
  }
  return dtype == TIB_F32 ? mem_walk_launch<float>(a, n_entries, stream) : mem_walk_launch<__nv_bfloat16>(a, n_entries, stream);
}
