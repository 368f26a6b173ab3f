// Layer norms of the 32-bit stream, on their own and behind a branch, and the depth average of a model whose layers read
// a weighted sum of everything that came before them.  All float32; means and variances in two passes over values held
// in registers or shared memory.
//
// layer_norm: out[r] = (x - mean) / sqrt(var + eps) * w (+ b) with x = row rows[r] (or r), var the mean of the squared
//   deviations, rounded once to the output's type.
// layer_norm_add: what a block does that norms a branch before it joins the stream, one kernel per branch:
//     x <- x + n(branch),   next = n'(x)
//   `branch` is a zeroed buffer that products added into and is handed back zeroed; `copy` receives the new stream in
//   bfloat16, and `next`, where asked for, what the norm ahead of the following branch makes of it (the same sums in the
//   same order as layer_norm's, so that it does not matter which kernel made them).
// post_norm_join: what a block does that norms the SUM of the stream and a branch (post-norm), one kernel per branch:
//     y = n(alpha * x + branch + out_bias),   x <- y
//   `branch` is a zeroed buffer that products added into and is handed back zeroed; `copy` receives the new stream in
//   bfloat16 for the next branch to read.  With stages X_0 .. X_(n-1) (stage j of row r at stages + j * stage_stride +
//   r * hidden) the row's result y is the next stage, stored behind them when `keep` says that a later layer reads it, and
//   what goes on is the depth average
//     x <- mix[0] X_0 + ... + mix[n-1] X_(n-1) + mix[n] y.
//   The stages' sum does not wait for the row's statistics: its loads are in flight while they are taken.
// depth_average: the same average behind a layer whose block does not norm the sum: x is the result, stored and averaged.
// row_add: x[r, :] += bias.
#include "common.cuh"

TLLM_DEFINE_LAST_ERROR

namespace tllm {

struct JoinArgs {
  float* branch;            // [rows, hidden]
  float* x;                 // [rows, hidden]: the stream, in place
  const float* out_bias;    // [hidden] or null
  const float *w, *b;       // [hidden]
  float alpha, eps;
  __nv_bfloat16* copy;      // [rows, hidden] or null
  float* stages;            // null: no depth average
  long long stage_stride;
  int n_stages, keep;
  const float* mix;         // [n_stages + 1]
  int n_rows, hidden;
};

__device__ __forceinline__ float4 fma4(float s, float4 v, float4 a) {
  return make_float4(fmaf(s, v.x, a.x), fmaf(s, v.y, a.y), fmaf(s, v.z, a.z), fmaf(s, v.w, a.w));
}

// Mean of a row of 4 * n4 values that the block holds in registers (thread t's i-th piece is piece t + i * blockDim; pieces
// past the row are zero) and its summed squared deviations, with ONE barrier: every warp takes those of its own values
// (shuffles only), and the warps' pairs are joined by
//   mean = sum_w n_w mean_w / N,   M2 = sum_w (M2_w + n_w (mean_w - mean)^2).
template <int VEC>
__device__ __forceinline__ void row_moments(const float4* z, int n4, float2* moments, float* counts, float& mean, float& m2) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float sum = 0.f, count = 0.f;
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    sum += (z[i].x + z[i].y) + (z[i].z + z[i].w);
    count += 4.f * fminf(32.f, fmaxf(0.f, (float)(n4 - (warp * 32 + i * (int)blockDim.x))));
  }
  const float own_mean = count > 0.f ? warp_sum(sum) / count : 0.f;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    if (threadIdx.x + i * blockDim.x < n4) {
      const float dx = z[i].x - own_mean, dy = z[i].y - own_mean, dz = z[i].z - own_mean, dw = z[i].w - own_mean;
      ss += (dx * dx + dy * dy) + (dz * dz + dw * dw);
    }
  }
  ss = warp_sum(ss);
  if (lane == 0) { moments[warp] = make_float2(own_mean, ss); counts[warp] = count; }
  __syncthreads();
  const bool has = lane < (int)(blockDim.x >> 5);
  const float2 pair = has ? moments[lane] : make_float2(0.f, 0.f);
  const float cnt = has ? counts[lane] : 0.f;
  mean = warp_sum(cnt * pair.x) / (4.f * (float)n4);
  const float off = pair.x - mean;
  m2 = warp_sum(fmaf(cnt * off, off, pair.y));
}

__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float4 v) {
  uint2 pk;
  *reinterpret_cast<__nv_bfloat162*>(&pk.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&pk.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = pk;
}

// (z - mean) * inv * w + b
__device__ __forceinline__ float4 norm4(float4 z, float mean, float inv, float4 w, float4 b) {
  return make_float4(fmaf((z.x - mean) * inv, w.x, b.x), fmaf((z.y - mean) * inv, w.y, b.y),
                     fmaf((z.z - mean) * inv, w.z, b.z), fmaf((z.w - mean) * inv, w.w, b.w));
}
__device__ __forceinline__ float4 ldg4_or(const float* p, int idx, float4 other) {
  return p != nullptr ? __ldg(reinterpret_cast<const float4*>(p) + idx) : other;
}

// The threads of a row depend on the width alone, so that a row's sums have the same order in every batch.
inline int row_threads(int n4) { return n4 <= 128 ? (n4 + 31) / 32 * 32 : (n4 <= 512 ? 256 : 512); }

// Rows in registers: hidden a multiple of 4, at most 4 * VEC * blockDim.
template <int VEC>
__global__ void post_norm_join_vec_kernel(JoinArgs a) {
  __shared__ float2 moments[32];
  __shared__ float counts[32];
  pdl_trigger();
  const int n4 = a.hidden / 4, r = blockIdx.x;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 ob[VEC];   // constants of the model are read ahead of the wait
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    ob[i] = a.out_bias != nullptr && idx < n4 ? __ldg(reinterpret_cast<const float4*>(a.out_bias) + idx) : zero;
  }
  pdl_wait();
  if (r >= a.n_rows) return;
  float4* br = reinterpret_cast<float4*>(a.branch + (size_t)r * a.hidden);
  float4* xr = reinterpret_cast<float4*>(a.x + (size_t)r * a.hidden);
  float4 z[VEC], acc[VEC], v[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    v[i] = idx < n4 ? br[idx] : zero;
    z[i] = idx < n4 ? xr[idx] : zero;
    acc[i] = zero;
  }
  if (a.stages != nullptr) {
#pragma unroll 4
    for (int j = 0; j < a.n_stages; ++j) {
      const float4* st = reinterpret_cast<const float4*>(a.stages + j * a.stage_stride + (size_t)r * a.hidden);
      const float m = a.mix[j];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const int idx = threadIdx.x + i * blockDim.x;
        if (idx < n4) acc[i] = fma4(m, st[idx], acc[i]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    z[i] = fma4(a.alpha, z[i], make_float4(v[i].x + ob[i].x, v[i].y + ob[i].y, v[i].z + ob[i].z, v[i].w + ob[i].w));
  }
  float mean, m2;
  row_moments<VEC>(z, n4, moments, counts, mean, m2);
  const float inv = 1.f / sqrtf(m2 / (float)a.hidden + a.eps);
  const float last = a.stages != nullptr ? a.mix[a.n_stages] : 0.f;
  float4* own = a.stages != nullptr ? reinterpret_cast<float4*>(a.stages + a.n_stages * a.stage_stride + (size_t)r * a.hidden) : nullptr;
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    if (idx >= n4) continue;
    const float4 w = __ldg(reinterpret_cast<const float4*>(a.w) + idx), b = __ldg(reinterpret_cast<const float4*>(a.b) + idx);
    float4 y = make_float4(fmaf((z[i].x - mean) * inv, w.x, b.x), fmaf((z[i].y - mean) * inv, w.y, b.y),
                           fmaf((z[i].z - mean) * inv, w.z, b.z), fmaf((z[i].w - mean) * inv, w.w, b.w));
    if (own != nullptr) {
      if (a.keep) own[idx] = y;
      y = fma4(last, y, acc[i]);
    }
    xr[idx] = y;
    br[idx] = zero;
    if (a.copy != nullptr) put4(a.copy + (size_t)r * a.hidden + 4 * idx, y);
  }
}

// Any width: the row waits in shared memory.
__global__ void post_norm_join_kernel(JoinArgs a) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  if (r >= a.n_rows) return;
  float* br = a.branch + (size_t)r * a.hidden;
  float* xr = a.x + (size_t)r * a.hidden;
  float sum = 0.f;
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {   // a thread meets the same elements in every pass
    const float z = fmaf(a.alpha, xr[i], br[i] + (a.out_bias ? a.out_bias[i] : 0.f));
    br[i] = 0.f;
    row[i] = z;
    sum += z;
  }
  const float mean = block_sum(sum, scratch) / (float)a.hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {
    const float d = row[i] - mean;
    row[i] = d;
    ss += d * d;
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / (float)a.hidden + a.eps);
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {
    float y = fmaf(row[i] * inv, a.w[i], a.b[i]);
    if (a.stages != nullptr) {
      float acc = 0.f;
      for (int j = 0; j < a.n_stages; ++j) acc = fmaf(a.mix[j], a.stages[j * a.stage_stride + (size_t)r * a.hidden + i], acc);
      if (a.keep) a.stages[a.n_stages * a.stage_stride + (size_t)r * a.hidden + i] = y;
      y = fmaf(a.mix[a.n_stages], y, acc);
    }
    xr[i] = y;
    if (a.copy) a.copy[(size_t)r * a.hidden + i] = __float2bfloat16_rn(y);
  }
}

template <typename T, int VEC>
__global__ void layer_norm_vec_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b,
                                      T* __restrict__ out, const int* __restrict__ rows, int n_rows, int hidden, float eps) {
  __shared__ float2 moments[32];
  __shared__ float counts[32];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x, n4 = hidden / 4;
  if (r >= n_rows) return;
  const float4* src = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * hidden);
  float4 z[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    z[i] = idx < n4 ? src[idx] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float mean, m2;
  row_moments<VEC>(z, n4, moments, counts, mean, m2);
  const float inv = 1.f / sqrtf(m2 / (float)hidden + eps);
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    if (idx >= n4) continue;
    const float4 wv = __ldg(reinterpret_cast<const float4*>(w) + idx), bv = ldg4_or(b, idx, make_float4(0.f, 0.f, 0.f, 0.f));
    put4(out + (size_t)r * hidden + 4 * idx, norm4(z[i], mean, inv, wv, bv));
  }
}

template <typename T>
__global__ void layer_norm_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b,
                                  T* __restrict__ out, const int* __restrict__ rows, int n_rows, int hidden, float eps) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  const float* src = x + (size_t)(rows ? rows[r] : r) * hidden;
  float sum = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    row[i] = src[i];
    sum += row[i];
  }
  const float mean = block_sum(sum, scratch) / (float)hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float d = row[i] - mean;
    row[i] = d;
    ss += d * d;
  }
  ss = block_sum(ss, scratch);
  const float inv = 1.f / sqrtf(ss / (float)hidden + eps);
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[(size_t)r * hidden + i] = from_f32<T>(fmaf(row[i] * inv, w[i], b ? b[i] : 0.f));
}

struct AddArgs {
  float* branch;            // [rows, hidden]
  float* x;                 // [rows, hidden]: the stream, in place
  const float *w, *b;       // [hidden]; b may be null
  float eps;
  __nv_bfloat16* copy;      // [rows, hidden] or null
  void* next;               // [rows, hidden] or null: the following norm's output
  const float *next_w, *next_b;
  float next_eps;
  int n_rows, hidden;
};

template <typename T, int VEC>
__global__ void layer_norm_add_vec_kernel(AddArgs a) {
  __shared__ float2 moments[2][32];
  __shared__ float counts[2][32];
  pdl_trigger();
  const int n4 = a.hidden / 4, r = blockIdx.x;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 w[VEC];   // constants of the model are read ahead of the wait
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    w[i] = idx < n4 ? __ldg(reinterpret_cast<const float4*>(a.w) + idx) : zero;
  }
  pdl_wait();
  if (r >= a.n_rows) return;
  float4* br = reinterpret_cast<float4*>(a.branch + (size_t)r * a.hidden);
  float4* xr = reinterpret_cast<float4*>(a.x + (size_t)r * a.hidden);
  float4 z[VEC], x[VEC];
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    z[i] = idx < n4 ? br[idx] : zero;
    x[i] = idx < n4 ? xr[idx] : zero;
  }
  float mean, m2;
  row_moments<VEC>(z, n4, moments[0], counts[0], mean, m2);
  float inv = 1.f / sqrtf(m2 / (float)a.hidden + a.eps);
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    if (idx >= n4) continue;
    const float4 y = norm4(z[i], mean, inv, w[i], ldg4_or(a.b, idx, zero));
    x[i] = make_float4(x[i].x + y.x, x[i].y + y.y, x[i].z + y.z, x[i].w + y.w);
    xr[idx] = x[i];
    br[idx] = zero;
    if (a.copy != nullptr) put4(a.copy + (size_t)r * a.hidden + 4 * idx, x[i]);
  }
  if (a.next == nullptr) return;
  row_moments<VEC>(x, n4, moments[1], counts[1], mean, m2);
  inv = 1.f / sqrtf(m2 / (float)a.hidden + a.next_eps);
#pragma unroll
  for (int i = 0; i < VEC; ++i) {
    const int idx = threadIdx.x + i * blockDim.x;
    if (idx >= n4) continue;
    put4((T*)a.next + (size_t)r * a.hidden + 4 * idx,
         norm4(x[i], mean, inv, __ldg(reinterpret_cast<const float4*>(a.next_w) + idx), ldg4_or(a.next_b, idx, zero)));
  }
}

// Mean of a row in shared memory, which becomes the row of deviations (a thread meets the same elements in every pass);
// returns 1 / sqrt(var + eps).
__device__ __forceinline__ float center_row(float* row, int hidden, float eps, float* scratch) {
  float sum = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) sum += row[i];
  const float mean = block_sum(sum, scratch) / (float)hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float d = row[i] - mean;
    row[i] = d;
    ss += d * d;
  }
  ss = block_sum(ss, scratch);
  return 1.f / sqrtf(ss / (float)hidden + eps);
}

// Any width: the row waits in shared memory.
template <typename T>
__global__ void layer_norm_add_kernel(AddArgs a) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  pdl_trigger();
  pdl_wait();
  const int r = blockIdx.x;
  if (r >= a.n_rows) return;
  float* br = a.branch + (size_t)r * a.hidden;
  float* xr = a.x + (size_t)r * a.hidden;
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) { row[i] = br[i]; br[i] = 0.f; }
  float inv = center_row(row, a.hidden, a.eps, scratch);
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x) {
    const float x = xr[i] + fmaf(row[i] * inv, a.w[i], a.b ? a.b[i] : 0.f);
    xr[i] = x;
    row[i] = x;
    if (a.copy) a.copy[(size_t)r * a.hidden + i] = __float2bfloat16_rn(x);
  }
  if (a.next == nullptr) return;
  inv = center_row(row, a.hidden, a.next_eps, scratch);
  for (int i = threadIdx.x; i < a.hidden; i += blockDim.x)
    ((T*)a.next)[(size_t)r * a.hidden + i] = from_f32<T>(fmaf(row[i] * inv, a.next_w[i], a.next_b ? a.next_b[i] : 0.f));
}

__global__ void depth_average_kernel(float* __restrict__ x, float* __restrict__ stages, long long stage_stride, int n_stages,
                                     int keep, const float* __restrict__ mix, long long n) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const float y = x[i];
    float acc = 0.f;
    for (int j = 0; j < n_stages; ++j) acc = fmaf(mix[j], stages[j * stage_stride + i], acc);
    if (keep) stages[n_stages * stage_stride + i] = y;
    x[i] = fmaf(mix[n_stages], y, acc);
  }
}

__global__ void row_add_kernel(float* __restrict__ x, const float* __restrict__ bias, long long n, int hidden) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
    x[i] += bias[i % hidden];
}

constexpr int MAX_WIDTH = (48 * 1024 - 256) / 4;   // values of a row that waits in shared memory beside the sums' scratch

}  // namespace tllm

using namespace tllm;

extern "C" int tllm_post_norm_join(float* branch, float* x, const float* out_bias, const float* w, const float* b, float alpha,
                                   float eps, void* copy_bf16, float* stages, long long stage_stride, int n_stages, int keep,
                                   const float* mix, int n_rows, int hidden, void* stream) {
  TLLM_REQUIRE(n_rows > 0 && hidden > 0 && branch && x && w && b, "post_norm_join: %d rows of %d values", n_rows, hidden);
  TLLM_REQUIRE(stages == nullptr || (mix != nullptr && n_stages >= 0), "post_norm_join: a depth average of %d stages needs weights", n_stages);
  JoinArgs a;
  a.branch = branch; a.x = x; a.out_bias = out_bias; a.w = w; a.b = b; a.alpha = alpha; a.eps = eps;
  a.copy = (__nv_bfloat16*)copy_bf16; a.stages = stages; a.stage_stride = stage_stride; a.n_stages = n_stages; a.keep = keep;
  a.mix = mix; a.n_rows = n_rows; a.hidden = hidden;
  cudaStream_t s = (cudaStream_t)stream;
  const auto off = [](const void* p, int to) { return ((uintptr_t)p % to) != 0; };
  if (hidden % 4 == 0 && hidden <= 4 * 4 * 512 && !off(branch, 16) && !off(x, 16) && !off(out_bias, 16) && !off(w, 16) && !off(b, 16) &&
      !off(copy_bf16, 8) && !off(stages, 16) && stage_stride % 4 == 0) {
    const int n4 = hidden / 4, threads = row_threads(n4);
    const int vec = (n4 + threads - 1) / threads;
    if (vec <= 1) TLLM_LAUNCH("post_norm_join", post_norm_join_vec_kernel<1>, n_rows, threads, 0, s, a);
    else if (vec == 2) TLLM_LAUNCH("post_norm_join", post_norm_join_vec_kernel<2>, n_rows, threads, 0, s, a);
    else TLLM_LAUNCH("post_norm_join", post_norm_join_vec_kernel<4>, n_rows, threads, 0, s, a);
    return TLLM_OK;
  }
  TLLM_REQUIRE(hidden <= MAX_WIDTH, "post_norm_join: rows of %d values (at most %d)", hidden, MAX_WIDTH);
  const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
  TLLM_LAUNCH("post_norm_join", post_norm_join_kernel, n_rows, threads, hidden * 4, s, a);
  return TLLM_OK;
}

template <typename T>
static int launch_layer_norm(const float* x, const float* w, const float* b, T* out, const int* rows, int n_rows, int hidden,
                             float eps, cudaStream_t s) {
  const auto aligned = [](const void* p) { return ((uintptr_t)p % 16) == 0; };   // (null is)
  if (hidden % 4 == 0 && hidden <= 4 * 4 * 512 && aligned(x) && aligned(w) && aligned(b) && aligned(out)) {
    const int n4 = hidden / 4, threads = row_threads(n4), vec = (n4 + threads - 1) / threads;
    if (vec <= 1) TLLM_LAUNCH("layer_norm", (layer_norm_vec_kernel<T, 1>), n_rows, threads, 0, s, x, w, b, out, rows, n_rows, hidden, eps);
    else if (vec == 2) TLLM_LAUNCH("layer_norm", (layer_norm_vec_kernel<T, 2>), n_rows, threads, 0, s, x, w, b, out, rows, n_rows, hidden, eps);
    else TLLM_LAUNCH("layer_norm", (layer_norm_vec_kernel<T, 4>), n_rows, threads, 0, s, x, w, b, out, rows, n_rows, hidden, eps);
    return TLLM_OK;
  }
  TLLM_REQUIRE(hidden <= MAX_WIDTH, "layer_norm: rows of %d values (at most %d)", hidden, MAX_WIDTH);
  const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
  TLLM_LAUNCH("layer_norm", layer_norm_kernel<T>, n_rows, threads, hidden * 4, s, x, w, b, out, rows, n_rows, hidden, eps);
  return TLLM_OK;
}

extern "C" int tllm_layer_norm(const float* x, const float* w, const float* b, void* out, const int* rows, int n_rows,
                               int hidden, float eps, int out_dtype, void* stream) {
  TLLM_REQUIRE(n_rows > 0 && hidden > 0, "layer_norm: %d rows of %d values", n_rows, hidden);
  cudaStream_t s = (cudaStream_t)stream;
  if (out_dtype == TLLM_F32) return launch_layer_norm<float>(x, w, b, (float*)out, rows, n_rows, hidden, eps, s);
  if (out_dtype == TLLM_BF16) return launch_layer_norm<__nv_bfloat16>(x, w, b, (__nv_bfloat16*)out, rows, n_rows, hidden, eps, s);
  TLLM_FAIL(TLLM_ERR_ARG, "layer_norm: unknown dtype code %d", out_dtype);
}

template <typename T>
static int launch_layer_norm_add(const AddArgs& a, cudaStream_t s) {
  const auto off = [](const void* p, int to) { return ((uintptr_t)p % to) != 0; };
  if (a.hidden % 4 == 0 && a.hidden <= 4 * 4 * 512 && !off(a.branch, 16) && !off(a.x, 16) && !off(a.w, 16) && !off(a.b, 16) &&
      !off(a.copy, 8) && !off(a.next, 16) && !off(a.next_w, 16) && !off(a.next_b, 16)) {
    const int n4 = a.hidden / 4, threads = row_threads(n4), vec = (n4 + threads - 1) / threads;
    if (vec <= 1) TLLM_LAUNCH("layer_norm_add", (layer_norm_add_vec_kernel<T, 1>), a.n_rows, threads, 0, s, a);
    else if (vec == 2) TLLM_LAUNCH("layer_norm_add", (layer_norm_add_vec_kernel<T, 2>), a.n_rows, threads, 0, s, a);
    else TLLM_LAUNCH("layer_norm_add", (layer_norm_add_vec_kernel<T, 4>), a.n_rows, threads, 0, s, a);
    return TLLM_OK;
  }
  TLLM_REQUIRE(a.hidden <= MAX_WIDTH, "layer_norm_add: rows of %d values (at most %d)", a.hidden, MAX_WIDTH);
  const int threads = a.hidden >= 2048 ? 512 : (a.hidden >= 512 ? 256 : 128);
  TLLM_LAUNCH("layer_norm_add", layer_norm_add_kernel<T>, a.n_rows, threads, a.hidden * 4, s, a);
  return TLLM_OK;
}

// next (of next_dtype), next_w, next_b, next_eps: the norm ahead of the following branch; next null: none.
extern "C" int tllm_layer_norm_add(float* branch, float* x, const float* w, const float* b, float eps, void* copy_bf16,
                                   void* next, const float* next_w, const float* next_b, float next_eps, int next_dtype,
                                   int n_rows, int hidden, void* stream) {
  TLLM_REQUIRE(n_rows > 0 && hidden > 0 && branch && x && w, "layer_norm_add: %d rows of %d values", n_rows, hidden);
  TLLM_REQUIRE(next == nullptr || next_w != nullptr, "layer_norm_add: the following norm needs a weight");
  AddArgs a;
  a.branch = branch; a.x = x; a.w = w; a.b = b; a.eps = eps; a.copy = (__nv_bfloat16*)copy_bf16; a.next = next;
  a.next_w = next_w; a.next_b = next_b; a.next_eps = next_eps; a.n_rows = n_rows; a.hidden = hidden;
  cudaStream_t s = (cudaStream_t)stream;
  if (next_dtype == TLLM_F32) return launch_layer_norm_add<float>(a, s);
  if (next_dtype == TLLM_BF16) return launch_layer_norm_add<__nv_bfloat16>(a, s);
  TLLM_FAIL(TLLM_ERR_ARG, "layer_norm_add: unknown dtype code %d", next_dtype);
}

extern "C" int tllm_depth_average(float* x, float* stages, long long stage_stride, int n_stages, int keep, const float* mix,
                                  long long n, void* stream) {
  TLLM_REQUIRE(n > 0 && n_stages >= 0 && x && stages && mix, "depth_average: %lld values, %d stages", n, n_stages);
  const int threads = 256;
  const long long want = (n + threads - 1) / threads;
  TLLM_LAUNCH("depth_average", depth_average_kernel, (unsigned)(want < 148 * 16 ? want : 148 * 16), threads, 0, (cudaStream_t)stream, x, stages, stage_stride, n_stages, keep, mix, n);
  return TLLM_OK;
}

extern "C" int tllm_row_add(float* x, const float* bias, long long n_rows, int hidden, void* stream) {
  TLLM_REQUIRE(n_rows > 0 && hidden > 0 && x && bias, "row_add: %lld rows of %d values", n_rows, hidden);
  const int threads = 256;
  const long long n = n_rows * hidden, want = (n + threads - 1) / threads;
  TLLM_LAUNCH("row_add", row_add_kernel, (unsigned)(want < 148 * 16 ? want : 148 * 16), threads, 0, (cudaStream_t)stream, x, bias, n, hidden);
  return TLLM_OK;
}
