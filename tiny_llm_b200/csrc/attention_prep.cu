// What lies between the input projection of an attention and its score kernel, and behind the score kernel, for
// attentions without the rotate-half form: biases, norms per head, a position-dependent stretch of the query, the
// latent form of keys and values, and output gates.  All statistics, angles and factors are 32-bit.
//
// qk_norm_kv_write: rows of the projection are [nq query heads | nkv key heads] of kd values, then nkv value heads of
//   vd values.  Optional biases are added; query and key heads are divided by sqrt(mean(x^2) + eps) and multiplied by
//   a weight of kd values shared by the heads (no weights: no norm); the query is further multiplied by
//   1 + coef * ln(floor((p + 1) / every) + 1) at position p (every = 0: not).  With a frequency table the first
//   rot_dims values of every query and key head are then turned by p * freq[i], value i with i + rot_dims / 2 or value
//   2i with 2i + 1, cos and sin times a constant.  Queries are rewritten in place, keys and values go to their pages.
//   One warp per head row.
// latent_kv_write: rows are [nq query heads of (nd plain | rd rotated) values | rank latent values | rd rotated key
//   values | ...].  The latent is normed (weight of rank values) and written both as the first `rank` values of the
//   token's key row and as its value row; the key's rotated part and every query head's rotated part are turned in
//   pairs (2i, 2i + 1) or halves (i, i + rot_dims / 2), i < rot_dims / 2, by p * freq[i]; the key part goes behind the
//   latent in the key row, the query parts to q_out[t, head, rank : rank + rd].  (The plain query parts reach q_out through a product with the
//   keys' up-projection, which is not this kernel's.)
// conv_norm_kv_write: rows are [nq query heads | nkv key heads] of kd values, then nkv value heads of vd values, all of
//   them channels of a short causal filter over time: y_t[c] = sum_j taps[j, c] x_(t - n_taps + 1 + j)[c] with x the
//   projection plus its bias, zero before the sequence's start; the last n_taps - 1 inputs of every channel are the
//   request's state.  The filtered queries TOGETHER (all heads of the token) are divided by sqrt(mean(y^2) + eps) and
//   multiplied by a weight per channel, and so are the keys.  With a frequency table the first rot_dims values of every
//   query and key head are then turned as in qk_norm_kv_write (a token's cosines and sines are taken once for all its
//   heads).  Queries go to a buffer of their own (other tokens' filters still read the projection), keys and values to
//   their pages.
// sigmoid_gate: out[t, h, :] = x[t, h, :] * sigmoid(gate), the gate one value per element or one per head.
#include "common.cuh"

TLLM_DEFINE_LAST_ERROR

namespace tllm {

constexpr int MAX_ROW = 512;   // values of a head row or of the latent

struct QkArgs {
  void* proj;
  int ld, nq, nkv, kd, vd;
  const float *bq, *bk, *bv;    // biases [nq * kd], [nkv * kd], [nkv * vd] or null
  const float *wq, *wk;         // norm weights [kd] or null
  float eps, coef;
  int every;
  const int* positions;
  void *kcache, *vcache;
  const int* slot_mapping;
  int page_size;
  long long k_page_stride, k_head_stride, v_page_stride, v_head_stride;
  int n_tokens;
  const float* freq;            // [rot_dims / 2] or null: query and key heads are rotated behind the norm
  int rot_dims, rot_pairs;      // the first rot_dims values of a head turn; pairs (2i, 2i + 1) or halves (i, i + rot_dims / 2)
  float rot_mag;                // cos and sin are multiplied by this
};

template <typename T>
__global__ void __launch_bounds__(128) qk_norm_kv_write_kernel(QkArgs a) {
  __shared__ float turned[4][MAX_ROW];
  pdl_trigger();
  pdl_wait();
  const int rows = a.nq + 2 * a.nkv;
  const long long task = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (task >= (long long)a.n_tokens * rows) return;
  const int lane = threadIdx.x & 31;
  const int t = (int)(task / rows), r = (int)(task % rows);
  T* row = (T*)a.proj + (size_t)t * a.ld;
  const int slot = a.slot_mapping[t];
  const long long page = slot / a.page_size, off = slot % a.page_size;
  if (r >= a.nq + a.nkv) {   // a value head: bias, then to its page
    if (slot < 0) return;
    const int h = r - a.nq - a.nkv;
    const T* src = row + (size_t)(a.nq + a.nkv) * a.kd + (size_t)h * a.vd;
    T* dst = (T*)a.vcache + page * a.v_page_stride + (long long)h * a.v_head_stride + off * a.vd;
    for (int d = lane; d < a.vd; d += 32)
      dst[d] = from_f32<T>(to_f32(src[d]) + (a.bv ? a.bv[h * a.vd + d] : 0.f));
    return;
  }
  const bool is_q = r < a.nq;
  if (!is_q && slot < 0) return;
  const int h = is_q ? r : r - a.nq;
  const float* bias = is_q ? a.bq : a.bk;
  const float* w = is_q ? a.wq : a.wk;
  T* src = row + (size_t)r * a.kd;
  float x[MAX_ROW / 32];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAX_ROW / 32; ++i) {
    const int d = lane + 32 * i;
    x[i] = d < a.kd ? to_f32(src[d]) + (bias ? bias[h * a.kd + d] : 0.f) : 0.f;
    ss = fmaf(x[i], x[i], ss);
  }
  float f = 1.f;
  if (w) f = 1.f / sqrtf(warp_sum(ss) / (float)a.kd + a.eps);
  float stretch = 1.f;
  if (is_q && a.every > 0) stretch = fmaf(a.coef, logf((float)((a.positions[t] + 1) / a.every + 1)), 1.f);
  T* dst = is_q ? src : (T*)a.kcache + page * a.k_page_stride + (long long)h * a.k_head_stride + off * a.kd;
  float* mine = turned[threadIdx.x >> 5];
#pragma unroll
  for (int i = 0; i < MAX_ROW / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < a.kd) {
      float y = w ? __fmul_rn(__fmul_rn(x[i], f), w[d]) : x[i];
      if (is_q) y = __fmul_rn(y, stretch);
      if (a.rot_dims > 0) mine[d] = y;
      else dst[d] = from_f32<T>(y);
    }
  }
  if (a.rot_dims == 0) return;
  // the rotation reads the normed values in 32-bit (the partner of a value lies with another lane) and rounds once
  __syncwarp();
  const float pos = (float)a.positions[t];
  const int half = a.rot_dims / 2;
  for (int d = lane; d < a.kd; d += 32) {
    float y = mine[d];
    if (d < a.rot_dims) {
      const int i = a.rot_pairs ? d >> 1 : (d < half ? d : d - half);
      const bool first = a.rot_pairs ? !(d & 1) : d < half;
      const float u = mine[a.rot_pairs ? 2 * i : i], v = mine[a.rot_pairs ? 2 * i + 1 : i + half];
      const float ang = __fmul_rn(pos, a.freq[i]);
      const float c = __fmul_rn(cosf(ang), a.rot_mag), sn = __fmul_rn(sinf(ang), a.rot_mag);
      y = first ? fmaf(u, c, -__fmul_rn(v, sn)) : fmaf(v, c, __fmul_rn(u, sn));
    }
    dst[d] = from_f32<T>(y);
  }
}

struct LatentArgs {
  const void* proj;
  int ld, nq, nd, rd, rank, rot_dims;
  const float* w_latent;     // [rank]
  const float* freq;         // [rot_dims / 2]
  float eps;
  const int* positions;
  void* q_out;               // [T, nq, rank + rd]
  void *kcache, *vcache;     // key rows of rank + rd values, value rows of rank values, one head
  const int* slot_mapping;
  int page_size;
  long long k_page_stride, v_page_stride;
  int n_tokens;
  float rot_mag;             // cos and sin are multiplied by this
  int rot_pairs;             // pairs (2i, 2i + 1), or halves (i, i + rot_dims / 2)
};

// With kcache == null the rows hold queries only: their rotated parts are turned and nothing is written to a cache
// (a mixer that reads the latents and key parts another layer cached).
// One CTA of 128 threads per token: warp 0 norms the latent, all threads turn the rotated parts.
template <typename T>
__global__ void __launch_bounds__(128) latent_kv_write_kernel(LatentArgs a) {
  __shared__ float cs[256], sn[256];   // rot_dims / 2 <= 256
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  if (t >= a.n_tokens) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float pos = (float)a.positions[t];
  for (int i = threadIdx.x; i < a.rot_dims / 2; i += blockDim.x) {
    const float ang = __fmul_rn(pos, a.freq[i]);
    cs[i] = __fmul_rn(cosf(ang), a.rot_mag);
    sn[i] = __fmul_rn(sinf(ang), a.rot_mag);
  }
  __syncthreads();
  const T* row = (const T*)a.proj + (size_t)t * a.ld;
  const int qd = a.nd + a.rd, kd = a.rank + a.rd;
  const T* lat = row + (size_t)a.nq * qd;
  const bool writes = a.kcache != nullptr;
  const int slot = writes ? a.slot_mapping[t] : -1;
  const long long page = slot / a.page_size, off = slot % a.page_size;
  T* krow = (T*)a.kcache + page * a.k_page_stride + off * kd;
  T* vrow = (T*)a.vcache + page * a.v_page_stride + off * a.rank;
  if (warp == 0 && slot >= 0) {
    float x[MAX_ROW / 32];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < MAX_ROW / 32; ++i) {
      const int d = lane + 32 * i;
      x[i] = d < a.rank ? to_f32(lat[d]) : 0.f;
      ss = fmaf(x[i], x[i], ss);
    }
    const float f = 1.f / sqrtf(warp_sum(ss) / (float)a.rank + a.eps);
#pragma unroll
    for (int i = 0; i < MAX_ROW / 32; ++i) {
      const int d = lane + 32 * i;
      if (d < a.rank) {
        const T y = from_f32<T>(__fmul_rn(__fmul_rn(x[i], f), a.w_latent[d]));
        krow[d] = y;
        vrow[d] = y;
      }
    }
  }
  // rotated parts: unit 0 is the key's, unit 1 + h query head h's
  const int half_rot = a.rot_dims / 2;
  if (!a.rot_pairs) {   // a unit's items: half_rot halves (i, i + half_rot), then the values that do not turn
    const int items = a.rd - half_rot;
    for (int idx = threadIdx.x; idx < (a.nq + 1) * items; idx += blockDim.x) {
      const int u = idx / items, i = idx % items;
      if (u == 0 && slot < 0) continue;
      const T* src = u == 0 ? lat + a.rank : row + (size_t)(u - 1) * qd + a.nd;
      T* dst = u == 0 ? krow + a.rank : (T*)a.q_out + ((size_t)t * a.nq + (u - 1)) * kd + a.rank;
      if (i < half_rot) {
        const float x = to_f32(src[i]), y = to_f32(src[i + half_rot]), c = cs[i], s = sn[i];
        dst[i] = from_f32<T>(fmaf(x, c, -__fmul_rn(y, s)));
        dst[i + half_rot] = from_f32<T>(fmaf(y, c, __fmul_rn(x, s)));
      } else {
        dst[i + half_rot] = src[i + half_rot];
      }
    }
    return;
  }
  const int half = (a.rd + 1) / 2;
  for (int idx = threadIdx.x; idx < (a.nq + 1) * half; idx += blockDim.x) {
    const int u = idx / half, i = idx % half;
    if (u == 0 && slot < 0) continue;
    const T* src = (u == 0 ? lat + a.rank : row + (size_t)(u - 1) * qd + a.nd) + 2 * i;
    T* dst = (u == 0 ? krow + a.rank : (T*)a.q_out + ((size_t)t * a.nq + (u - 1)) * kd + a.rank) + 2 * i;
    const bool pair = 2 * i + 1 < a.rd;
    const float x = to_f32(src[0]), y = pair ? to_f32(src[1]) : 0.f;
    float ox = x, oy = y;
    if (i < half_rot) {
      const float c = cs[i], s = sn[i];
      ox = fmaf(x, c, -__fmul_rn(y, s));
      oy = fmaf(y, c, __fmul_rn(x, s));
    }
    dst[0] = from_f32<T>(ox);
    if (pair) dst[1] = from_f32<T>(oy);
  }
}

struct ConvArgs {
  const void* proj;             // [T, ld], channels [queries | keys | values] first
  int ld, nq, nkv, kd, vd;
  const float* bias;            // [channels] or null
  const float* taps;            // [n_taps, channels]; null: no filter (n_taps = 1)
  int n_taps;
  float* kept;                  // [slots, n_taps - 1, channels]: inputs of the tokens before this step, oldest first
  const int *slots, *cu_q, *token_request;
  const float *wq, *wk;         // norm weights [nq * kd], [nkv * kd] or null
  float eps;
  void* q_out;                  // [T, nq * kd]
  void *kcache, *vcache;
  const int* slot_mapping;
  int page_size;
  long long k_page_stride, k_head_stride, v_page_stride, v_head_stride;
  int n_tokens;
  int update;                   // every request brings one token: its kept inputs move up here
  const int* positions;
  const float* freq;            // [rot_dims / 2] or null: query and key heads are rotated behind the norm
  int rot_dims, rot_pairs;      // the first rot_dims values of a head turn; pairs (2i, 2i + 1) or halves (i, i + rot_dims / 2)
  float rot_mag;                // cos and sin are multiplied by this
};

template <typename T, int V> struct Piece { T v[V]; };   // V neighbouring channels; 8 of them are 16-byte aligned
template <> struct __align__(16) Piece<float, 8> { float v[8]; };
template <> struct __align__(16) Piece<__nv_bfloat16, 8> { __nv_bfloat16 v[8]; };

// A CTA takes TOK consecutive tokens of the step with all their channels, V channels per thread and turn; the filtered
// queries and keys wait in shared memory for their sums of squares.  NT: the number of taps (0: any).  Which thread meets
// which channel depends on the sizes alone, so a token's sums have the same order in every batch.  Where a tile's tokens
// are one request's and their filters reach no kept input, the inputs of the tile are all asked for at once.
constexpr int CONV_THREADS = 384;
template <typename T, int V, int TOK, int NT>
__global__ void __launch_bounds__(CONV_THREADS) conv_norm_kv_write_kernel(ConvArgs a) {
  extern __shared__ __align__(16) float ys[];        // [TOK, (nq + nkv) * kd], then [TOK, rot_dims / 2] cosines and sines
  __shared__ float part[2 * TOK][33];
  pdl_trigger();
  const int nqc = a.nq * a.kd, nkc = a.nkv * a.kd, nvc = a.nkv * a.vd, channels = nqc + nkc + nvc, nqk = nqc + nkc;
  const int taps_n = NT ? NT : a.n_taps;
  const int t0 = blockIdx.x * TOK;
  pdl_wait();
  const T* proj = (const T*)a.proj;
  float ssq[TOK], ssk[TOK];
#pragma unroll
  for (int i = 0; i < TOK; ++i) ssq[i] = ssk[i] = 0.f;
  const int half = a.rot_dims / 2;
  float *turn_c = ys + (size_t)TOK * nqk, *turn_s = turn_c + TOK * half;
  for (int i = threadIdx.x; i < TOK * half; i += blockDim.x) {
    const int t = t0 + i / half;
    if (t >= a.n_tokens) continue;
    const float ang = __fmul_rn((float)a.positions[t], a.freq[i % half]);
    turn_c[i] = __fmul_rn(cosf(ang), a.rot_mag);
    turn_s[i] = __fmul_rn(sinf(ang), a.rot_mag);
  }
  bool inside = false;
  if (NT == 1) {
    inside = TOK > 1 && t0 + TOK <= a.n_tokens;    // one tap reads the token itself, whatever its request
  } else if (TOK > 1 && NT > 0 && t0 + TOK <= a.n_tokens) {
    const int req = a.token_request[t0];
    inside = req == a.token_request[t0 + TOK - 1] && t0 - a.cu_q[req] >= NT - 1;
  }
  for (int c = threadIdx.x * V; c < channels; c += blockDim.x * V) {
    Piece<T, V> in[NT && TOK > 1 ? TOK + NT - 1 : 1];
    if (inside) {
#pragma unroll
      for (int j = 0; j < (NT && TOK > 1 ? TOK + NT - 1 : 1); ++j)
        in[j] = *reinterpret_cast<const Piece<T, V>*>(proj + (size_t)(t0 - (NT - 1) + j) * a.ld + c);
    }
    Piece<float, V> w[NT ? NT : 1];
    if (NT) {
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        if (NT == 1 && a.taps == nullptr) {          // no filter
#pragma unroll
          for (int e = 0; e < V; ++e) w[j].v[e] = 1.f;
        } else {
          w[j] = *reinterpret_cast<const Piece<float, V>*>(a.taps + (size_t)j * channels + c);
        }
      }
    }
    Piece<float, V> add;
    if (a.bias) {
      add = *reinterpret_cast<const Piece<float, V>*>(a.bias + c);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) add.v[e] = 0.f;
    }
    const float* bias = add.v;
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
      const int t = t0 + i;
      if (t >= a.n_tokens) continue;
      float y[V], x[V];
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = 0.f;
      if (inside) {
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
          for (int e = 0; e < V; ++e)
            y[e] = fmaf(w[NT ? j : 0].v[e], to_f32(in[NT && TOK > 1 ? i + j : 0].v[e]) + bias[e], y[e]);
      } else {
        const int req = a.token_request[t], first = a.cu_q[req];
        float* kept = taps_n > 1 ? a.kept + (size_t)a.slots[req] * (taps_n - 1) * channels : nullptr;
#pragma unroll
        for (int j = 0; j < taps_n; ++j) {
          const int n = t - first - (taps_n - 1) + j;   // index among the request's tokens of this step; < 0: kept ones
          if (n >= 0) {
            const Piece<T, V> p = *reinterpret_cast<const Piece<T, V>*>(proj + (size_t)(first + n) * a.ld + c);
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] = to_f32(p.v[e]) + bias[e];
          } else {
            const Piece<float, V> p = *reinterpret_cast<const Piece<float, V>*>(kept + (size_t)(taps_n - 1 + n) * channels + c);
#pragma unroll
            for (int e = 0; e < V; ++e) x[e] = p.v[e];
            // this thread is the entry's only reader: what it holds next is the entry behind it
            if (a.update && j > 0) *reinterpret_cast<Piece<float, V>*>(kept + (size_t)(j - 1) * channels + c) = p;
          }
#pragma unroll
          for (int e = 0; e < V; ++e) {
            const float f = NT ? w[NT ? j : 0].v[e] : (a.taps ? a.taps[(size_t)j * channels + c + e] : 1.f);
            y[e] = fmaf(f, x[e], y[e]);
          }
        }
        if (a.update && taps_n > 1) {   // x is the token's own input now
          Piece<float, V> p;
#pragma unroll
          for (int e = 0; e < V; ++e) p.v[e] = x[e];
          *reinterpret_cast<Piece<float, V>*>(kept + (size_t)(taps_n - 2) * channels + c) = p;
        }
      }
      if (c >= nqk) {   // values have no norm
        const int slot = a.slot_mapping[t];
        if (slot < 0) continue;
        const int h = (c - nqk) / a.vd, d = (c - nqk) % a.vd;
        Piece<T, V> p;
#pragma unroll
        for (int e = 0; e < V; ++e) p.v[e] = from_f32<T>(y[e]);
        *reinterpret_cast<Piece<T, V>*>((T*)a.vcache + (long long)(slot / a.page_size) * a.v_page_stride +
                                        (long long)h * a.v_head_stride + (long long)(slot % a.page_size) * a.vd + d) = p;
        continue;
      }
      float ss = 0.f;
      float* keep_y = ys + (size_t)i * nqk + c;
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(y[e], y[e], ss);
      if (V == 8) {
        *reinterpret_cast<float4*>(keep_y) = make_float4(y[0], y[1 % V], y[2 % V], y[3 % V]);
        *reinterpret_cast<float4*>(keep_y + 4) = make_float4(y[4 % V], y[5 % V], y[6 % V], y[7 % V]);
      } else {
        keep_y[0] = y[0];
      }
      if (c < nqc) ssq[i] += ss; else ssk[i] += ss;
    }
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
#pragma unroll
  for (int i = 0; i < TOK; ++i) {
    const float q = warp_sum(ssq[i]), k = warp_sum(ssk[i]);
    if (lane == 0) { part[2 * i][warp] = q; part[2 * i + 1][warp] = k; }
  }
  __syncthreads();
  for (int s = warp; s < 2 * TOK; s += warps) {
    const float v = warp_sum(lane < warps ? part[s][lane] : 0.f);
    if (lane == 0) part[s][32] = 1.f / sqrtf(v / (float)((s & 1) ? nkc : nqc) + a.eps);
  }
  __syncthreads();
  for (int c = threadIdx.x * V; c < nqk; c += blockDim.x * V) {
    const bool is_q = c < nqc;
    const float* wn = is_q ? a.wq : a.wk;
    Piece<float, V> w;
    if (wn) {
      w = *reinterpret_cast<const Piece<float, V>*>(wn + (is_q ? c : c - nqc));
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) w.v[e] = 1.f;
    }
    const int h = (c - nqc) / a.kd, d = (c - nqc) % a.kd;
#pragma unroll
    for (int i = 0; i < TOK; ++i) {
      const int t = t0 + i;
      if (t >= a.n_tokens) continue;
      T* dst;
      if (is_q) {
        dst = (T*)a.q_out + (size_t)t * nqc + c;
      } else {
        const int slot = a.slot_mapping[t];
        if (slot < 0) continue;
        dst = (T*)a.kcache + (long long)(slot / a.page_size) * a.k_page_stride + (long long)h * a.k_head_stride +
              (long long)(slot % a.page_size) * a.kd + d;
      }
      const float f = wn ? part[2 * i + (is_q ? 0 : 1)][32] : 1.f;
      const float* keep_y = ys + (size_t)i * nqk + c;   // this thread wrote these values itself
      float y[V];
      if (V == 8) {
        const float4 lo = *reinterpret_cast<const float4*>(keep_y), hi = *reinterpret_cast<const float4*>(keep_y + 4);
        y[0] = lo.x; y[1 % V] = lo.y; y[2 % V] = lo.z; y[3 % V] = lo.w; y[4 % V] = hi.x; y[5 % V] = hi.y; y[6 % V] = hi.z; y[7 % V] = hi.w;
      } else {
        y[0] = keep_y[0];
      }
      Piece<T, V> p;
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = __fmul_rn(__fmul_rn(y[e], f), w.v[e]);
      const int d0 = is_q ? c % a.kd : d;             // the piece's place in its head (a head is whole pieces)
      if (half > 0 && d0 < a.rot_dims) {
        const float* row = ys + (size_t)i * nqk + (c - d0);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          const int at = d0 + e;
          if (at >= a.rot_dims) continue;
          const bool first = a.rot_pairs ? !(at & 1) : at < half;
          const int other = a.rot_pairs ? at ^ 1 : (first ? at + half : at - half);
          const int pair = i * half + (a.rot_pairs ? at >> 1 : (first ? at : at - half));
          const float cs = turn_c[pair], sn = turn_s[pair];
          const float wo = wn ? wn[(is_q ? c : c - nqc) - d0 + other] : 1.f;
          const float yo = __fmul_rn(__fmul_rn(row[other], f), wo);
          y[e] = first ? fmaf(y[e], cs, -__fmul_rn(yo, sn)) : fmaf(y[e], cs, __fmul_rn(yo, sn));
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) p.v[e] = from_f32<T>(y[e]);
      *reinterpret_cast<Piece<T, V>*>(dst) = p;
    }
  }
}

template <typename T, int V, int TOK, int NT>
static int launch_conv(const ConvArgs& a, cudaStream_t s) {
  const int channels = (a.nq + a.nkv) * a.kd + a.nkv * a.vd, pieces = channels / V;
  const int threads = pieces >= CONV_THREADS ? CONV_THREADS : (pieces + 31) / 32 * 32;
  const size_t smem = (size_t)TOK * ((a.nq + a.nkv) * a.kd + a.rot_dims) * 4;
  static size_t configured = 48 * 1024;
  if (smem + 2 * TOK * 33 * 4 > configured) {
    cudaError_t e = cudaFuncSetAttribute(conv_norm_kv_write_kernel<T, V, TOK, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) TLLM_FAIL(TLLM_ERR_CUDA, "conv_norm_kv_write: cannot reserve %d bytes of shared memory: %s", (int)smem, cudaGetErrorString(e));
    configured = smem + 2 * TOK * 33 * 4;
  }
  TLLM_LAUNCH("conv_norm_kv_write", (conv_norm_kv_write_kernel<T, V, TOK, NT>), (unsigned)((a.n_tokens + TOK - 1) / TOK), threads, smem, s, a);
  return TLLM_OK;
}

template <typename T>
static int launch_conv_sizes(const ConvArgs& a, bool vec, cudaStream_t s) {
  constexpr int TOK = 4;
  const bool many = !a.update && a.n_tokens >= 148 * TOK && (size_t)TOK * ((a.nq + a.nkv) * a.kd + a.rot_dims) * 4 <= 160 * 1024;
  if (!vec) return launch_conv<T, 1, 1, 0>(a, s);
  if (a.n_taps == 1) return many ? launch_conv<T, 8, TOK, 1>(a, s) : launch_conv<T, 8, 1, 1>(a, s);
  if (a.taps && a.n_taps == 4) return many ? launch_conv<T, 8, TOK, 4>(a, s) : launch_conv<T, 8, 1, 4>(a, s);
  return many ? launch_conv<T, 8, TOK, 0>(a, s) : launch_conv<T, 8, 1, 0>(a, s);
}

// x float32 [T, heads * vd]; gate rows of ldg values in the engine's dtype, heads * vd of them (per_head = 0) or
// `heads` (per_head = 1); out [T, heads * vd] in the engine's dtype.
template <typename T>
__global__ void sigmoid_gate_kernel(const float* __restrict__ x, const T* __restrict__ gate, int ldg, int per_head,
                                    T* __restrict__ out, long long n_tokens, int heads, int vd) {
  pdl_trigger();
  pdl_wait();
  const long long width = (long long)heads * vd, total = n_tokens * width;
  for (long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (long long)gridDim.x * blockDim.x) {
    const long long t = idx / width;
    const int c = (int)(idx % width);
    const float g = to_f32(gate[t * ldg + (per_head ? c / vd : c)]);
    out[idx] = from_f32<T>(x[idx] / (1.f + expf(-g)));
  }
}

}  // namespace tllm

using namespace tllm;

extern "C" int tllm_qk_norm_kv_write(void* proj, int ld, int nq, int nkv, int kd, int vd, const float* bq, const float* bk,
                                     const float* bv, const float* wq, const float* wk, float eps, float coef, int every,
                                     const int* positions, void* kcache, void* vcache, const int* slot_mapping,
                                     int page_size, long long k_page_stride, long long k_head_stride,
                                     long long v_page_stride, long long v_head_stride, int n_tokens, const float* freq,
                                     int rot_dims, int rot_pairs, float rot_mag, int dtype, void* stream) {
  TLLM_REQUIRE(n_tokens > 0 && nq > 0 && nkv > 0 && kd > 0 && kd <= MAX_ROW && vd > 0,
               "qk_norm_kv_write: %d tokens, %d / %d heads, key size %d (at most %d), value size %d", n_tokens, nq, nkv, kd, MAX_ROW, vd);
  TLLM_REQUIRE((wq == nullptr) == (wk == nullptr) && every >= 0 && page_size > 0 && kcache && vcache && slot_mapping && positions,
               "qk_norm_kv_write: norm weights for both of queries and keys or neither; caches, slots and positions are needed");
  QkArgs a;
  a.proj = proj; a.ld = ld; a.nq = nq; a.nkv = nkv; a.kd = kd; a.vd = vd; a.bq = bq; a.bk = bk; a.bv = bv; a.wq = wq; a.wk = wk;
  a.eps = eps; a.coef = coef; a.every = every; a.positions = positions; a.kcache = kcache; a.vcache = vcache;
  a.slot_mapping = slot_mapping; a.page_size = page_size; a.k_page_stride = k_page_stride; a.k_head_stride = k_head_stride;
  a.v_page_stride = v_page_stride; a.v_head_stride = v_head_stride; a.n_tokens = n_tokens;
  TLLM_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= kd && (rot_dims == 0 || freq),
               "qk_norm_kv_write: %d rotated values of %d (even, at most the head's size, with a frequency table)", rot_dims, kd);
  a.freq = freq; a.rot_dims = rot_dims; a.rot_pairs = rot_pairs; a.rot_mag = rot_mag;
  const long long tasks = (long long)n_tokens * (nq + 2 * nkv), blocks = (tasks + 3) / 4;
  TLLM_REQUIRE(blocks <= 2147483647LL, "qk_norm_kv_write: %lld rows exceed the grid", tasks);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == TLLM_F32) TLLM_LAUNCH("qk_norm_kv_write", qk_norm_kv_write_kernel<float>, (unsigned)blocks, 128, 0, s, a);
  else if (dtype == TLLM_BF16) TLLM_LAUNCH("qk_norm_kv_write", qk_norm_kv_write_kernel<__nv_bfloat16>, (unsigned)blocks, 128, 0, s, a);
  else TLLM_FAIL(TLLM_ERR_ARG, "qk_norm_kv_write: unknown dtype code %d", dtype);
  return TLLM_OK;
}

extern "C" int tllm_latent_kv_write(const void* proj, int ld, int nq, int nd, int rd, int rank, int rot_dims,
                                    const float* w_latent, const float* freq, float eps, const int* positions, void* q_out,
                                    void* kcache, void* vcache, const int* slot_mapping, int page_size,
                                    long long k_page_stride, long long v_page_stride, int n_tokens, float rot_mag,
                                    int rot_pairs, int dtype, void* stream) {
  TLLM_REQUIRE(n_tokens > 0 && nq > 0 && nd >= 0 && rd >= 0 && rank > 0 && rank <= MAX_ROW,
               "latent_kv_write: %d tokens, %d heads, sizes %d + %d, latent %d (at most %d)", n_tokens, nq, nd, rd, rank, MAX_ROW);
  TLLM_REQUIRE(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= rd && rot_dims <= 512 && (rot_dims == 0 || freq),
               "latent_kv_write: %d rotated values of %d (even, at most the part's size and 512, with a frequency table)", rot_dims, rd);
  TLLM_REQUIRE(positions && q_out && page_size > 0 && (kcache == nullptr || (w_latent && vcache && slot_mapping)), "latent_kv_write: a pointer is missing");
  LatentArgs a;
  a.proj = proj; a.ld = ld; a.nq = nq; a.nd = nd; a.rd = rd; a.rank = rank; a.rot_dims = rot_dims; a.w_latent = w_latent;
  a.freq = freq; a.eps = eps; a.positions = positions; a.q_out = q_out; a.kcache = kcache; a.vcache = vcache;
  a.slot_mapping = slot_mapping; a.page_size = page_size; a.k_page_stride = k_page_stride; a.v_page_stride = v_page_stride;
  a.n_tokens = n_tokens; a.rot_mag = rot_mag; a.rot_pairs = rot_pairs;
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == TLLM_F32) TLLM_LAUNCH("latent_kv_write", latent_kv_write_kernel<float>, n_tokens, 128, 0, s, a);
  else if (dtype == TLLM_BF16) TLLM_LAUNCH("latent_kv_write", latent_kv_write_kernel<__nv_bfloat16>, n_tokens, 128, 0, s, a);
  else TLLM_FAIL(TLLM_ERR_ARG, "latent_kv_write: unknown dtype code %d", dtype);
  return TLLM_OK;
}

extern "C" int tllm_conv_norm_kv_write(const void* proj, int ld, int nq, int nkv, int kd, int vd, const float* bias,
                                       const float* taps, int n_taps, float* kept, const int* slots, const int* cu_q,
                                       const int* token_request, const float* wq, const float* wk, float eps, void* q_out,
                                       void* kcache, void* vcache, const int* slot_mapping, int page_size,
                                       long long k_page_stride, long long k_head_stride, long long v_page_stride,
                                       long long v_head_stride, int n_tokens, int update, const int* positions,
                                       const float* freq, int rot_dims, int rot_pairs, float rot_mag, int dtype, void* stream) {
  TLLM_REQUIRE(n_tokens > 0 && nq > 0 && nkv > 0 && kd > 0 && vd > 0 && rot_dims >= 0 && ((long long)(nq + nkv) * kd + rot_dims) * 4 <= 220 * 1024,
               "conv_norm_kv_write: %d tokens, %d / %d heads, key size %d, value size %d (queries and keys of a token: at most %d values)",
               n_tokens, nq, nkv, kd, vd, 220 * 256);
  TLLM_REQUIRE(n_taps >= 1 && (n_taps == 1 || (taps && kept && slots)) && proj && q_out && kcache && vcache && slot_mapping && cu_q &&
               token_request && page_size > 0 && (wq == nullptr) == (wk == nullptr),
               "conv_norm_kv_write: %d taps; a filter needs weights, kept inputs and slots; norm weights for both or neither", n_taps);
  TLLM_REQUIRE(rot_dims % 2 == 0 && rot_dims <= kd && (rot_dims == 0 || (freq && positions)),
               "conv_norm_kv_write: %d rotated values of %d (even, at most the head's size, with a frequency table and positions)", rot_dims, kd);
  ConvArgs a;
  a.positions = positions; a.freq = freq; a.rot_dims = rot_dims; a.rot_pairs = rot_pairs; a.rot_mag = rot_mag;
  a.proj = proj; a.ld = ld; a.nq = nq; a.nkv = nkv; a.kd = kd; a.vd = vd; a.bias = bias; a.taps = taps; a.n_taps = n_taps;
  a.kept = kept; a.slots = slots; a.cu_q = cu_q; a.token_request = token_request; a.wq = wq; a.wk = wk; a.eps = eps;
  a.q_out = q_out; a.kcache = kcache; a.vcache = vcache; a.slot_mapping = slot_mapping; a.page_size = page_size;
  a.k_page_stride = k_page_stride; a.k_head_stride = k_head_stride; a.v_page_stride = v_page_stride;
  a.v_head_stride = v_head_stride; a.n_tokens = n_tokens; a.update = update;
  const int esz = dtype == TLLM_F32 ? 4 : 2;
  const auto ok16 = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
  const bool vec = kd % 8 == 0 && vd % 8 == 0 && ok16(proj) && ok16(q_out) && ok16(kcache) && ok16(vcache) && ok16(kept) && ok16(bias) && ok16(taps) && ok16(wq) && ok16(wk) &&
                   ((long long)ld * esz) % 16 == 0 && (k_page_stride * esz) % 16 == 0 && (k_head_stride * esz) % 16 == 0 &&
                   (v_page_stride * esz) % 16 == 0 && (v_head_stride * esz) % 16 == 0;
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == TLLM_F32) return launch_conv_sizes<float>(a, vec, s);
  if (dtype == TLLM_BF16) return launch_conv_sizes<__nv_bfloat16>(a, vec, s);
  TLLM_FAIL(TLLM_ERR_ARG, "conv_norm_kv_write: unknown dtype code %d", dtype);
}

extern "C" int tllm_sigmoid_gate(const float* x, const void* gate, int ldg, int per_head, void* out, long long n_tokens,
                                 int heads, int vd, int dtype, void* stream) {
  TLLM_REQUIRE(n_tokens > 0 && heads > 0 && vd > 0, "sigmoid_gate: %lld tokens, %d heads of %d values", n_tokens, heads, vd);
  const long long total = n_tokens * heads * vd;
  const int threads = 256;
  const long long want = (total + threads - 1) / threads;
  const int blocks = (int)(want < 148 * 16 ? want : 148 * 16);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == TLLM_F32)
    TLLM_LAUNCH("sigmoid_gate", sigmoid_gate_kernel<float>, blocks, threads, 0, s, x, (const float*)gate, ldg, per_head, (float*)out, n_tokens, heads, vd);
  else if (dtype == TLLM_BF16)
    TLLM_LAUNCH("sigmoid_gate", sigmoid_gate_kernel<__nv_bfloat16>, blocks, threads, 0, s, x, (const __nv_bfloat16*)gate, ldg, per_head, (__nv_bfloat16*)out, n_tokens, heads, vd);
  else TLLM_FAIL(TLLM_ERR_ARG, "sigmoid_gate: unknown dtype code %d", dtype);
  return TLLM_OK;
}
