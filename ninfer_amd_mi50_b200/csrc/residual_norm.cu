// What lies between two sublayers of a block with a norm before and after each of them: the sublayer's
// output is put together, normed and scaled per channel, added to the residual stream, and the stream is
// normed again for the next sublayer - one pass over the row.
//
//   d = ca * a + cb * b                   two mixers side by side, each with its factor (b, or both, may be absent)
//     + sum_j wts[t, j] * y[inv[t, j]]    the routed experts' pending sum (j ascending, rounded to T as the separate
//                                         combine kernel rounds it)
//     + bias                              a projection's bias that was left to this kernel
//   h <- h + (d / sqrt(mean(d^2) + eps1)) * w1           w1 null: h <- h + d
//   out = (h / sqrt(mean(h^2) + eps2)) * w2              w2 null: out = h in the engine's type
//
// w1 holds the norm's weight and the channel scale multiplied.  With `rows`, row r reads h[rows[r]] and the
// sources' row rows[r], writes out[r] and leaves h alone.  `out` may be null (only the stream is updated) and may
// be a column range of wider rows (ldo).  All sums and products are float32.
//
// VEC: the width is a multiple of 4 and every operand is aligned: a thread owns R runs of four consecutive
// elements, keeps them in registers from the first pass to the last, and asks for the weights before it waits
// for the kernel before it.  Otherwise the row waits in shared memory, element by element.
#define NF_CHAIN_CLASS 2
#include "common.cuh"

namespace nf {

template <typename T>
struct SublayerOutput {
  const T* a;
  const T* b;
  const T* y;
  const int* inv;
  const float* wts;
  const float* bias;
  float ca, cb;
  int k;
};

template <typename T, int R>
__global__ void __launch_bounds__(512)
residual_norm_vec_kernel(float* __restrict__ h, SublayerOutput<T> s, const float* __restrict__ w1, float eps1,
                         const int* __restrict__ rows, const float* __restrict__ w2, float eps2, T* __restrict__ out,
                         int ldo, int hidden) {
  __shared__ float red[33];
  const int r = blockIdx.x;
  chain_release_if_small();
  float4 w1v[R], w2v[R], bv[R];
#pragma unroll
  for (int c = 0; c < R; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    w1v[c] = w2v[c] = bv[c] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < hidden) {
      if (w1) w1v[c] = *reinterpret_cast<const float4*>(w1 + i);
      if (w2) w2v[c] = *reinterpret_cast<const float4*>(w2 + i);
      if (s.bias) bv[c] = *reinterpret_cast<const float4*>(s.bias + i);
    }
  }
  chain_wait(h, s.a, s.b, s.y, s.inv, s.wts, rows);
  const int src = rows ? rows[r] : r;
  float* hr = h + (size_t)src * hidden;
  float v[R][4], d[R][4];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < R; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) v[c][e] = d[c][e] = 0.f;
    if (i >= hidden) continue;
    load4(hr + i, v[c]);
    float x[4];
    if (s.a) {
      load4(s.a + (size_t)src * hidden + i, x);
#pragma unroll
      for (int e = 0; e < 4; ++e) d[c][e] = s.ca * x[e];
    }
    if (s.b) {
      load4(s.b + (size_t)src * hidden + i, x);
#pragma unroll
      for (int e = 0; e < 4; ++e) d[c][e] += s.cb * x[e];
    }
    if (s.y) {
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      for (int j = 0; j < s.k; ++j) {
        const float wt = s.wts ? s.wts[(size_t)src * s.k + j] : 1.f;
        load4(s.y + (size_t)s.inv[(size_t)src * s.k + j] * hidden + i, x);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] += wt * x[e];
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) d[c][e] += to_float(from_float<T>(acc[e]));
    }
    d[c][0] += bv[c].x; d[c][1] += bv[c].y; d[c][2] += bv[c].z; d[c][3] += bv[c].w;
#pragma unroll
    for (int e = 0; e < 4; ++e) ss = fmaf(d[c][e], d[c][e], ss);
  }
  if (w1) {
    const float inv1 = 1.f / sqrtf(block_sum(ss, red) / (float)hidden + eps1);
#pragma unroll
    for (int c = 0; c < R; ++c) {
      d[c][0] *= inv1 * w1v[c].x; d[c][1] *= inv1 * w1v[c].y;
      d[c][2] *= inv1 * w1v[c].z; d[c][3] *= inv1 * w1v[c].w;
    }
  }
  const bool changed = s.a || s.b || s.y || s.bias;
  float s2 = 0.f;
#pragma unroll
  for (int c = 0; c < R; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i >= hidden) continue;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      v[c][e] += d[c][e];
      s2 = fmaf(v[c][e], v[c][e], s2);
    }
    if (changed && !rows) store4(hr + i, v[c]);
  }
  if (!out) return;
  float inv2 = 1.f;
  if (w2) inv2 = 1.f / sqrtf(block_sum(s2, red) / (float)hidden + eps2);
#pragma unroll
  for (int c = 0; c < R; ++c) {
    const int i = (c * blockDim.x + threadIdx.x) * 4;
    if (i >= hidden) continue;
    if (w2) {
      v[c][0] *= inv2 * w2v[c].x; v[c][1] *= inv2 * w2v[c].y;
      v[c][2] *= inv2 * w2v[c].z; v[c][3] *= inv2 * w2v[c].w;
    }
    store4(out + (size_t)r * ldo + i, v[c]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
residual_norm_kernel(float* __restrict__ h, SublayerOutput<T> s, const float* __restrict__ w1, float eps1,
                     const int* __restrict__ rows, const float* __restrict__ w2, float eps2, T* __restrict__ out, int ldo,
                     int hidden) {
  extern __shared__ float row[];      // [hidden]
  __shared__ float red[33];
  const int r = blockIdx.x;
  chain_release_if_small();
  chain_wait(h, s.a, s.b, s.y, s.inv, s.wts, rows);
  const int src = rows ? rows[r] : r;
  float* hr = h + (size_t)src * hidden;
  float ss = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    float d = 0.f;
    if (s.a) d = s.ca * to_float(s.a[(size_t)src * hidden + i]);
    if (s.b) d += s.cb * to_float(s.b[(size_t)src * hidden + i]);
    if (s.y) {
      float acc = 0.f;
      for (int j = 0; j < s.k; ++j)
        acc += (s.wts ? s.wts[(size_t)src * s.k + j] : 1.f) *
               to_float(s.y[(size_t)s.inv[(size_t)src * s.k + j] * hidden + i]);
      d += to_float(from_float<T>(acc));
    }
    if (s.bias) d += s.bias[i];
    row[i] = d;
    ss = fmaf(d, d, ss);
  }
  float inv1 = 1.f;
  if (w1) inv1 = 1.f / sqrtf(block_sum(ss, red) / (float)hidden + eps1);
  const bool changed = s.a || s.b || s.y || s.bias;
  float s2 = 0.f;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float v = hr[i] + (w1 ? row[i] * (inv1 * w1[i]) : row[i]);
    if (changed && !rows) hr[i] = v;
    row[i] = v;
    s2 = fmaf(v, v, s2);
  }
  if (!out) return;
  float inv2 = 1.f;
  if (w2) inv2 = 1.f / sqrtf(block_sum(s2, red) / (float)hidden + eps2);
  for (int i = threadIdx.x; i < hidden; i += blockDim.x)
    out[(size_t)r * ldo + i] = from_float<T>(w2 ? row[i] * (inv2 * w2[i]) : row[i]);
}

template <typename T>
static int launch_residual_norm(float* h, const SublayerOutput<T>& s, const float* w1, float eps1, const int* rows,
                                const float* w2, float eps2, T* out, int ldo, int R, int hidden, cudaStream_t stream) {
  auto fits = [](const void* p, size_t bytes) { return (uintptr_t)p % bytes == 0; };
  const size_t el = 4 * sizeof(T);
  const bool vec = hidden % 4 == 0 && hidden <= 8192 && ldo % 4 == 0 && fits(h, 16) && fits(w1, 16) && fits(w2, 16) &&
                   fits(s.bias, 16) && fits(s.a, el) && fits(s.b, el) && fits(s.y, el) && fits(out, el);
  if (vec) {
    const int units = hidden / 4;
    const int runs = units <= 512 ? 1 : (units <= 1024 ? 2 : 4);
    const int th = ((units + runs - 1) / runs + 31) / 32 * 32;
#define NF_RN(RR) launch_chained(residual_norm_vec_kernel<T, RR>, dim3(R), dim3(th), 0, stream, h, s, w1, eps1, rows, w2, eps2, out, ldo, hidden)
    if (runs == 1) NF_RN(1); else if (runs == 2) NF_RN(2); else NF_RN(4);
#undef NF_RN
  } else {
    const size_t smem = (size_t)hidden * sizeof(float);
    NF_REQUIRE(smem <= 160 * 1024, "residual_norm: a row of %d does not fit shared memory", hidden);
    if (smem > 48 * 1024) cudaFuncSetAttribute(residual_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    launch_chained(residual_norm_kernel<T>, dim3(R), dim3(256), smem, stream, h, s, w1, eps1, rows, w2, eps2, out, ldo, hidden);
  }
  return check_launch("residual_norm");
}

}  // namespace nf

using namespace nf;

// h float32 [T, hidden]; a, b [T, hidden], y [pairs, hidden] and out [R, ldo] of `dtype` or null; inv int32 [T * k],
// wts float32 [T, k] or null; bias, w1, w2 float32 [hidden] or null; rows int32 [R] or null.
extern "C" int nf_residual_norm(float* h, const void* a, float ca, const void* b, float cb, const void* y, const int* inv,
                                const float* wts, int k, const float* bias, const float* w1, float eps1, const int* rows,
                                const float* w2, float eps2, void* out, int ldo, int R, int hidden, int dtype,
                                cudaStream_t stream) {
  if (R == 0) return 0;
  NF_REQUIRE(R > 0 && hidden > 0 && h && (!out || ldo >= hidden), "residual_norm: bad sizes R=%d hidden=%d", R, hidden);
  NF_REQUIRE(!y || (inv && k > 0), "residual_norm: routed rows without their plan");
  if (dtype == kF32) {
    const SublayerOutput<float> s = {(const float*)a, (const float*)b, (const float*)y, inv, wts, bias, ca, cb, k};
    return launch_residual_norm<float>(h, s, w1, eps1, rows, w2, eps2, (float*)out, ldo, R, hidden, stream);
  }
  typedef __nv_bfloat16 B;
  const SublayerOutput<B> s = {(const B*)a, (const B*)b, (const B*)y, inv, wts, bias, ca, cb, k};
  return launch_residual_norm<B>(h, s, w1, eps1, rows, w2, eps2, (B*)out, ldo, R, hidden, stream);
}
