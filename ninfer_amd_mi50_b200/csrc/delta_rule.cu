// The gated delta rule: a recurrence over each request's rows, from and into the request's state slot.
//
//   S <- g_t S;  u_t = beta_t (v_t - S^T k_t);  S <- S + k_t u_t^T;  o_t = S^T q_t
//
// per head, S is D x V (float32, zero for a new request), k_t and q_t unit vectors (q_t also times a scale),
// g_t = exp(-exp(A_log) softplus(a_t + dt_bias)), beta_t = sigmoid(b_t).  Several heads may share a query and key
// head.  q, k, v arrive after their short convolution (ssm.cu), a and b as projections; everything from there on
// is float32.
//
// A step with prompt portions runs two kernels over chunks of kDrChunk rows counted from a segment's first row:
//
//  * `delta_rule_prepare_kernel`, one CTA a (chunk, query/key head): the unit vectors, the dot products of the
//    chunk's keys among one another and with its queries, and from them, for every head that shares them, a
//    record a row.  With G_t = g_1 ... g_t inside the chunk and D(s, t) = g_{s+1} ... g_t:
//        ck[s] = D(s, t) k_s.k_t  (s < t),   cq[s] = D(s, t) k_s.q_t  (s <= t),   G_t,  beta_t,  D(t, last).
//    Products of decays, never quotients: a decay near zero does no harm.
//
//  * `delta_rule_chunks_kernel`, one CTA a (request, head, 16 or 8 value columns), walks the chunks in order.  A column's
//    D state entries lie in the registers of LANES lanes, four consecutive entries every 4 * LANES.  With the state
//    S_0 at a chunk's start the rule for the whole chunk is
//        u_t = beta_t (v_t - G_t S_0^T k_t - sum_{s<t} ck_t[s] u_s)
//        o_t = G_t S_0^T q_t + sum_{s<=t} cq_t[s] u_s
//        S   = G_last S_0 + sum_s D(s, last) k_s u_s^T
//    so the sums over D of all its rows are taken of the same registers, independent of one another, and only the
//    short triangle in u is sequential.  Chunk c + 1's vectors and records are on their way (cp.async) meanwhile.
//
// A step of single rows is one kernel: every group of LANES lanes takes the vectors' norms itself, along with the
// state's products (the norms are factors of those sums).
//
// The state of a slot is laid out [head][value column][D].
#define NF_CHAIN_CLASS 2
#include "common.cuh"

namespace nf {

constexpr int kDrThreads = 128;
constexpr int kDrChunk = 8;
constexpr int kDrRecord = 2 * kDrChunk + 4;      // ck, cq, (G, beta, D(t, last), 0)

__device__ __forceinline__ float dr_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float dr_decay(float a, float dt_bias, float A_log) { return expf(-expf(A_log) * dr_softplus(a + dt_bias)); }
__device__ __forceinline__ float dr_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// vectors [T][G][2][DP]: unit q (times q_scale) and unit k, zeros from D to DP (the chunks' kernel's row, DPAD there);
// records [T][H][kDrRecord].
template <typename T>
__global__ void __launch_bounds__(32 * kDrChunk)
delta_rule_prepare_kernel(const T* __restrict__ qkv, int ld, int q_col0, int k_col0, const T* __restrict__ ab, int ld_ab,
                          int a_col0, int b_col0, const float* __restrict__ dt_bias, const float* __restrict__ A_log,
                          float q_scale, const int* __restrict__ seg_row0, float* __restrict__ vectors,
                          float* __restrict__ records, int H, int G, int D, int DP) {
  extern __shared__ float sm[];                  // [chunk][q: D + 1 | k: D + 1], dots [chunk][2][chunk], decays [chunk][heads a group]
  const int c0 = blockIdx.x * kDrChunk, seg = blockIdx.y, grp = blockIdx.z;
  chain_release_if_small();
  chain_wait(qkv, ab);
  const int row0 = seg_row0[seg], n = min(kDrChunk, seg_row0[seg + 1] - row0 - c0);
  if (n <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per = H / G;
  const int stride = D + 1;
  float* sq = sm;
  float* sk = sq + kDrChunk * stride;
  float* dots = sk + kDrChunk * stride;
  float* dec = dots + 2 * kDrChunk * kDrChunk;
  if (warp < n) {
    const size_t t = (size_t)(row0 + c0 + warp);
    const T* qr = qkv + t * ld + q_col0 + (size_t)grp * D;
    const T* kr = qkv + t * ld + k_col0 + (size_t)grp * D;
    float qq = 0.f, kk = 0.f;
    for (int d = lane; d < D; d += 32) {
      const float q = to_float(qr[d]), k = to_float(kr[d]);
      sq[warp * stride + d] = q;
      sk[warp * stride + d] = k;
      qq = fmaf(q, q, qq);
      kk = fmaf(k, k, kk);
    }
    const float iq = q_scale / sqrtf(warp_sum(qq) + 1e-6f), ik = 1.f / sqrtf(warp_sum(kk) + 1e-6f);
    float* vo = vectors + (t * G + grp) * 2 * DP;
    for (int d = lane; d < DP; d += 32) {
      const float q = d < D ? sq[warp * stride + d] * iq : 0.f, k = d < D ? sk[warp * stride + d] * ik : 0.f;
      if (d < D) { sq[warp * stride + d] = q; sk[warp * stride + d] = k; }
      vo[d] = q;
      vo[DP + d] = k;
    }
    for (int j = lane; j < per; j += 32) {
      const int hd = grp * per + j;
      dec[warp * per + j] = dr_decay(to_float(ab[t * ld_ab + a_col0 + hd]), dt_bias[hd], A_log[hd]);
    }
  }
  __syncthreads();
  // warp t: k_s . k_t and k_s . q_t for all s of the chunk; a lane has one of the 16 dots over one half of D
  if (warp < n) {
    const int s = lane & (kDrChunk - 1), which = (lane >> 3) & 1, half = lane >> 4;
    const float* mine = (which ? sq : sk) + warp * stride;
    const float* other = sk + s * stride;
    float acc = 0.f;
    if (s < n)
      for (int d = half * ((D + 1) / 2), e = half ? D : (D + 1) / 2; d < e; ++d) acc = fmaf(mine[d], other[d], acc);
    acc += __shfl_xor_sync(0xffffffffu, acc, 16);
    if (half == 0) dots[(warp * 2 + which) * kDrChunk + s] = acc;
  }
  __syncthreads();
  // a thread a (row, head): its record
  for (int x = threadIdx.x; x < n * per; x += blockDim.x) {
    const int t = x / per, j = x - t * per, hd = grp * per + j;
    const size_t row = (size_t)(row0 + c0 + t);
    float rec[kDrRecord];
#pragma unroll
    for (int i = 0; i < kDrRecord; ++i) rec[i] = 0.f;
    float run = 1.f;                             // D(s, t), from s = t downwards
#pragma unroll
    for (int s = kDrChunk - 1; s >= 0; --s) {
      if (s > t) continue;
      if (s < t) rec[s] = run * dots[(t * 2) * kDrChunk + s];
      rec[kDrChunk + s] = run * dots[(t * 2 + 1) * kDrChunk + s];
      run *= dec[s * per + j];
    }
    rec[2 * kDrChunk] = run;                     // all decays up to t
    rec[2 * kDrChunk + 1] = dr_sigmoid(to_float(ab[row * ld_ab + b_col0 + hd]));
    float after = 1.f;
    for (int s = t + 1; s < n; ++s) after *= dec[s * per + j];
    rec[2 * kDrChunk + 2] = after;
    float* ro = records + (row * H + hd) * kDrRecord;
#pragma unroll
    for (int i = 0; i < kDrRecord; i += 4) *reinterpret_cast<float4*>(ro + i) = make_float4(rec[i], rec[i + 1], rec[i + 2], rec[i + 3]);
  }
}

__device__ __forceinline__ void dr_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

template <int EPL, int LANES>
__device__ __forceinline__ void dr_load_state(const float* sp, int D, int lane, bool live, bool vec, float (&S)[EPL]) {
#pragma unroll
  for (int e = 0; e < EPL / 4; ++e) {
    const int d = (e * LANES + lane) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && vec) {
      if (d < D) v = *reinterpret_cast<const float4*>(sp + d);
    } else if (live) {
      if (d < D) v.x = sp[d];
      if (d + 1 < D) v.y = sp[d + 1];
      if (d + 2 < D) v.z = sp[d + 2];
      if (d + 3 < D) v.w = sp[d + 3];
    }
    S[4 * e] = v.x; S[4 * e + 1] = v.y; S[4 * e + 2] = v.z; S[4 * e + 3] = v.w;
  }
}
template <int EPL, int LANES>
__device__ __forceinline__ void dr_store_state(float* sp, int D, int lane, bool live, bool vec, const float (&S)[EPL]) {
  if (!live) return;
#pragma unroll
  for (int e = 0; e < EPL / 4; ++e) {
    const int d = (e * LANES + lane) * 4;
    if (vec) {
      if (d < D) *reinterpret_cast<float4*>(sp + d) = make_float4(S[4 * e], S[4 * e + 1], S[4 * e + 2], S[4 * e + 3]);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (d + i < D) sp[d + i] = S[4 * e + i];
    }
  }
}

// CP: value columns a thread works on; with two, the vectors it reads from shared memory serve both.
template <typename T, int EPL, int LANES, int CP>        // D <= EPL * LANES
__global__ void __launch_bounds__(kDrThreads / CP)
delta_rule_chunks_kernel(const float* __restrict__ vectors, const float* __restrict__ records, const T* __restrict__ vsrc,
                         int ld, int v_col0, float* __restrict__ state, long slot_stride, const int* __restrict__ seg_row0,
                         const int* __restrict__ seg_slot, float* __restrict__ out, int H, int G, int D, int V) {
  constexpr int NTH = kDrThreads / CP;
  constexpr int COLS = kDrThreads / LANES;
  constexpr int DPAD = EPL * LANES;
  constexpr int VR = (kDrChunk * COLS + NTH - 1) / NTH;
  __shared__ __align__(16) float sq[2][kDrChunk][DPAD];
  __shared__ __align__(16) float sk[2][kDrChunk][DPAD];
  __shared__ __align__(16) float srec[2][kDrChunk][kDrRecord];
  __shared__ float sv[2][kDrChunk][COLS];
  const int seg = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * COLS, grp = head / (H / G);
  const int tid = threadIdx.x, lane = tid % LANES, cidx = tid / LANES * CP;
  // rows beyond a short first chunk are read and multiplied by zeros
  for (int i = tid; i < 2 * kDrChunk * DPAD; i += NTH) { (&sq[0][0][0])[i] = 0.f; (&sk[0][0][0])[i] = 0.f; }
  for (int i = tid; i < 2 * kDrChunk * kDrRecord; i += NTH) (&srec[0][0][0])[i] = 0.f;
  for (int i = tid; i < 2 * kDrChunk * COLS; i += NTH) (&sv[0][0][0])[i] = 0.f;
  chain_release_if_small();
  chain_wait(vectors, records, vsrc, state);
  const int row0 = seg_row0[seg], rows = seg_row0[seg + 1] - row0;
  if (rows <= 0) return;
  float* slot = state + (size_t)seg_slot[seg] * slot_stride + (size_t)head * V * D;
  const bool vec = D % 4 == 0 && slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
  float S[CP][EPL];
#pragma unroll
  for (int c = 0; c < CP; ++c) {
    const int col = col0 + cidx + c;
    dr_load_state<EPL, LANES>(slot + (size_t)(col < V ? col : 0) * D, D, lane, col < V, vec, S[c]);
  }
  __syncthreads();                               // the zeros are in place before the first copies land
  T rv[VR];
  const float* vec_src = vectors + ((size_t)row0 * G + grp) * 2 * DPAD;
  const float* rec_src = records + ((size_t)row0 * H + head) * kDrRecord;
  auto fetch = [&](int c0, int b) {
    const int n = min(kDrChunk, rows - c0);
    constexpr int PIECES = DPAD / 2, RECS = kDrRecord / 4;       // 16-byte pieces of a row's two vectors, of its record
#pragma unroll
    for (int r = 0; r < kDrChunk * PIECES / NTH; ++r) {
      const int x = tid + r * NTH, t = x / PIECES, i = x % PIECES;
      if (t < n) dr_cp16(i < PIECES / 2 ? &sq[b][t][4 * i] : &sk[b][t][4 * (i - PIECES / 2)], vec_src + (size_t)(c0 + t) * G * 2 * DPAD + 4 * i);
    }
#pragma unroll
    for (int r = 0; r < (kDrChunk * RECS + NTH - 1) / NTH; ++r) {
      const int x = tid + r * NTH, t = x / RECS, i = x % RECS;
      if (t < n) dr_cp16(&srec[b][t][4 * i], rec_src + (size_t)(c0 + t) * H * kDrRecord + 4 * i);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll
    for (int r = 0; r < VR; ++r) {
      const int x = tid + r * NTH, t = x / COLS, j = x - t * COLS;
      rv[r] = from_float<T>(0.f);
      if (t < n && col0 + j < V) rv[r] = vsrc[(size_t)(row0 + c0 + t) * ld + v_col0 + (size_t)head * V + col0 + j];
    }
  };
  fetch(0, 0);
  int b = 0;
  for (int c0 = 0; c0 < rows; c0 += kDrChunk, b ^= 1) {
    const int n = min(kDrChunk, rows - c0);
#pragma unroll
    for (int r = 0; r < VR; ++r) {
      const int x = tid + r * NTH;
      if (x < kDrChunk * COLS) sv[b][x / COLS][x % COLS] = to_float(rv[r]);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                             // chunk c0 has landed; everyone is done with the other buffer
    if (n < kDrChunk) {
      // the last, short chunk: rows left over from the chunk before last count nothing (no write, no decay)
      for (int x = tid; x < (kDrChunk - n) * DPAD; x += NTH) { (&sq[b][n][0])[x] = 0.f; (&sk[b][n][0])[x] = 0.f; }
      for (int x = tid; x < (kDrChunk - n) * kDrRecord; x += NTH) (&srec[b][n][0])[x] = 0.f;
      __syncthreads();
    } else if (c0 + kDrChunk < rows) {
      fetch(c0 + kDrChunk, b ^ 1);
    }
    float dk[CP][kDrChunk], dq[CP][kDrChunk];
#pragma unroll
    for (int c = 0; c < CP; ++c)
#pragma unroll
      for (int t = 0; t < kDrChunk; ++t) dk[c][t] = dq[c][t] = 0.f;
#pragma unroll
    for (int e = 0; e < EPL / 4; ++e) {
#pragma unroll
      for (int t = 0; t < kDrChunk; ++t) {
        const float4 k4 = *reinterpret_cast<const float4*>(&sk[b][t][(e * LANES + lane) * 4]);
        const float4 q4 = *reinterpret_cast<const float4*>(&sq[b][t][(e * LANES + lane) * 4]);
#pragma unroll
        for (int c = 0; c < CP; ++c) {
          dk[c][t] = fmaf(S[c][4 * e], k4.x, dk[c][t]); dk[c][t] = fmaf(S[c][4 * e + 1], k4.y, dk[c][t]);
          dk[c][t] = fmaf(S[c][4 * e + 2], k4.z, dk[c][t]); dk[c][t] = fmaf(S[c][4 * e + 3], k4.w, dk[c][t]);
          dq[c][t] = fmaf(S[c][4 * e], q4.x, dq[c][t]); dq[c][t] = fmaf(S[c][4 * e + 1], q4.y, dq[c][t]);
          dq[c][t] = fmaf(S[c][4 * e + 2], q4.z, dq[c][t]); dq[c][t] = fmaf(S[c][4 * e + 3], q4.w, dq[c][t]);
        }
      }
    }
#pragma unroll
    for (int w = LANES / 2; w > 0; w >>= 1)
#pragma unroll
      for (int c = 0; c < CP; ++c)
#pragma unroll
        for (int t = 0; t < kDrChunk; ++t) {
          dk[c][t] += __shfl_xor_sync(0xffffffffu, dk[c][t], w);
          dq[c][t] += __shfl_xor_sync(0xffffffffu, dq[c][t], w);
        }
    // the triangle: every lane of a column works it out for itself (u takes dk's place, o dq's)
#pragma unroll
    for (int t = 0; t < kDrChunk; ++t) {
      float rec[kDrRecord];
#pragma unroll
      for (int i = 0; i < kDrRecord; i += 4) load4(&srec[b][t][i], rec + i);
#pragma unroll
      for (int c = 0; c < CP; ++c) {
        float r = rec[2 * kDrChunk] * dk[c][t];
#pragma unroll
        for (int s = 0; s < t; ++s) r = fmaf(rec[s], dk[c][s], r);
        dk[c][t] = rec[2 * kDrChunk + 1] * (sv[b][t][cidx + c] - r);
        float y = rec[2 * kDrChunk] * dq[c][t];
#pragma unroll
        for (int s = 0; s <= t; ++s) y = fmaf(rec[kDrChunk + s], dk[c][s], y);
        dq[c][t] = y;
      }
    }
    const float all = srec[b][n - 1][2 * kDrChunk];
#pragma unroll
    for (int c = 0; c < CP; ++c) {
#pragma unroll
      for (int i = 0; i < EPL; ++i) S[c][i] *= all;
      // lane t of a column stores row t
      const int col = col0 + cidx + c;
#pragma unroll
      for (int t = 0; t < kDrChunk; ++t) {
        if (t < n && col < V && lane == t % LANES) out[(size_t)(row0 + c0 + t) * H * V + (size_t)head * V + col] = dq[c][t];
        dk[c][t] *= srec[b][t][2 * kDrChunk + 2];
      }
    }
#pragma unroll
    for (int t = 0; t < kDrChunk; ++t) {
#pragma unroll
      for (int e = 0; e < EPL / 4; ++e) {
        const float4 k4 = *reinterpret_cast<const float4*>(&sk[b][t][(e * LANES + lane) * 4]);
#pragma unroll
        for (int c = 0; c < CP; ++c) {
          S[c][4 * e] = fmaf(k4.x, dk[c][t], S[c][4 * e]); S[c][4 * e + 1] = fmaf(k4.y, dk[c][t], S[c][4 * e + 1]);
          S[c][4 * e + 2] = fmaf(k4.z, dk[c][t], S[c][4 * e + 2]); S[c][4 * e + 3] = fmaf(k4.w, dk[c][t], S[c][4 * e + 3]);
        }
      }
    }
  }
#pragma unroll
  for (int c = 0; c < CP; ++c) {
    const int col = col0 + cidx + c;
    dr_store_state<EPL, LANES>(slot + (size_t)(col < V ? col : 0) * D, D, lane, col < V, vec, S[c]);
  }
}

// Every segment brings one row.
template <typename T, int EPL, int LANES>
__global__ void __launch_bounds__(kDrThreads)
delta_rule_step_kernel(const T* __restrict__ qkv, int ld, int q_col0, int k_col0, int v_col0, const T* __restrict__ ab,
                       int ld_ab, int a_col0, int b_col0, const float* __restrict__ dt_bias, const float* __restrict__ A_log,
                       float q_scale, float* __restrict__ state, long slot_stride, const int* __restrict__ seg_row0,
                       const int* __restrict__ seg_slot, float* __restrict__ out, int H, int G, int D, int V, int vec_in) {
  constexpr int COLS = kDrThreads / LANES;
  const int seg = blockIdx.x, head = blockIdx.y, grp = head / (H / G);
  const int lane = threadIdx.x % LANES, col = blockIdx.z * COLS + threadIdx.x / LANES;
  const bool live = col < V;
  chain_release_if_small();
  const float dtb = dt_bias[head], alog = A_log[head];
  chain_wait(qkv, ab, state);
  const size_t t = (size_t)seg_row0[seg];
  float* sp = state + (size_t)seg_slot[seg] * slot_stride + ((size_t)head * V + (live ? col : 0)) * D;
  const bool vec = D % 4 == 0 && slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
  float S[EPL], q[EPL], k[EPL];
  dr_load_state<EPL, LANES>(sp, D, lane, live, vec, S);
  const T* qr = qkv + t * ld + q_col0 + (size_t)grp * D;
  const T* kr = qkv + t * ld + k_col0 + (size_t)grp * D;
#pragma unroll
  for (int e = 0; e < EPL / 4; ++e) {
    const int d = (e * LANES + lane) * 4;
    if (vec_in) {
#pragma unroll
      for (int i = 0; i < 4; ++i) q[4 * e + i] = k[4 * e + i] = 0.f;
      if (d < D) { load4(qr + d, q + 4 * e); load4(kr + d, k + 4 * e); }
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        q[4 * e + i] = d + i < D ? to_float(qr[d + i]) : 0.f;
        k[4 * e + i] = d + i < D ? to_float(kr[d + i]) : 0.f;
      }
    }
  }
  const float v = live ? to_float(qkv[t * ld + v_col0 + (size_t)head * V + col]) : 0.f;
  const float g = dr_decay(to_float(ab[t * ld_ab + a_col0 + head]), dtb, alog);
  const float beta = dr_sigmoid(to_float(ab[t * ld_ab + b_col0 + head]));
  float sum[5] = {0.f, 0.f, 0.f, 0.f, 0.f};      // q.q, k.k, k.q, S^T k, S^T q
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    sum[0] = fmaf(q[i], q[i], sum[0]);
    sum[1] = fmaf(k[i], k[i], sum[1]);
    sum[2] = fmaf(k[i], q[i], sum[2]);
    sum[3] = fmaf(S[i], k[i], sum[3]);
    sum[4] = fmaf(S[i], q[i], sum[4]);
  }
#pragma unroll
  for (int w = LANES / 2; w > 0; w >>= 1)
#pragma unroll
    for (int j = 0; j < 5; ++j) sum[j] += __shfl_xor_sync(0xffffffffu, sum[j], w);
  const float iq = q_scale / sqrtf(sum[0] + 1e-6f), ik = 1.f / sqrtf(sum[1] + 1e-6f);
  const float u = beta * (v - g * (sum[3] * ik));
  const float o = g * (sum[4] * iq) + (sum[2] * ik) * iq * u;
  const float f = ik * u;
#pragma unroll
  for (int i = 0; i < EPL; ++i) S[i] = fmaf(g, S[i], k[i] * f);
  dr_store_state<EPL, LANES>(sp, D, lane, live, vec, S);
  if (live && lane == 0) out[t * H * V + (size_t)head * V + col] = o;
}

static int g_delta_columns = 0;      // nf_set_delta_rule_columns(): 1 or 2 forces the choice below (measurement)

template <typename T>
static int run_delta_rule(const void* qkv, int ld, int q0, int k0, int v0, const void* ab, int ld_ab, int a0, int b0,
                          const float* dt_bias, const float* A_log, float q_scale, float* state, long slot_stride,
                          const int* seg_row0, const int* seg_slot, float* vectors, float* records, float* out, int S,
                          int max_rows, int H, int G, int D, int DP, int V, cudaStream_t stream) {
  if (max_rows == 1) {
    const int vec_in = D % 4 == 0 && ld % 4 == 0 && q0 % 4 == 0 && k0 % 4 == 0 && (uintptr_t)qkv % (4 * sizeof(T)) == 0;
#define NF_DR(E, L)                                                                                                   \
  launch_chained(delta_rule_step_kernel<T, E, L>, dim3(S, H, (V + kDrThreads / L - 1) / (kDrThreads / L)), dim3(kDrThreads), 0, \
                 stream, (const T*)qkv, ld, q0, k0, v0, (const T*)ab, ld_ab, a0, b0, dt_bias, A_log, q_scale, state,  \
                 slot_stride, seg_row0, seg_slot, out, H, G, D, V, vec_in)
    if (D <= 32) NF_DR(4, 8); else if (D <= 64) NF_DR(8, 8); else if (D <= 128) NF_DR(16, 8); else NF_DR(16, 16);
#undef NF_DR
    return check_launch("delta_rule_step");
  }
  const size_t smem = (size_t)(2 * kDrChunk * (D + 1) + 2 * kDrChunk * kDrChunk + kDrChunk * (H / G)) * sizeof(float);
  launch_chained(delta_rule_prepare_kernel<T>, dim3((max_rows + kDrChunk - 1) / kDrChunk, S, G), dim3(32 * kDrChunk), smem, stream,
                 (const T*)qkv, ld, q0, k0, (const T*)ab, ld_ab, a0, b0, dt_bias, A_log, q_scale, seg_row0, vectors, records,
                 H, G, D, DP);
  if (int rc = check_launch("delta_rule_prepare")) return rc;
  // two columns a thread once there are CTAs enough (one prompt of 2,048 tokens, heads of 128 x 128: with 16 heads 433 us
  // with one column, 523 with two; with 28 heads 675 and 581)
  const long ctas = (long)S * H * ((V + kDrThreads / 8 - 1) / (kDrThreads / 8));
  const bool two = g_delta_columns ? g_delta_columns == 2 : ctas >= 200;
#define NF_DR(E, L)  do { if (two) NF_DR_C(E, L, 2); else NF_DR_C(E, L, 1); } while (0)
#define NF_DR_C(E, L, CC)                                                                                             \
  launch_chained(delta_rule_chunks_kernel<T, E, L, CC>, dim3(S, H, (V + kDrThreads / L - 1) / (kDrThreads / L)),      \
                 dim3(kDrThreads / CC), 0, stream, (const float*)vectors, (const float*)records, (const T*)qkv, ld, v0, \
                 state, slot_stride, seg_row0, seg_slot, out, H, G, D, V)
  if (D <= 32) NF_DR(4, 8); else if (D <= 64) NF_DR(8, 8); else if (D <= 128) NF_DR(16, 8); else NF_DR(16, 16);
#undef NF_DR
  return check_launch("delta_rule_chunks");
}

}  // namespace nf

using namespace nf;

extern "C" void nf_set_delta_rule_columns(int columns) { g_delta_columns = columns; }

extern "C" int nf_delta_rule_record() { return kDrRecord; }
extern "C" int nf_delta_rule_row(int D) { return D <= 32 ? 32 : (D <= 64 ? 64 : (D <= 128 ? 128 : 256)); }

// qkv [T, ld]: q (G x D) at q0, k (G x D) at k0, v (H x V) at v0; ab [T, ld_ab]: a (H) at a0, b (H) at b0; all of
// `dtype`.  dt_bias, A_log float32 [H]; state float32, slot s at state + s * slot_stride: [H][V][D]; out float32
// [T, H * V].  max_rows: the most rows a segment brings; 1: steps of single rows.  Otherwise vectors float32
// [T, G, 2, nf_delta_rule_row(D)] and records float32 [T, H, nf_delta_rule_record()] are scratch.
extern "C" int nf_delta_rule(const void* qkv, int ld, int q0, int k0, int v0, const void* ab, int ld_ab, int a0, int b0,
                             const float* dt_bias, const float* A_log, float q_scale, float* state, long long slot_stride,
                             const int* seg_row0, const int* seg_slot, float* vectors, float* records, float* out, int S,
                             int max_rows, int H, int G, int D, int V, int dtype, cudaStream_t stream) {
  if (S == 0) return 0;
  NF_REQUIRE(S > 0 && max_rows > 0 && H > 0 && G > 0 && H % G == 0 && D > 0 && D <= 256 && V > 0, "delta rule: bad sizes S=%d H=%d G=%d D=%d V=%d", S, H, G, D, V);
  NF_REQUIRE(H <= 65535 && (V + 7) / 8 <= 65535 && S <= 65535 && H / G <= 512, "delta rule: too many heads, columns or requests");
  NF_REQUIRE(q0 >= 0 && k0 >= 0 && v0 >= 0 && q0 + G * D <= ld && k0 + G * D <= ld && v0 + H * V <= ld && a0 >= 0 && b0 >= 0 &&
             a0 + H <= ld_ab && b0 + H <= ld_ab, "delta rule: the column ranges leave their rows");
  const int DP = nf_delta_rule_row(D);
  NF_REQUIRE(max_rows == 1 || (vectors && records && (uintptr_t)vectors % 16 == 0 && (uintptr_t)records % 16 == 0), "delta rule: prompt portions need their scratch");
  if (dtype == kF32)
    return run_delta_rule<float>(qkv, ld, q0, k0, v0, ab, ld_ab, a0, b0, dt_bias, A_log, q_scale, state, (long)slot_stride, seg_row0, seg_slot, vectors, records, out, S, max_rows, H, G, D, DP, V, stream);
  return run_delta_rule<__nv_bfloat16>(qkv, ld, q0, k0, v0, ab, ld_ab, a0, b0, dt_bias, A_log, q_scale, state, (long)slot_stride, seg_row0, seg_slot, vectors, records, out, S, max_rows, H, G, D, DP, V, stream);
}
