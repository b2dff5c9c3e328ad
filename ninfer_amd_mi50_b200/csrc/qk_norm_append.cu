// The stage after the projection of an attention whose values are its keys: add the biases, take
// the queries and the keys each over the root mean square of the WHOLE projection (all heads'
// rows at once, before they are split into heads) times a weight, write the normed keys into the
// key half of the request's cache page and the keys as projected (bias added, not normed) into the
// value half.  Nothing is rotated.  The projection arrives as float32 sums, so a key is rounded
// to the cache's type once.
//
// Cache page layout: [2 (k, v)][kv_heads][page_size][head_dim], as rope_append.cu writes it.
//
// A second kernel serves an attention with values of their own and a rotation after the same
// whole-projection norms or none (in either page layout; the values may be turned as well), a third its
// elementwise output gate, and a fourth turns attention outputs back.
#define NF_CHAIN_CLASS 4
#include "common.cuh"

namespace nf {

template <typename T>
__global__ void __launch_bounds__(256)
qk_whole_norm_append_kernel(const float* __restrict__ proj, int ld, int q_col0, int k_col0,
                            const float* __restrict__ bias_q, const float* __restrict__ bias_k,
                            const float* __restrict__ wq, const float* __restrict__ wk, float eps,
                            const int* __restrict__ positions, const int* __restrict__ row_seg,
                            T* __restrict__ q_out, int Hq, int Hkv, int D, T* __restrict__ pages,
                            const int* __restrict__ block_table, int bt_width, int page_size, int num_pages,
                            int append) {
  __shared__ float red[33];
  const int t = blockIdx.x;
  chain_release_if_small();
  chain_wait(proj);
  const float* row = proj + (size_t)t * ld;
  const int QW = Hq * D, KW = Hkv * D;
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < QW; i += blockDim.x) {
    const float v = row[q_col0 + i] + (bias_q ? bias_q[i] : 0.f);
    sq += v * v;
  }
  for (int i = threadIdx.x; i < KW; i += blockDim.x) {
    const float v = row[k_col0 + i] + (bias_k ? bias_k[i] : 0.f);
    sk += v * v;
  }
  const float inv_q = rsqrtf(block_sum(sq, red) / (float)QW + eps);
  const float inv_k = rsqrtf(block_sum(sk, red) / (float)KW + eps);
  T* qo = q_out + (size_t)t * QW;
  for (int i = threadIdx.x; i < QW; i += blockDim.x) {
    const float v = row[q_col0 + i] + (bias_q ? bias_q[i] : 0.f);
    qo[i] = from_float<T>(v * inv_q * wq[i]);
  }
  if (!append) return;
  const int pos = positions[t], seg = row_seg[t];
  const int lp = pos / page_size;
  const int page = (lp >= 0 && lp < bt_width) ? block_table[(size_t)seg * bt_width + lp] : -1;
  if (page < 0 || page >= num_pages) return;               // no page reserved: never write out of bounds
  T* kdst = pages + ((size_t)page * 2 * Hkv * page_size + (size_t)(pos - lp * page_size)) * D;
  const size_t head_stride = (size_t)page_size * D;
  for (int i = threadIdx.x; i < KW; i += blockDim.x) {
    const int head = i / D, d = i - head * D;
    const float v = row[k_col0 + i] + (bias_k ? bias_k[i] : 0.f);
    kdst[(size_t)head * head_stride + d] = from_float<T>(v * inv_k * wk[i]);
    kdst[(size_t)(Hkv + head) * head_stride + d] = from_float<T>(v);
  }
}


// The same stage for an attention with values of their own and a rotation: biases; q and k each over
// the root mean square of the WHOLE projection times a weight of the projection's width; then the first
// `rot` dimensions of every q and k head turned by the row's position (pair (i, i + rot/2), angle
// pos * inv_freq[i] in float32), cosine and sine both times `mag`; q goes out in the cache's type, the
// key and the value (bias added) into the request's page.  Two page layouts:
//   rows == 0: [2 (k, v)][kv_heads][page_size][P], what the flash and decode kernels read; P >= D and P >= Dv, the
//   rest of a key, a value and a query (rows of Hq * P) is zero, so that sizes those kernels do not take, or that
//   differ, can be widened to one that they take;
//   rows == 1: [page_size][kv_heads * D | kv_heads * Dv], one row a token, for key and value sizes that differ.
// Hkv == 0: a layer that reads another layer's keys brings queries only.
// Further forms: wq null - no norms; interleaved - pairs (2i, 2i + 1) instead of (i, i + rot/2); v_freq - the value is
// turned too, over all its Dv dimensions in the same layout of pairs, pair m by pos * v_freq[m] (no magnitude).
// The row's normed values wait in shared memory (float32) between the two passes.
// VEC: all sizes are multiples of 4 (the turned halves too): runs of four elements an access, and the norm's
// factors are applied where the values are read for the second time.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
whole_norm_rope_append_kernel(const float* __restrict__ proj, int ld, int q_col0, int k_col0, int v_col0,
                              const float* __restrict__ bias_q, const float* __restrict__ bias_k,
                              const float* __restrict__ bias_v, const float* __restrict__ wq,
                              const float* __restrict__ wk, float eps, const float* __restrict__ inv_freq, int rot,
                              float mag, const int* __restrict__ positions, const int* __restrict__ row_seg,
                              T* __restrict__ q_out, int Hq, int Hkv, int D, int Dv, T* __restrict__ pages,
                              const int* __restrict__ block_table, int bt_width, int page_size, int num_pages,
                              int rows_layout, int P, int interleaved, const float* __restrict__ v_freq) {
  // [Hq * D + Hkv * D], cosine and sine of the row's rot / 2 angles, and of its Dv / 2 angles if values are turned
  extern __shared__ __align__(16) float y[];
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int QW = Hq * D, KW = Hkv * D;
  const int half = rot / 2;
  float* cs_s = y + QW + KW;
  float* sn_s = cs_s + half;
  float* vcs_s = sn_s + half;
  float* vsn_s = vcs_s + Dv / 2;
  chain_release_if_small();
  // the angles depend on the position alone (a step's input, not the kernel before's output): all heads share them
  const int pos = positions[t];
  for (int u = threadIdx.x; u < half; u += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * inv_freq[u], &sn, &cs);
    cs_s[u] = cs * mag;
    sn_s[u] = sn * mag;
  }
  if (v_freq)
    for (int u = threadIdx.x; u < Dv / 2; u += blockDim.x) {
      float sn, cs;
      sincosf((float)pos * v_freq[u], &sn, &cs);
      vcs_s[u] = cs;
      vsn_s[u] = sn;
    }
  chain_wait(proj);
  const float* row = proj + (size_t)t * ld;
  float sq = 0.f, sk = 0.f;
  // (which of the two forms runs depends on sizes and addresses that are the same in every step of a model)
  const bool vec = (ld | q_col0 | k_col0 | QW | KW) % 4 == 0 && (uintptr_t)proj % 16 == 0 &&
                   (!bias_q || (uintptr_t)bias_q % 16 == 0) && (!bias_k || (uintptr_t)bias_k % 16 == 0);
  if (vec) {
    for (int i = threadIdx.x * 4; i < QW + KW; i += blockDim.x * 4) {
      const bool is_q = i < QW;
      const int c = is_q ? i : i - QW;
      const float* bp = is_q ? bias_q : bias_k;
      float4 v = *reinterpret_cast<const float4*>(row + (is_q ? q_col0 : k_col0) + c);
      if (bp) {
        const float4 b = *reinterpret_cast<const float4*>(bp + c);
        v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
      }
      *reinterpret_cast<float4*>(y + i) = v;
      const float s4 = fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, v.x * v.x)));
      if (is_q) sq += s4; else sk += s4;
    }
  } else {
    for (int i = threadIdx.x; i < QW; i += blockDim.x) {
      const float v = row[q_col0 + i] + (bias_q ? bias_q[i] : 0.f);
      y[i] = v;
      sq = fmaf(v, v, sq);
    }
    for (int i = threadIdx.x; i < KW; i += blockDim.x) {
      const float v = row[k_col0 + i] + (bias_k ? bias_k[i] : 0.f);
      y[QW + i] = v;
      sk = fmaf(v, v, sk);
    }
  }
  float inv_q = 1.f, inv_k = 1.f;
  if (wq) {
    inv_q = 1.f / sqrtf(block_sum(sq, red) / (float)QW + eps);
    inv_k = KW ? 1.f / sqrtf(block_sum(sk, red) / (float)KW + eps) : 0.f;
  }
  if (!VEC && wq) {
    for (int i = threadIdx.x; i < QW; i += blockDim.x) y[i] = y[i] * inv_q * wq[i];
    for (int i = threadIdx.x; i < KW; i += blockDim.x) y[QW + i] = y[QW + i] * inv_k * wk[i];
  }
  __syncthreads();
  T* krow = nullptr;                           // where head 0's key of this token starts
  size_t k_head_stride = 0, v_head_stride = 0;
  T* vrow = nullptr;
  if (Hkv > 0) {
    const int lp = pos / page_size;
    const int page = (lp >= 0 && lp < bt_width) ? block_table[(size_t)row_seg[t] * bt_width + lp] : -1;
    if (page >= 0 && page < num_pages) {       // no page reserved: never write out of bounds
      const int in_page = pos - lp * page_size;
      if (rows_layout) {
        krow = pages + ((size_t)page * page_size + in_page) * ((size_t)Hkv * (D + Dv));
        vrow = krow + (size_t)Hkv * D;
        k_head_stride = D; v_head_stride = Dv;
      } else {
        krow = pages + ((size_t)page * 2 * Hkv * page_size + in_page) * P;
        k_head_stride = v_head_stride = (size_t)page_size * P;
        vrow = krow + (size_t)Hkv * k_head_stride;
      }
    }
  }
  // a unit is a turned pair (u, u + rot/2) of a head, whose angle is worked out once, or a single dimension beyond
  const int units = D - half;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
  for (int hh = warp; hh < Hq + Hkv; hh += nwarp) {       // a warp a head: q heads first, then k heads, as they lie in y
    const bool is_q = hh < Hq;
    const float* yy = y + (size_t)hh * D;
    T* dst = is_q ? q_out + ((size_t)t * Hq + hh) * P
                  : (krow ? krow + (size_t)(hh - Hq) * k_head_stride : nullptr);
    if (!dst) continue;
    if constexpr (VEC) {
      const float* w = wq ? (is_q ? wq + (size_t)hh * D : wk + (size_t)(hh - Hq) * D) : nullptr;
      const float inv = is_q ? inv_q : inv_k;
      auto read4 = [&](int d, float* v) {
        load4(yy + d, v);
        if (w) {
          float wv[4];
          load4(w + d, wv);
#pragma unroll
          for (int e = 0; e < 4; ++e) v[e] = v[e] * inv * wv[e];
        }
      };
      const int turned = interleaved ? half / 2 : half / 4;              // runs that hold pairs
      for (int u = lane; u < turned + (D - rot) / 4; u += 32) {
        float a[4], b[4], r[4], q[4];
        if (u >= turned) {
          const int d = rot + (u - turned) * 4;
          read4(d, a);
          store4(dst + d, a);
        } else if (interleaved) {
          const int d = u * 4;
          read4(d, a);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float sn = sn_s[2 * u + e], cs = cs_s[2 * u + e];
            r[2 * e] = a[2 * e] * cs - a[2 * e + 1] * sn;
            r[2 * e + 1] = a[2 * e + 1] * cs + a[2 * e] * sn;
          }
          store4(dst + d, r);
        } else {
          const int d = u * 4;
          read4(d, a);
          read4(d + half, b);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float sn = sn_s[d + e], cs = cs_s[d + e];
            r[e] = a[e] * cs - b[e] * sn;
            q[e] = b[e] * cs + a[e] * sn;
          }
          store4(dst + d, r);
          store4(dst + d + half, q);
        }
      }
    } else
    for (int u = lane; u < units; u += 32) {
      if (u < half) {
        const int i0 = interleaved ? 2 * u : u, i1 = interleaved ? 2 * u + 1 : u + half;
        const float a = yy[i0], b = yy[i1];
        const float sn = sn_s[u], cs = cs_s[u];
        dst[i0] = from_float<T>(a * cs - b * sn);
        dst[i1] = from_float<T>(b * cs + a * sn);
      } else {
        const int d = rot + (u - half);
        dst[d] = from_float<T>(yy[d]);
      }
    }
    if (is_q || !rows_layout)
      for (int d = D + lane; d < P; d += 32) dst[d] = from_float<T>(0.f);
  }
  if (vrow) {
    const int vhalf = v_freq ? Dv / 2 : 0;
    for (int head = warp; head < Hkv; head += nwarp) {
      T* dst = vrow + (size_t)head * v_head_stride;
      const float* src = row + v_col0 + (size_t)head * Dv;
      const float* b = bias_v ? bias_v + (size_t)head * Dv : nullptr;
      if constexpr (VEC) {
        auto read4 = [&](int d, float* v) {
          load4(src + d, v);
          if (b) {
            float bv[4];
            load4(b + d, bv);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] += bv[e];
          }
        };
        for (int u = lane; u < Dv / 4; u += 32) {
          float x[4], z[4], r[4], q[4];
          const int d = u * 4;
          if (!v_freq) {
            read4(d, x);
            store4(dst + d, x);
          } else if (interleaved) {
            read4(d, x);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const float sn = vsn_s[2 * u + e], cs = vcs_s[2 * u + e];
              r[2 * e] = x[2 * e] * cs - x[2 * e + 1] * sn;
              r[2 * e + 1] = x[2 * e + 1] * cs + x[2 * e] * sn;
            }
            store4(dst + d, r);
          } else if (d < vhalf) {
            read4(d, x);
            read4(d + vhalf, z);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float sn = vsn_s[d + e], cs = vcs_s[d + e];
              r[e] = x[e] * cs - z[e] * sn;
              q[e] = z[e] * cs + x[e] * sn;
            }
            store4(dst + d, r);
            store4(dst + d + vhalf, q);
          }
        }
        if (!rows_layout)
          for (int d = Dv + lane; d < P; d += 32) dst[d] = from_float<T>(0.f);
        continue;
      }
      for (int u = lane; u < vhalf; u += 32) {
        const int i0 = interleaved ? 2 * u : u, i1 = interleaved ? 2 * u + 1 : u + vhalf;
        const float x0 = src[i0] + (b ? b[i0] : 0.f), x1 = src[i1] + (b ? b[i1] : 0.f);
        const float sn = vsn_s[u], cs = vcs_s[u];
        dst[i0] = from_float<T>(x0 * cs - x1 * sn);
        dst[i1] = from_float<T>(x1 * cs + x0 * sn);
      }
      for (int d = 2 * vhalf + lane; d < Dv; d += 32) dst[d] = from_float<T>(src[d] + (b ? b[d] : 0.f));
      if (!rows_layout)
        for (int d = Dv + lane; d < P; d += 32) dst[d] = from_float<T>(0.f);
    }
  }
}

// In place: every head of o [T, H * P] has its first Dv dimensions turned by -pos * freq[m] (pairs (m, m + Dv/2), or
// (2m, 2m + 1) interleaved): what attention over turned values leaves is turned back by the row's own position.
// VEC: four pairs a thread, 16- or 8-byte accesses.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
turn_back_kernel(T* __restrict__ o, const int* __restrict__ positions, const float* __restrict__ freq, int H, int Dv,
                 int P, int interleaved) {
  extern __shared__ __align__(16) float cs_s[];       // [Dv / 2] cosines, [Dv / 2] sines
  const int t = blockIdx.x, half = Dv / 2;
  float* sn_s = cs_s + half;
  chain_release_if_small();
  const int pos = positions[t];                       // a step's input, not the kernel before's output
  for (int u = threadIdx.x; u < half; u += blockDim.x) {
    float sn, cs;
    sincosf((float)pos * freq[u], &sn, &cs);
    cs_s[u] = cs;
    sn_s[u] = sn;
  }
  __syncthreads();
  chain_wait(o);
  T* row = o + (size_t)t * H * P;
  if constexpr (VEC) {
    const int q = half / 4;
    for (int i = threadIdx.x; i < H * q; i += blockDim.x) {
      const int hd = i / q, m = (i - hd * q) * 4;
      T* p = row + (size_t)hd * P;
      T* p0 = interleaved ? p + 2 * m : p + m;
      T* p1 = interleaved ? p + 2 * m + 4 : p + m + half;
      float x[4], z[4], a[4], b[4];
      load4(p0, x);
      load4(p1, z);
      // interleaved: x = (a0 b0 a1 b1), z = (a2 b2 a3 b3)
      const float u0[4] = {x[0], interleaved ? x[2] : x[1], interleaved ? z[0] : x[2], interleaved ? z[2] : x[3]};
      const float u1[4] = {interleaved ? x[1] : z[0], interleaved ? x[3] : z[1], interleaved ? z[1] : z[2], z[3]};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        a[e] = u0[e] * cs_s[m + e] + u1[e] * sn_s[m + e];
        b[e] = u1[e] * cs_s[m + e] - u0[e] * sn_s[m + e];
      }
      const float w0[4] = {a[0], interleaved ? b[0] : a[1], interleaved ? a[1] : a[2], interleaved ? b[1] : a[3]};
      const float w1[4] = {interleaved ? a[2] : b[0], interleaved ? b[2] : b[1], interleaved ? a[3] : b[2], b[3]};
      store4(p0, w0);
      store4(p1, w1);
    }
  } else {
    for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
      const int hd = i / half, m = i - hd * half;
      T* p = row + (size_t)hd * P;
      const int i0 = interleaved ? 2 * m : m, i1 = interleaved ? 2 * m + 1 : m + half;
      const float a = to_float(p[i0]), b = to_float(p[i1]);
      p[i0] = from_float<T>(a * cs_s[m] + b * sn_s[m]);
      p[i1] = from_float<T>(b * cs_s[m] - a * sn_s[m]);
    }
  }
}

// out[t, h * Dv + d] = o[t, h * P + d] * sigmoid(g[t, g_col0 + h * Dv + d]), d < Dv: an output gate element by element;
// the gate's logits are float32 sums or of the rows' type.  P > Dv: the heads of o are wider than the values (widened
// with zeros), out has the values side by side.
// VEC: four consecutive elements a thread, each operand's run in one access.
template <typename T, typename TG, bool VEC>
__global__ void sigmoid_gate_rows_kernel(const T* __restrict__ o, const TG* __restrict__ g, int ldg, int g_col0,
                                         T* __restrict__ out, int width, int Dv, int P) {
  const int t = blockIdx.y;
  chain_wait(o, g);
  constexpr int W = VEC ? 4 : 1;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * W;
  if (c >= width) return;
  const size_t oc = P == Dv ? (size_t)t * width + c : (size_t)t * (width / Dv) * P + (size_t)(c / Dv) * P + c % Dv;
  if constexpr (VEC) {
    float ov[4], gv[4];
    load4(o + oc, ov);
    load4(g + (size_t)t * ldg + g_col0 + c, gv);
#pragma unroll
    for (int e = 0; e < 4; ++e) ov[e] = ov[e] * (1.f / (1.f + expf(-gv[e])));
    store4(out + (size_t)t * width + c, ov);
  } else {
    const float gv = to_float(g[(size_t)t * ldg + g_col0 + c]);
    out[(size_t)t * width + c] = from_float<T>(to_float(o[oc]) * (1.f / (1.f + expf(-gv))));
  }
}

}  // namespace nf

using namespace nf;

extern "C" int nf_qk_whole_norm_append(const float* proj, int ld, int q_col0, int k_col0, const float* bias_q,
                                       const float* bias_k, const float* wq, const float* wk, float eps,
                                       const int* positions, const int* row_seg, void* q_out, int T, int Hq, int Hkv,
                                       int D, void* pages, const int* block_table, int bt_width, int page_size,
                                       int num_pages, int append, int dtype, cudaStream_t stream) {
  if (T == 0) return 0;
  NF_REQUIRE(T > 0 && Hq > 0 && Hkv > 0 && D > 0 && wq && wk, "qk_whole_norm_append: bad arguments");
  NF_REQUIRE(q_col0 >= 0 && k_col0 >= 0 && q_col0 + Hq * D <= ld && k_col0 + Hkv * D <= ld,
             "qk_whole_norm_append: the column ranges leave the projection");
  if (dtype == kF32)
    launch_chained(qk_whole_norm_append_kernel<float>, dim3(T), dim3(256), 0, stream, proj, ld, q_col0, k_col0, bias_q, bias_k, wq, wk, eps, positions, row_seg, (float*)q_out, Hq, Hkv, D, (float*)pages, block_table, bt_width, page_size, num_pages, append);
  else
    launch_chained(qk_whole_norm_append_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, stream, proj, ld, q_col0, k_col0, bias_q, bias_k, wq, wk, eps, positions, row_seg, (__nv_bfloat16*)q_out, Hq, Hkv, D, (__nv_bfloat16*)pages, block_table, bt_width, page_size, num_pages, append);
  return check_launch("qk_whole_norm_append");
}

// proj float32 [T, ld]: q (Hq x D) at q_col0, and with Hkv > 0 k (Hkv x D) at k_col0 and v (Hkv x Dv) at
// v_col0.  rows_layout 0: pages [.., 2, Hkv, page_size, P], P >= max(D, Dv); 1: pages [.., page_size, Hkv * (D + Dv)].
// q_out [T, Hq * P].  wq (and wk) null: no norms.  v_freq float32 [Dv / 2] or null: values turned.
extern "C" int nf_whole_norm_rope_append(const float* proj, int ld, int q_col0, int k_col0, int v_col0,
                                         const float* bias_q, const float* bias_k, const float* bias_v,
                                         const float* wq, const float* wk, float eps, const float* inv_freq, int rot,
                                         float mag, const int* positions, const int* row_seg, void* q_out, int T,
                                         int Hq, int Hkv, int D, int Dv, void* pages, const int* block_table,
                                         int bt_width, int page_size, int num_pages, int rows_layout, int P,
                                         int interleaved, const float* v_freq, int dtype, cudaStream_t stream) {
  if (T == 0) return 0;
  NF_REQUIRE(T > 0 && Hq > 0 && Hkv >= 0 && D > 0 && Dv > 0 && (!wq || Hkv == 0 || wk), "whole_norm_rope_append: bad arguments");
  NF_REQUIRE(q_col0 >= 0 && q_col0 + Hq * D <= ld, "whole_norm_rope_append: the queries leave the projection");
  NF_REQUIRE(Hkv == 0 || (k_col0 >= 0 && v_col0 >= 0 && k_col0 + Hkv * D <= ld && v_col0 + Hkv * Dv <= ld),
             "whole_norm_rope_append: keys or values leave the projection");
  NF_REQUIRE(Hkv == 0 || (pages && block_table), "whole_norm_rope_append: keys without a cache");
  NF_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= D && (rot == 0 || inv_freq), "whole_norm_rope_append: %d turned dimensions of %d", rot, D);
  NF_REQUIRE(P >= D && (rows_layout || Hkv == 0 || P >= Dv), "whole_norm_rope_append: heads of %d and %d do not fit rows of %d", D, Dv, P);
  NF_REQUIRE(!v_freq || Dv % 2 == 0, "whole_norm_rope_append: values of %d cannot be turned in pairs", Dv);
  const size_t smem = ((size_t)(Hq + Hkv) * D + rot + (v_freq ? Dv : 0)) * sizeof(float);
  NF_REQUIRE(smem <= 200 * 1024, "whole_norm_rope_append: %d values a row do not fit shared memory", (Hq + Hkv) * D);
  // (which form runs depends on sizes and addresses that are the same in every step of a model)
  const size_t el = dtype == kF32 ? 4 : 2;
  const bool vec = ((D | Dv | P | ld | q_col0 | k_col0 | v_col0) & 3) == 0 && rot % (interleaved ? 4 : 8) == 0 &&
                   (!v_freq || interleaved || Dv % 8 == 0) && (uintptr_t)proj % 16 == 0 && (uintptr_t)q_out % (4 * el) == 0 &&
                   (uintptr_t)pages % (4 * el) == 0 && (uintptr_t)wq % 16 == 0 && (uintptr_t)wk % 16 == 0 &&
                   (uintptr_t)bias_q % 16 == 0 && (uintptr_t)bias_k % 16 == 0 && (uintptr_t)bias_v % 16 == 0;
#define NF_WN(TT, VE)                                                                                                  \
  do {                                                                                                                \
    if (smem > 48 * 1024) cudaFuncSetAttribute(whole_norm_rope_append_kernel<TT, VE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    launch_chained(whole_norm_rope_append_kernel<TT, VE>, dim3(T), dim3(256), smem, stream, proj, ld, q_col0, k_col0, \
                   v_col0, bias_q, bias_k, bias_v, wq, wk, eps, inv_freq, rot, mag, positions, row_seg, (TT*)q_out,   \
                   Hq, Hkv, D, Dv, (TT*)pages, block_table, bt_width, page_size, num_pages, rows_layout, P,           \
                   interleaved, v_freq);                                                                              \
  } while (0)
  if (dtype == kF32) { if (vec) NF_WN(float, true); else NF_WN(float, false); }
  else { if (vec) NF_WN(__nv_bfloat16, true); else NF_WN(__nv_bfloat16, false); }
#undef NF_WN
  return check_launch("whole_norm_rope_append");
}

// o [T, H * P] of `dtype`, in place; freq float32 [Dv / 2].
extern "C" int nf_turn_back(void* o, const int* positions, const float* freq, int T, int H, int Dv, int P,
                            int interleaved, int dtype, cudaStream_t stream) {
  if (T == 0) return 0;
  NF_REQUIRE(T > 0 && H > 0 && Dv > 0 && Dv % 2 == 0 && P >= Dv && Dv <= 8192, "turn_back: bad sizes H=%d Dv=%d P=%d", H, Dv, P);
  const size_t el = dtype == kF32 ? 4 : 2;
  const bool vec = Dv % 8 == 0 && P % 4 == 0 && (uintptr_t)o % (4 * el) == 0;
  const size_t smem = (size_t)Dv * sizeof(float);
  const int units = vec ? H * Dv / 8 : H * Dv / 2;
  int th = 32;
  while (th < units && th < 256) th <<= 1;
  if (dtype == kF32) {
    if (vec) launch_chained(turn_back_kernel<float, true>, dim3(T), dim3(th), smem, stream, (float*)o, positions, freq, H, Dv, P, interleaved);
    else launch_chained(turn_back_kernel<float, false>, dim3(T), dim3(th), smem, stream, (float*)o, positions, freq, H, Dv, P, interleaved);
  } else {
    if (vec) launch_chained(turn_back_kernel<__nv_bfloat16, true>, dim3(T), dim3(th), smem, stream, (__nv_bfloat16*)o, positions, freq, H, Dv, P, interleaved);
    else launch_chained(turn_back_kernel<__nv_bfloat16, false>, dim3(T), dim3(th), smem, stream, (__nv_bfloat16*)o, positions, freq, H, Dv, P, interleaved);
  }
  return check_launch("turn_back");
}

// out [T, width] of `dtype`, width = heads * Dv; o [T, heads * P]; g [T, ldg] float32 (g_dtype 0) or of `dtype`.
extern "C" int nf_sigmoid_gate_rows(const void* o, const void* g, int g_dtype, int ldg, int g_col0, void* out, int T,
                                    int width, int Dv, int P, int dtype, cudaStream_t stream) {
  if (T == 0) return 0;
  NF_REQUIRE(T > 0 && T <= 65535 * 1024 && width > 0 && g_col0 >= 0 && g_col0 + width <= ldg, "sigmoid_gate_rows: bad sizes");
  NF_REQUIRE(Dv > 0 && width % Dv == 0 && P >= Dv, "sigmoid_gate_rows: heads of %d in rows of %d, %d in all", Dv, P, width);
  NF_REQUIRE(g_dtype == kF32 || g_dtype == dtype, "sigmoid_gate_rows: the gate is float32 or of the rows' type");
  const size_t tsize = dtype == kF32 ? 4 : 2, gsize = g_dtype == kF32 ? 4 : 2;
  const bool vec = width % 4 == 0 && (P == Dv || (P % 4 == 0 && Dv % 4 == 0)) && ldg % 4 == 0 && g_col0 % 4 == 0 && (uintptr_t)o % (4 * tsize) == 0 &&
                   (uintptr_t)out % (4 * tsize) == 0 && (uintptr_t)g % (4 * gsize) == 0;
  for (int t0 = 0; t0 < T; t0 += 65535) {
    const int rows = T - t0 < 65535 ? T - t0 : 65535;
    const dim3 grid(((vec ? width / 4 : width) + 255) / 256, rows);
    const size_t off = (size_t)t0 * width, ooff = (size_t)t0 * (width / Dv) * P, goff = (size_t)t0 * ldg;
#define NF_SG(TT, TG_, V) \
  launch_chained(sigmoid_gate_rows_kernel<TT, TG_, V>, grid, dim3(256), 0, stream, (const TT*)o + ooff, (const TG_*)g + goff, ldg, g_col0, (TT*)out + off, width, Dv, P)
    if (dtype == kF32) { if (vec) NF_SG(float, float, true); else NF_SG(float, float, false); }
    else if (g_dtype == kF32) { if (vec) NF_SG(__nv_bfloat16, float, true); else NF_SG(__nv_bfloat16, float, false); }
    else { if (vec) NF_SG(__nv_bfloat16, __nv_bfloat16, true); else NF_SG(__nv_bfloat16, __nv_bfloat16, false); }
#undef NF_SG
  }
  return check_launch("sigmoid_gate_rows");
}
