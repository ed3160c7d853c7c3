// Recurrent token mixers: per-head matrix states (generalized delta rule, scalar-decay linear attention) and the
// element-wise minimal GRU, plus the gated group norm behind the matrix states.  Everything that enters a recurrence
// and the states themselves are f32.
//
// state_scan_kernel.  The columns of a head's state are independent of one another given the head's key-side vectors:
// S[:, j] <- w o S[:, j] - (a o u)(u . S[:, j]) + k v_j, o_j = q . S[:, j].  So a CTA owns a block of columns of one
// (sequence, head), KS neighbouring lanes share a column pair and hold kRows key channels of it each in registers, and
// the tokens go by one after the other: exact f32 arithmetic, and the result does not depend on how a prompt was cut.
//   warps 0 .. n-1    consumers: per token 5 (delta) or 3 (decay) packed f32x2 operations per channel pair and column,
//                     key-side vectors by 16-byte broadcast loads from shared memory, one butterfly over the KS lanes
//                     for u . S and one for the output.
//   last four warps   producers: read the raw projections of the next kChunk tokens, evaluate unit norms, decays,
//                     rates and activations once per (token, channel) and leave them in the other shared-memory buffer.
// The buffers change hands through named barriers (bar.sync / bar.arrive).
#include <atomic>

#include "common.cuh"
#include "kernels.h"

namespace teeny {

namespace {

constexpr int kRows = 16;        // key channels per consumer lane
constexpr int kChunk = 16;       // tokens per shared-memory buffer
constexpr int kProducers = 128;  // threads
constexpr int kMaxConsumers = 512;

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }

// Barrier FIRST + buf (buf 0 or 1); the numbers are immediates so that the kernel claims no more barriers than it uses.
template <int FIRST>
__device__ __forceinline__ void buffer_sync(int buf, int nthreads) {
  if (buf == 0) asm volatile("bar.sync %0, %1;" ::"n"(FIRST), "r"(nthreads) : "memory");
  else asm volatile("bar.sync %0, %1;" ::"n"(FIRST + 1), "r"(nthreads) : "memory");
}
template <int FIRST>
__device__ __forceinline__ void buffer_arrive(int buf, int nthreads) {
  if (buf == 0) asm volatile("bar.arrive %0, %1;" ::"n"(FIRST), "r"(nthreads) : "memory");
  else asm volatile("bar.arrive %0, %1;" ::"n"(FIRST + 1), "r"(nthreads) : "memory");
}
constexpr int kBarFull = 1, kBarEmpty = 3;

typedef unsigned long long f32x2;  // two packed f32
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

template <int KS>
__device__ __forceinline__ float lane_group_sum(float v) {
#pragma unroll
  for (int o = KS / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

constexpr int scan_vectors(int mode) { return mode == kScanDelta ? 5 : 2; }  // key-side vectors per token

template <typename T, int MODE, int KS>
__global__ void __launch_bounds__(kMaxConsumers + kProducers)
state_scan_kernel(const StateScan a, const SeqDesc* __restrict__ seqs, int col_groups) {
  constexpr int DKP = KS * kRows, NV = scan_vectors(MODE), NCH = (DKP + 31) / 32;
  extern __shared__ __align__(16) float scan_smem[];
  const int cols = 2 * col_groups;
  float* vec = scan_smem;                              // [2][kChunk][NV][DKP]
  float* val = scan_smem + 2 * kChunk * NV * DKP;      // [2][kChunk][cols]
  const int n_cons = blockDim.x - kProducers, all = blockDim.x;
  pdl_wait();
  const SeqDesc seq = seqs[blockIdx.z];
  const int h = blockIdx.y, col0 = blockIdx.x * cols;
  const int n_chunks = (seq.len + kChunk - 1) / kChunk;

  if (static_cast<int>(threadIdx.x) >= n_cons) {
    // ---------------- producers ----------------
    const int pw = (threadIdx.x - n_cons) >> 5, lane = threadIdx.x & 31;
    float wb[NCH], ab[NCH];
    if (MODE == kScanDelta) {
#pragma unroll
      for (int i = 0; i < NCH; ++i) {
        const int ch = lane + 32 * i;
        wb[i] = ch < a.DK ? a.w_bias[h * a.DK + ch] : 0.0f;
        ab[i] = ch < a.DK ? a.a_bias[h * a.DK + ch] : 0.0f;
      }
    }
    const T* proj = static_cast<const T*>(a.proj);
    for (int c = 0; c < n_chunks; ++c) {
      const int buf = c & 1;
      if (c >= 2) buffer_sync<kBarEmpty>(buf, all);
      const int n = min(kChunk, seq.len - c * kChunk);
#pragma unroll 2
      for (int t = pw; t < n; t += kProducers / 32) {
        const size_t row = static_cast<size_t>(seq.row0) + c * kChunk + t;
        const T* pr = proj + row * a.ld;
        float* dst = vec + (buf * kChunk + t) * NV * DKP;
        float kk[NCH], rr[NCH];
#pragma unroll
        for (int i = 0; i < NCH; ++i) {
          const int ch = lane + 32 * i;
          const bool in = ch < a.DK;
          kk[i] = in ? ldf(pr + a.off_k + h * a.DK + ch) : 0.0f;
          rr[i] = in ? ldf(pr + a.off_q + h * a.DK + ch) : 0.0f;
        }
        if (MODE == kScanDelta) {
          float wz[NCH], az[NCH], ss = 0.0f;
          const T* wr = static_cast<const T*>(a.wz) + row * a.ld_wz;
#pragma unroll
          for (int i = 0; i < NCH; ++i) {
            const int ch = lane + 32 * i;
            const bool in = ch < a.DK;
            wz[i] = in ? ldf(wr + h * a.DK + ch) : 0.0f;
            az[i] = in ? ldf(pr + a.off_a + h * a.DK + ch) : 0.0f;
            ss = fmaf(kk[i], kk[i], ss);
          }
          const float inv = 1.0f / sqrtf(warp_sum(ss) + a.unit_eps);
#pragma unroll
          for (int i = 0; i < NCH; ++i) {
            const int ch = lane + 32 * i;
            if (ch < DKP) {
              const float u = kk[i] * inv;
              dst[ch] = u;
              dst[DKP + ch] = expf(-a.decay_coef * sigmoid_f(wz[i] + wb[i]));
              dst[2 * DKP + ch] = -sigmoid_f(az[i] + ab[i]) * u;
              dst[3 * DKP + ch] = kk[i];
              dst[4 * DKP + ch] = rr[i];
            }
          }
        } else {
#pragma unroll
          for (int i = 0; i < NCH; ++i) {
            const int ch = lane + 32 * i;
            if (ch < DKP) {
              dst[ch] = silu_f(kk[i]);
              dst[DKP + ch] = silu_f(rr[i]);
            }
          }
        }
        for (int cc = lane; cc < cols; cc += 32) {
          float v = col0 + cc < a.DV ? ldf(pr + a.off_v + h * a.DV + col0 + cc) : 0.0f;
          if (MODE == kScanDecay) v = silu_f(v);
          val[(buf * kChunk + t) * cols + cc] = v;
        }
      }
      buffer_arrive<kBarFull>(buf, all);
    }
    return;
  }

  // ---------------- consumers ----------------
  const int ks = threadIdx.x % KS, cg = threadIdx.x / KS;
  const bool live = cg < col_groups;
  const int col = col0 + 2 * cg;
  const bool in0 = live && col < a.DV, in1 = live && col + 1 < a.DV;
  const bool pair = in1 && (a.DV & 1) == 0;  // the two columns as one 8-byte access
  float* state = a.state + (static_cast<size_t>(seq.slot) * a.H + h) * a.DK * a.DV;
  f32x2 S0[kRows / 2], S1[kRows / 2];  // columns col, col + 1; channels 4 (m KS + ks) + {0, 1}, {2, 3}
#pragma unroll
  for (int m = 0; m < kRows / 4; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float s[2][2];
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int ch = 4 * (m * KS + ks) + 2 * e + f;
        const bool in = seq.pos > 0 && ch < a.DK;
        if (pair) {
          const float2 p = in ? *reinterpret_cast<const float2*>(state + static_cast<size_t>(ch) * a.DV + col) : make_float2(0.0f, 0.0f);
          s[f][0] = p.x; s[f][1] = p.y;
        } else {
          s[f][0] = in && in0 ? state[static_cast<size_t>(ch) * a.DV + col] : 0.0f;
          s[f][1] = in && in1 ? state[static_cast<size_t>(ch) * a.DV + col + 1] : 0.0f;
        }
      }
      S0[2 * m + e] = pack2(s[0][0], s[1][0]);
      S1[2 * m + e] = pack2(s[0][1], s[1][1]);
    }
  const f32x2 dec2 = MODE == kScanDecay ? pack2(a.decay[h], a.decay[h]) : 0ull;
  const int vcol = live ? 2 * cg : 0;
  float* orow = a.o + static_cast<size_t>(seq.row0) * a.ldo + h * a.DV + col;
  const bool opair = pair && (a.ldo & 1) == 0;

  for (int c = 0; c < n_chunks; ++c) {
    const int buf = c & 1;
    buffer_sync<kBarFull>(buf, all);
    const int n = min(kChunk, seq.len - c * kChunk);
    const ulonglong2* vp = reinterpret_cast<const ulonglong2*>(vec + buf * kChunk * NV * DKP) + ks;
    const float* vv = val + buf * kChunk * cols + vcol;
#pragma unroll 2
    for (int t = 0; t < n; ++t, vp += NV * DKP / 4, vv += cols) {
      const float2 v = *reinterpret_cast<const float2*>(vv);
      const f32x2 v0 = pack2(v.x, v.x), v1 = pack2(v.y, v.y);
      f32x2 o0 = 0ull, o1 = 0ull;
      if (MODE == kScanDelta) {
        f32x2 p0 = 0ull, p1 = 0ull, q0 = 0ull, q1 = 0ull;
#pragma unroll
        for (int m = 0; m < kRows / 4; ++m) {
          const ulonglong2 u = vp[m * KS];
          p0 = fma2(u.x, S0[2 * m], p0);
          p1 = fma2(u.x, S1[2 * m], p1);
          q0 = fma2(u.y, S0[2 * m + 1], q0);
          q1 = fma2(u.y, S1[2 * m + 1], q1);
        }
        const float2 a0 = unpack2(p0), b0 = unpack2(q0), a1 = unpack2(p1), b1 = unpack2(q1);
        const float s0 = lane_group_sum<KS>((a0.x + a0.y) + (b0.x + b0.y));
        const float s1 = lane_group_sum<KS>((a1.x + a1.y) + (b1.x + b1.y));
        const f32x2 x0 = pack2(s0, s0), x1 = pack2(s1, s1);
#pragma unroll
        for (int m = 0; m < kRows / 4; ++m) {
          const ulonglong2 w = vp[DKP / 4 + m * KS], na = vp[2 * DKP / 4 + m * KS], k = vp[3 * DKP / 4 + m * KS],
                           r = vp[4 * DKP / 4 + m * KS];
          S0[2 * m] = fma2(w.x, S0[2 * m], fma2(na.x, x0, mul2(k.x, v0)));
          S1[2 * m] = fma2(w.x, S1[2 * m], fma2(na.x, x1, mul2(k.x, v1)));
          S0[2 * m + 1] = fma2(w.y, S0[2 * m + 1], fma2(na.y, x0, mul2(k.y, v0)));
          S1[2 * m + 1] = fma2(w.y, S1[2 * m + 1], fma2(na.y, x1, mul2(k.y, v1)));
          o0 = fma2(r.y, S0[2 * m + 1], fma2(r.x, S0[2 * m], o0));
          o1 = fma2(r.y, S1[2 * m + 1], fma2(r.x, S1[2 * m], o1));
        }
      } else {
#pragma unroll
        for (int m = 0; m < kRows / 4; ++m) {
          const ulonglong2 k = vp[m * KS], r = vp[DKP / 4 + m * KS];
          S0[2 * m] = fma2(dec2, S0[2 * m], mul2(k.x, v0));
          S1[2 * m] = fma2(dec2, S1[2 * m], mul2(k.x, v1));
          S0[2 * m + 1] = fma2(dec2, S0[2 * m + 1], mul2(k.y, v0));
          S1[2 * m + 1] = fma2(dec2, S1[2 * m + 1], mul2(k.y, v1));
          o0 = fma2(r.y, S0[2 * m + 1], fma2(r.x, S0[2 * m], o0));
          o1 = fma2(r.y, S1[2 * m + 1], fma2(r.x, S1[2 * m], o1));
        }
      }
      const float2 e0 = unpack2(o0), e1 = unpack2(o1);
      const float y0 = lane_group_sum<KS>(e0.x + e0.y), y1 = lane_group_sum<KS>(e1.x + e1.y);
      if (ks == 0) {
        if (opair) {
          *reinterpret_cast<float2*>(orow) = make_float2(y0, y1);
        } else {
          if (in0) orow[0] = y0;
          if (in1) orow[1] = y1;
        }
      }
      orow += a.ldo;
    }
    if (c + 2 < n_chunks) buffer_arrive<kBarEmpty>(buf, all);
  }
  pdl_trigger();
#pragma unroll
  for (int m = 0; m < kRows / 4; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float2 s0 = unpack2(S0[2 * m + e]), s1 = unpack2(S1[2 * m + e]);
#pragma unroll
      for (int f = 0; f < 2; ++f) {
        const int ch = 4 * (m * KS + ks) + 2 * e + f;
        if (ch >= a.DK) continue;
        float* p = state + static_cast<size_t>(ch) * a.DV + col;
        const float c0 = f ? s0.y : s0.x, c1 = f ? s1.y : s1.x;
        if (pair) {
          *reinterpret_cast<float2*>(p) = make_float2(c0, c1);
        } else {
          if (in0) p[0] = c0;
          if (in1) p[1] = c1;
        }
      }
    }
}

// four consecutive elements
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const bf16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(bf16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// ---- group norm with a sigmoid gate behind a matrix-state mixer ----
// Vector form: LPG lanes hold a whole group of 4 * LPG elements; LPG = 0: the CTA holds the whole row, which is one group
// (VPT vectors per thread).
template <typename T, int LPG, int VPT>
__global__ void __launch_bounds__(256) gated_rms_norm_vec_kernel(const float* __restrict__ o, long long ldo, const T* __restrict__ gate,
                                                                 long long ldg, const float* __restrict__ w, T* __restrict__ out,
                                                                 long long ldout, int T_rows, int cols, float eps, float scale) {
  pdl_wait();
  pdl_trigger();
  __shared__ float red[8];
  const int nv = cols >> 2;
  float4 v[VPT], g[VPT];
  long long row[VPT];
  int c[VPT];
  bool in[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    if (LPG) {
      const unsigned idx = (blockIdx.x * VPT + i) * 256u + threadIdx.x;  // vectors of all rows in order
      in[i] = idx < static_cast<unsigned>(T_rows) * static_cast<unsigned>(nv);
      row[i] = in[i] ? idx / static_cast<unsigned>(nv) : 0;
      c[i] = in[i] ? static_cast<int>(idx % static_cast<unsigned>(nv)) * 4 : 0;
    } else {
      row[i] = blockIdx.x;
      in[i] = static_cast<int>(threadIdx.x) + i * 256 < nv;
      c[i] = in[i] ? (threadIdx.x + i * 256) * 4 : 0;
    }
    v[i] = ld4(o + row[i] * ldo + c[i]);
    g[i] = ld4(gate + row[i] * ldg + c[i]);
  }
  float total = 0.0f, sq[VPT];
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    sq[i] = in[i] ? fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, v[i].w * v[i].w))) : 0.0f;
    if (LPG) {
#pragma unroll
      for (int d = LPG / 2; d > 0; d >>= 1) sq[i] += __shfl_xor_sync(0xffffffffu, sq[i], d);
    }
    total += sq[i];
  }
  if (!LPG) {
    total = warp_sum(total);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = total;
    __syncthreads();
    total = warp_sum((threadIdx.x & 31) < 8 ? red[threadIdx.x & 31] : 0.0f);
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    if (!in[i]) continue;
    const float rr = scale / sqrtf(LPG ? sq[i] / (4.0f * LPG) + eps : total / static_cast<float>(cols) + eps);
    const float4 wv = __ldg(reinterpret_cast<const float4*>(w + c[i]));
    st4(out + row[i] * ldout + c[i],
        make_float4(v[i].x * rr * wv.x * sigmoid_f(g[i].x), v[i].y * rr * wv.y * sigmoid_f(g[i].y),
                    v[i].z * rr * wv.z * sigmoid_f(g[i].z), v[i].w * rr * wv.w * sigmoid_f(g[i].w)));
  }
}

// Any group size and alignment: a warp per (token, group), scalar accesses.
template <typename T>
__global__ void gated_rms_norm_kernel(const float* __restrict__ o, long long ldo, const T* __restrict__ gate, long long ldg,
                                      const float* __restrict__ w, T* __restrict__ out, long long ldout, int T_rows, int groups,
                                      int group_size, float eps, float scale) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const long long unit = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(T_rows) * groups) return;
  const long long row = unit / groups;
  const int c0 = static_cast<int>(unit % groups) * group_size;
  const float* src = o + row * ldo + c0;
  float sq = 0.0f;
  for (int c = lane; c < group_size; c += 32) sq = fmaf(src[c], src[c], sq);
  const float rr = scale / sqrtf(warp_sum(sq) / static_cast<float>(group_size) + eps);
  const T* g = gate + row * ldg + c0;
  T* dst = out + row * ldout + c0;
  for (int c = lane; c < group_size; c += 32) stf(dst + c, src[c] * rr * w[c0 + c] * sigmoid_f(ldf(g + c)));
}

// ---- minimal GRU.  The gates read only the current token, so S_t = A_t S_{t-1} + B_t is a scan of affine maps: warp w of
// a CTA takes TS consecutive tokens of 64 channels (a pair per lane), composes their maps, the compositions meet in shared
// memory, and every warp finishes its own tokens from the state that enters them.  The raw projections of the next tile are
// requested before the exchange. ----
// Two neighbouring elements as loaded: converted where they are used, not where they are requested.
template <typename T> struct Pair;
template <> struct Pair<float> { typedef float2 raw; static __device__ float2 f(raw v) { return v; } };
template <> struct Pair<bf16> { typedef uint32_t raw; static __device__ float2 f(raw v) { return make_float2(bf16_lo(v), bf16_hi(v)); } };
template <bool VEC>
__device__ __forceinline__ float2 ld_two(const float* p, bool second) {
  if (VEC) return *reinterpret_cast<const float2*>(p);
  return make_float2(p[0], second ? p[1] : 0.0f);
}
template <bool VEC>
__device__ __forceinline__ uint32_t ld_two(const bf16* p, bool second) {
  if (VEC) return *reinterpret_cast<const uint32_t*>(p);
  const uint16_t* q = reinterpret_cast<const uint16_t*>(p);
  return q[0] | (second ? static_cast<uint32_t>(q[1]) << 16 : 0u);
}
template <bool VEC>
__device__ __forceinline__ void st_two(float* p, float2 v, bool second) {
  if (VEC) { *reinterpret_cast<float2*>(p) = v; return; }
  p[0] = v.x;
  if (second) p[1] = v.y;
}
template <bool VEC>
__device__ __forceinline__ void st_two(bf16* p, float2 v, bool second) {
  if (VEC) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(v.x, v.y); return; }
  p[0] = __float2bfloat16_rn(v.x);
  if (second) p[1] = __float2bfloat16_rn(v.y);
}

// sigmoid at the accuracy the element type calls for: f32 models get the full-precision functions
template <typename T> __device__ __forceinline__ float sigmoid_as(float x);
template <> __device__ __forceinline__ float sigmoid_as<float>(float x) { return sigmoid_f(x); }
template <> __device__ __forceinline__ float sigmoid_as<bf16>(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float gru_candidate(float u) { return u >= 0.0f ? u + 0.5f : sigmoid_as<T>(u); }

template <typename T, int TS, bool VEC>
__global__ void __launch_bounds__(512) min_gru_kernel(const MinGru a, const SeqDesc* __restrict__ seqs) {
  __shared__ float2 sA[2][16][32], sB[2][16][32];
  const SeqDesc seq = seqs[blockIdx.y];  // written well before the kernel in front of this one
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int ch = blockIdx.x * 64 + 2 * lane;
  const bool in = ch < a.W, second = ch + 1 < a.W;
  const int cl = in ? ch : 0;
  const float2 zb = in ? make_float2(a.z_bias[ch], second ? a.z_bias[ch + 1] : 0.0f) : make_float2(0.0f, 0.0f);
  const float2 xb = in ? make_float2(a.x_bias[ch], second ? a.x_bias[ch + 1] : 0.0f) : make_float2(0.0f, 0.0f);
  pdl_wait();
  pdl_trigger();
  float* st = a.state + static_cast<size_t>(seq.slot) * a.W + cl;
  float2 S = make_float2(0.0f, 0.0f);
  if (seq.pos > 0) S = make_float2(st[0], second ? st[1] : 0.0f);
  const int tile = warps * TS;
  typename Pair<T>::raw z[TS], u[TS], g[TS];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < TS; ++i) {
      const int t = t0 + warp * TS + i;
      const T* p = static_cast<const T*>(a.proj) + (static_cast<size_t>(seq.row0) + (t < seq.len ? t : 0)) * a.ld + cl;
      z[i] = ld_two<VEC>(p + a.off_z, second);
      u[i] = ld_two<VEC>(p + a.off_x, second);
      g[i] = ld_two<VEC>(p + a.off_g, second);
    }
  };
  fetch(0);
  int par = 0;
  for (int t0 = 0; t0 < seq.len; t0 += tile, par ^= 1) {
    const int first = t0 + warp * TS;
    float2 A[TS], B[TS], G[TS], pa = make_float2(1.0f, 1.0f), pb = make_float2(0.0f, 0.0f);
#pragma unroll
    for (int i = 0; i < TS; ++i) {
      const float2 zr = Pair<T>::f(z[i]), ur = Pair<T>::f(u[i]), gr = Pair<T>::f(g[i]);
      const float2 zz = make_float2(sigmoid_as<T>(zr.x + zb.x), sigmoid_as<T>(zr.y + zb.y));
      const bool on = first + i < seq.len;
      A[i] = on ? make_float2(1.0f - zz.x, 1.0f - zz.y) : make_float2(1.0f, 1.0f);
      B[i] = on ? make_float2(zz.x * gru_candidate<T>(ur.x + xb.x), zz.y * gru_candidate<T>(ur.y + xb.y)) : make_float2(0.0f, 0.0f);
      G[i] = make_float2(gr.x * sigmoid_as<T>(gr.x) * a.scale, gr.y * sigmoid_as<T>(gr.y) * a.scale);
      pa = make_float2(pa.x * A[i].x, pa.y * A[i].y);
      pb = make_float2(fmaf(A[i].x, pb.x, B[i].x), fmaf(A[i].y, pb.y, B[i].y));
    }
    if (t0 + tile < seq.len) fetch(t0 + tile);
    float2 mine = S;
    if (warps > 1) {
      sA[par][warp][lane] = pa;
      sB[par][warp][lane] = pb;
      __syncthreads();  // the other parity's buffer is rewritten only behind the next tile's barrier
      for (int w = 0; w < warps; ++w) {
        if (w == warp) mine = S;
        const float2 wa = sA[par][w][lane], wb = sB[par][w][lane];
        S = make_float2(fmaf(wa.x, S.x, wb.x), fmaf(wa.y, S.y, wb.y));
      }
    } else {
      S = make_float2(fmaf(pa.x, S.x, pb.x), fmaf(pa.y, S.y, pb.y));
    }
#pragma unroll
    for (int i = 0; i < TS; ++i) {
      if (in && first + i < seq.len) {
        mine = make_float2(fmaf(A[i].x, mine.x, B[i].x), fmaf(A[i].y, mine.y, B[i].y));
        st_two<VEC>(static_cast<T*>(a.out) + (static_cast<size_t>(seq.row0) + first + i) * a.ldout + ch,
                    make_float2(mine.x * G[i].x, mine.y * G[i].y), second);
      }
    }
  }
  if (in && warp == 0) {
    st[0] = S.x;
    if (second) st[1] = S.y;
  }
}

// ---- one token per sequence (decode): the state streams through once ----
// CTA = one (sequence, head): a thread holds RPT rows x 4 columns of the state, requested before the dependency wait (the
// state was written a whole step ago), so the whole state of the head is in flight while the projections are finished
// and the key-side vectors are built in shared memory.  Row groups meet in shared memory for u^T S and for the output.
// With a.norm_w (delta) the head's group norm and gate are applied on the way out.
template <typename T, int MODE, int RPT>
__global__ void __launch_bounds__(512) state_step_kernel(const StateScan a, const SeqDesc* __restrict__ seqs, int groups) {
  constexpr bool DELTA = MODE == kScanDelta;
  extern __shared__ __align__(16) float step_sh[];
  const int dkp = (a.DK + 3) & ~3;
  float* vec = step_sh;                          // [5][dkp], rows 1 .. 4: w, -a, k, q
  float* val = vec + 5 * dkp;                    // [DV]
  float* red = val + a.DV;                       // [groups][DV]
  const SeqDesc seq = seqs[blockIdx.y];
  const int h = blockIdx.x, c4 = (threadIdx.x % (a.DV >> 2)) * 4, rg = threadIdx.x / (a.DV >> 2);
  const bool live = rg < groups;
  float* state = a.state + (static_cast<size_t>(seq.slot) * a.H + h) * a.DK * a.DV + c4;
  float4 S[RPT];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int ch = rg * RPT + r;
    S[r] = live && seq.pos > 0 && ch < a.DK ? ld4(state + static_cast<size_t>(ch) * a.DV) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  }
  pdl_wait();
  pdl_trigger();
  const size_t row = seq.row0;
  const T* pr = static_cast<const T*>(a.proj) + row * a.ld;
  const int hk = h * a.DK, hv = h * a.DV;
  for (int c = threadIdx.x; c < a.DK; c += blockDim.x) {
    const float k = ldf(pr + a.off_k + hk + c), q = ldf(pr + a.off_q + hk + c);
    if (DELTA) {
      vec[dkp + c] = expf(-a.decay_coef * sigmoid_f(ldf(static_cast<const T*>(a.wz) + row * a.ld_wz + hk + c) + a.w_bias[hk + c]));
      vec[2 * dkp + c] = -sigmoid_f(ldf(pr + a.off_a + hk + c) + a.a_bias[hk + c]);
    }
    vec[3 * dkp + c] = DELTA ? k : silu_f(k);
    vec[4 * dkp + c] = DELTA ? q : silu_f(q);
  }
  for (int c = threadIdx.x; c < a.DV; c += blockDim.x) {
    const float v = ldf(pr + a.off_v + hv + c);
    val[c] = DELTA ? v : silu_f(v);
  }
  __syncthreads();
  const float4 v = live ? *reinterpret_cast<const float4*>(val + c4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
  float4 p = make_float4(0.0f, 0.0f, 0.0f, 0.0f), o = p;
  float inv = 1.0f;
  if (DELTA) {
    float ss = 0.0f;
    for (int c = threadIdx.x & 31; c < a.DK; c += 32) ss = fmaf(vec[3 * dkp + c], vec[3 * dkp + c], ss);
    inv = 1.0f / sqrtf(warp_sum(ss) + a.unit_eps);  // u = k * inv, the same in every warp
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int ch = rg * RPT + r;
      const float k = live && ch < a.DK ? vec[3 * dkp + ch] * inv : 0.0f;
      p = make_float4(fmaf(k, S[r].x, p.x), fmaf(k, S[r].y, p.y), fmaf(k, S[r].z, p.z), fmaf(k, S[r].w, p.w));
    }
    if (live) *reinterpret_cast<float4*>(red + rg * a.DV + c4) = p;
    __syncthreads();
    p = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (live)
      for (int g = 0; g < groups; ++g) {
        const float4 x = *reinterpret_cast<const float4*>(red + g * a.DV + c4);
        p = make_float4(p.x + x.x, p.y + x.y, p.z + x.z, p.w + x.w);
      }
    __syncthreads();
  }
  const float dec = DELTA ? 0.0f : a.decay[h];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int ch = rg * RPT + r;
    if (!live || ch >= a.DK) continue;
    const float w = DELTA ? vec[dkp + ch] : dec, k = vec[3 * dkp + ch], q = vec[4 * dkp + ch];
    const float au = DELTA ? vec[2 * dkp + ch] * k * inv : 0.0f;
    S[r] = make_float4(fmaf(w, S[r].x, fmaf(au, p.x, k * v.x)), fmaf(w, S[r].y, fmaf(au, p.y, k * v.y)),
                       fmaf(w, S[r].z, fmaf(au, p.z, k * v.z)), fmaf(w, S[r].w, fmaf(au, p.w, k * v.w)));
    o = make_float4(fmaf(q, S[r].x, o.x), fmaf(q, S[r].y, o.y), fmaf(q, S[r].z, o.z), fmaf(q, S[r].w, o.w));
    st4(state + static_cast<size_t>(ch) * a.DV, S[r]);
  }
  if (live) *reinterpret_cast<float4*>(red + rg * a.DV + c4) = o;
  __syncthreads();
  float sq = 0.0f;
  for (int c = threadIdx.x; c < a.DV; c += blockDim.x) {
    float y = 0.0f;
    for (int g = 0; g < groups; ++g) y += red[g * a.DV + c];
    if (a.norm_w) val[c] = y;  // (v has been read)
    else a.o[row * a.ldo + hv + c] = y;
    sq = fmaf(y, y, sq);
  }
  if (!a.norm_w) return;
  __syncthreads();
  sq = 0.0f;
  for (int c = threadIdx.x & 31; c < a.DV; c += 32) sq = fmaf(val[c], val[c], sq);
  const float rr = a.out_scale / sqrtf(warp_sum(sq) / static_cast<float>(a.DV) + a.norm_eps);
  for (int c = threadIdx.x; c < a.DV; c += blockDim.x)
    stf(static_cast<T*>(a.out) + row * a.ldout + hv + c, val[c] * rr * a.norm_w[hv + c] * sigmoid_f(ldf(pr + a.off_g + hv + c)));
}

// Rows per thread and row groups of the one-token kernel; false if the head does not fit it.
bool step_shape(const StateScan& a, int& rpt, int& groups) {
  if (a.DV & 3) return false;
  rpt = (a.DV / 4) * ((a.DK + 7) / 8) <= 512 ? 8 : 16;
  groups = (a.DK + rpt - 1) / rpt;
  return (a.DV / 4) * groups <= 512;
}
int step_smem(const StateScan& a, int groups) { return (5 * ((a.DK + 3) & ~3) + a.DV + groups * a.DV) * static_cast<int>(sizeof(float)); }

template <typename T, int MODE>
int launch_step(const StateScan& a, const SeqDesc* seqs, int n_seqs, int rpt, int groups, cudaStream_t st) {
  const int threads = ((a.DV / 4) * groups + 31) / 32 * 32, smem = step_smem(a, groups);
  if (rpt == 8) launch_kernel(state_step_kernel<T, MODE, 8>, dim3(a.H, n_seqs), dim3(threads), smem, st, 1, a, seqs, groups);
  else launch_kernel(state_step_kernel<T, MODE, 16>, dim3(a.H, n_seqs), dim3(threads), smem, st, 1, a, seqs, groups);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int MODE, int KS>
int launch_scan(const StateScan& a, const SeqDesc* seqs, int n_seqs, bool prepare_only, cudaStream_t st) {
  constexpr int NV = scan_vectors(MODE), DKP = KS * kRows;
  constexpr int max_groups = kMaxConsumers / KS;
  static std::atomic<unsigned long long> done{0};  // one bit per device; threads may race to set it
  int dev = 0;
  cudaGetDevice(&dev);
  if (!(dev < 64 && (done.load(std::memory_order_acquire) >> dev) & 1ull)) {
    const int most = 2 * kChunk * (NV * DKP + 2 * max_groups) * static_cast<int>(sizeof(float));
    const cudaError_t e = cudaFuncSetAttribute(state_scan_kernel<T, MODE, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e != cudaSuccess) return static_cast<int>(e);
    if (dev < 64) done.fetch_or(1ull << dev, std::memory_order_release);
  }
  if (prepare_only) return 0;
  int groups = (a.DV + 1) / 2;
  if (groups > max_groups) groups = max_groups;
  const int threads = (groups * KS + 31) / 32 * 32 + kProducers;
  const int smem = 2 * kChunk * (NV * DKP + 2 * groups) * static_cast<int>(sizeof(float));
  const dim3 grid((a.DV + 2 * groups - 1) / (2 * groups), a.H, n_seqs);
  launch_kernel(state_scan_kernel<T, MODE, KS>, grid, dim3(threads), smem, st, 1, a, seqs, groups);
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int MODE>
int dispatch_scan(const StateScan& a, const SeqDesc* seqs, int n_seqs, bool prep, cudaStream_t st) {
  if (a.DK <= 16) return launch_scan<T, MODE, 1>(a, seqs, n_seqs, prep, st);
  if (a.DK <= 32) return launch_scan<T, MODE, 2>(a, seqs, n_seqs, prep, st);
  if (a.DK <= 64) return launch_scan<T, MODE, 4>(a, seqs, n_seqs, prep, st);
  if (a.DK <= 128) return launch_scan<T, MODE, 8>(a, seqs, n_seqs, prep, st);
  return launch_scan<T, MODE, 16>(a, seqs, n_seqs, prep, st);
}

int scan_any(const StateScan& a, const SeqDesc* seqs, int n_seqs, bool prep, cudaStream_t st) {
  if (a.mode == kScanDelta)
    return a.f32 ? dispatch_scan<float, kScanDelta>(a, seqs, n_seqs, prep, st) : dispatch_scan<bf16, kScanDelta>(a, seqs, n_seqs, prep, st);
  return a.f32 ? dispatch_scan<float, kScanDecay>(a, seqs, n_seqs, prep, st) : dispatch_scan<bf16, kScanDecay>(a, seqs, n_seqs, prep, st);
}

}  // namespace

bool state_scan_supports(int dk, int dv) { return dk >= 1 && dk <= 256 && dv >= 1; }

// Function attributes of every variant, outside any stream capture.
int state_scan_prepare() {
  for (int mode = 0; mode < 2; ++mode)
    for (int f32 = 0; f32 < 2; ++f32)
      for (int dk : {16, 32, 64, 128, 256}) {
        StateScan a{};
        a.mode = mode; a.f32 = f32; a.DK = dk;
        const int rc = scan_any(a, nullptr, 0, true, nullptr);
        if (rc) return rc;
      }
  return chunk_scan_prepare();
}

int state_scan(const StateScan& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st, bool* normed) {
  if (!a.proj || !a.state || !a.o || !seqs || n_seqs <= 0 || n_seqs > 65535 || max_len <= 0 || a.H <= 0 || a.H > 65535 ||
      !state_scan_supports(a.DK, a.DV))
    return TEENY_ERR_BAD_ARG;
  if (a.mode == kScanDelta ? (!a.wz || !a.w_bias || !a.a_bias) : (a.mode != kScanDecay || !a.decay)) return TEENY_ERR_BAD_ARG;
  if (normed) *normed = false;
  // prompts in bf16: 16 tokens at a time on the tensor cores; single tokens: one pass over the state; else token by token
  if (chunk_scan_supports(a, max_len)) return chunk_scan(a, seqs, n_seqs, st);
  int rpt, groups;
  if (max_len == 1 && step_shape(a, rpt, groups)) {
    StateScan b = a;
    if (!normed || !a.out) b.norm_w = nullptr;
    if (normed) *normed = b.norm_w != nullptr;
    if (a.mode == kScanDelta)
      return a.f32 ? launch_step<float, kScanDelta>(b, seqs, n_seqs, rpt, groups, st) : launch_step<bf16, kScanDelta>(b, seqs, n_seqs, rpt, groups, st);
    return a.f32 ? launch_step<float, kScanDecay>(b, seqs, n_seqs, rpt, groups, st) : launch_step<bf16, kScanDecay>(b, seqs, n_seqs, rpt, groups, st);
  }
  return scan_any(a, seqs, n_seqs, false, st);
}

namespace {
template <typename T>
int launch_gated_norm(const float* o, long long ldo, const void* gate, long long ldg, const float* w, void* out, long long ldout, int T_rows,
                      int cols, int group_size, float eps, float scale, cudaStream_t st) {
  const T* g = static_cast<const T*>(gate);
  T* y = static_cast<T*>(out);
  const uintptr_t bases = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) |
                          reinterpret_cast<uintptr_t>(out);
  const bool vec = (bases & 15) == 0 && ((ldo | ldg | ldout | cols) & 3) == 0 && static_cast<long long>(T_rows) * cols < (1ll << 32);
  const dim3 block(256);
#define TEENY_GRN(LPG, VPT, GRID) \
  launch_kernel(gated_rms_norm_vec_kernel<T, LPG, VPT>, dim3(GRID), block, 0, st, 1, o, ldo, g, ldg, w, y, ldout, T_rows, cols, eps, scale)
  if (vec && (group_size == 16 || group_size == 32 || group_size == 64 || group_size == 128)) {
    const long long vectors = static_cast<long long>(T_rows) * (cols / 4);
    const unsigned grid = static_cast<unsigned>((vectors + 511) / 512);
    if (group_size == 16) TEENY_GRN(4, 2, grid);
    else if (group_size == 32) TEENY_GRN(8, 2, grid);
    else if (group_size == 64) TEENY_GRN(16, 2, grid);
    else TEENY_GRN(32, 2, grid);
  } else if (vec && group_size == cols && cols <= 8 * 1024) {
    if (cols <= 1024) TEENY_GRN(0, 1, T_rows);
    else if (cols <= 2048) TEENY_GRN(0, 2, T_rows);
    else if (cols <= 4096) TEENY_GRN(0, 4, T_rows);
    else TEENY_GRN(0, 8, T_rows);
  } else {
    const int groups = cols / group_size;
    const long long blocks = (static_cast<long long>(T_rows) * groups + 7) / 8;
    if (blocks > 0x7fffffffLL) return TEENY_ERR_BAD_ARG;
    launch_kernel(gated_rms_norm_kernel<T>, dim3(static_cast<unsigned>(blocks)), block, 0, st, 1, o, ldo, g, ldg, w, y, ldout, T_rows, groups,
                  group_size, eps, scale);
  }
#undef TEENY_GRN
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int launch_min_gru(const MinGru& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  constexpr int TS = 8;
  const dim3 grid((a.W + 63) / 64, n_seqs);
  const bool vec = ((a.W | a.off_z | a.off_x | a.off_g) & 1) == 0 && ((a.ld | a.ldout) & 1) == 0 && (reinterpret_cast<uintptr_t>(a.out) & 7) == 0;
  int warps = (max_len + TS - 1) / TS;
  if (warps > 16) warps = 16;
#define TEENY_GRU(N) \
  vec ? launch_kernel(min_gru_kernel<T, N, true>, grid, dim3(32 * warps), 0, st, 1, a, seqs) \
      : launch_kernel(min_gru_kernel<T, N, false>, grid, dim3(32 * warps), 0, st, 1, a, seqs)
  if (max_len == 1) TEENY_GRU(1);
  else TEENY_GRU(TS);
#undef TEENY_GRU
  return static_cast<int>(cudaGetLastError());
}
}  // namespace

int gated_rms_norm(const float* o, long long ldo, const void* gate, long long ldg, const float* w, void* out, long long ldout,
                   int T, int cols, int group_size, float eps, float scale, bool f32, cudaStream_t st) {
  if (!o || !gate || !w || !out || T <= 0 || cols <= 0 || group_size <= 0 || cols % group_size) return TEENY_ERR_BAD_ARG;
  return f32 ? launch_gated_norm<float>(o, ldo, gate, ldg, w, out, ldout, T, cols, group_size, eps, scale, st)
             : launch_gated_norm<bf16>(o, ldo, gate, ldg, w, out, ldout, T, cols, group_size, eps, scale, st);
}

int min_gru(const MinGru& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  if (!a.proj || !a.z_bias || !a.x_bias || !a.state || !a.out || !seqs || n_seqs <= 0 || n_seqs > 65535 || max_len <= 0 || a.W <= 0)
    return TEENY_ERR_BAD_ARG;
  return a.f32 ? launch_min_gru<float>(a, seqs, n_seqs, max_len, st) : launch_min_gru<bf16>(a, seqs, n_seqs, max_len, st);
}

}  // namespace teeny
