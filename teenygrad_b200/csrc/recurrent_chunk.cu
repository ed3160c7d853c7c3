// Matrix-state recurrences over a prompt, 16 tokens at a time on the tensor cores (bf16 activations).
//
// Delta rule.  With L_t the running sum of log w over a chunk and W_t = exp(L_t) (per key channel), S_t = diag(W_t) X_t
// turns the recurrence into rank-one updates without a decay:
//   p_t = u_t^T S_{t-1} = U_t X_0 + sum_{s<t} (U_t . Ka_s) p_s + (U_t . Kk_s) v_s      U_t = W_{t-1} o u_t
//   o_t = r_t^T S_t     = R_t X_0 + sum_{s<=t} (R_t . Ka_s) p_s + (R_t . Kk_s) v_s     R_t = W_t o r_t
//   S_16 = diag(W_16) (X_0 + sum_s Ka_s p_s + Kk_s v_s)                                Ka_s = -a_s u_s / W_s, Kk_s = k_s / W_s
// so a chunk is four 16 x 16 matrices, one triangular inverse T = (1 - U Ka^T)^{-1} and products with the state.
// Scalar decay.  o_t = d^{t+1} q_t^T S_0 + sum_{s<=t} d^{t-s} (q_t . k_s) v_s, S_n = d^n S_0 + sum_s k_s (d^{n-1-s} v_s); no
// division by a power of d, however small d is.  q, k, v are the activated projections, bf16 tensors.
//
// 32-bit accuracy from bf16 tensor cores: every f32 operand goes in as hi + lo (2^-17), a product of two as hi hi + hi lo
// + lo hi with f32 accumulation, projections as they are (one term); the carried state itself is never rounded (f32
// accumulators from chunk to chunk).
//
// One CTA per (head, sequence).  Warps 0 .. n-1, the consumers, own 16 value columns each and keep S^T [16, DK] as C
// fragments: those are, packed, the A operand of S^T U^T and S^T R^T, whose results (P^T, O^T) are in turn the A operand
// and the layout of the update, so the chain never leaves the registers.  The last eight warps, the producers, build the
// B operands: nothing in them depends on the state, so two groups of four warps take alternate chunks, each in its own
// shared-memory buffer.  Buffers change hands through named barriers.  A group requests the raw projections of its
// next chunk before it turns to the matrices of the current one, in one batch of unconditional loads (branches around
// the loads made every one of them wait for its predecessor: 13 000 cycles per chunk instead of a few hundred).
#include <atomic>

#include "common.cuh"
#include "kernels.h"
#include "mma.cuh"

namespace teeny {

namespace {

constexpr int kC = 16;          // tokens per chunk
constexpr int kGroup = 128;     // threads of a producer group
constexpr int kProducers = 2 * kGroup;
constexpr int kMatLd = 24;      // row stride of the 16 x 16 matrices (48 bytes: conflict-free ldmatrix)
constexpr int kMaxDV = 192;     // 12 consumer warps
constexpr int kBarFull = 1, kBarEmpty = 3, kBarProducers = 5;

__device__ __forceinline__ float sigmoid_f(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return __fdividef(x, 1.0f + __expf(-x)); }

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
__device__ __forceinline__ void group_sync(int group) { buffer_sync<kBarProducers>(group, kGroup); }

// Shared memory of one buffer, byte offsets.  Row tiles [16][DKP + 8] bf16: delta U, R, Ka, Kk, each as hi then lo; decay q
// (in the place of R hi) and k (of Kk hi).  V: delta v; decay v, then d^{n-1-s} v as hi and lo.
template <int DKP>
struct Lay {
  static constexpr int kLd = DKP + 8;
  static constexpr int kTile = kC * kLd * 2;
  static constexpr int tile(int which, int lo) { return (2 * which + lo) * kTile; }
  static constexpr int kMats = 8 * kTile;                      // T, A2, B1, B2: hi, lo [16][24] bf16 each
  static constexpr int mat(int which, int lo) { return kMats + (2 * which + lo) * kC * kMatLd * 2; }
  static constexpr int kScale = kMats + 8 * kC * kMatLd * 2;   // f32 [DKP]: decay of the chunk per key channel
  static constexpr int kV = kScale + DKP * 4;                  // V hi, then lo: [16][DVP + 8] bf16
  static __host__ __device__ constexpr int bytes(int dvp) { return kV + 3 * kC * (dvp + 8) * 2; }
};
constexpr int kU = 0, kR = 1, kKa = 2, kKk = 3;
constexpr int kT = 0, kA2 = 1, kB1 = 2, kB2 = 3;

// Two neighbouring elements of a bf16 row of n as loaded, unconditionally; what lies beyond n is any element of the row (the
// caller clears it when it uses the pair: a select here would wait for the load).  VEC: the pair is 4-byte aligned, n even.
template <bool VEC>
__device__ __forceinline__ uint32_t ld_pair(const bf16* p, int i, int n) {
  if (VEC) return *reinterpret_cast<const uint32_t*>(p + (i < n ? i : 0));
  const uint16_t* q = reinterpret_cast<const uint16_t*>(p);
  return q[i < n ? i : 0] | (static_cast<uint32_t>(q[i + 1 < n ? i + 1 : 0]) << 16);
}
__device__ __forceinline__ uint32_t keep_pair(uint32_t v, int i, int n) {
  return i + 1 < n ? v : (i < n ? v & 0xffffu : 0u);
}
__device__ __forceinline__ float2 f2(uint32_t v) { return make_float2(bf16_lo(v), bf16_hi(v)); }

__device__ __forceinline__ void st_split(uint8_t* tile_hi, uint8_t* tile_lo, int byte_off, float x, float y) {
  uint32_t hi, lo;
  split_bf16x2(x, y, hi, lo);
  *reinterpret_cast<uint32_t*>(tile_hi + byte_off) = hi;
  *reinterpret_cast<uint32_t*>(tile_lo + byte_off) = lo;
}

// acc[2][4] (16 rows x 16 columns) += A B^T for row tiles A, B [16][LD] given as hi / lo, over NK 16-deep steps.
template <int NK, int LD, bool SPLIT>
__device__ __forceinline__ void rows_product(float (&acc)[2][4], uint32_t a_hi, uint32_t a_lo, uint32_t b_hi, uint32_t b_lo, int lane) {
  const uint32_t ao = static_cast<uint32_t>(((lane & 7) + ((lane >> 3) & 1) * 8) * LD + (lane >> 4) * 8) * 2;
  const uint32_t bo = static_cast<uint32_t>(((lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8) * 2;
  float acc2[2][4] = {};
#pragma unroll
  for (int k = 0; k < NK; ++k) {
    uint32_t ah[4], al[4], bh[4], bl[4];
    ldsm_x4(ah, a_hi + ao + k * 32);
    ldsm_x4(bh, b_hi + bo + k * 32);
    if (SPLIT) {
      ldsm_x4(al, a_lo + ao + k * 32);
      ldsm_x4(bl, b_lo + bo + k * 32);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      mma_bf16_16816(acc[n], ah[0], ah[1], ah[2], ah[3], bh[2 * n], bh[2 * n + 1]);
      if (!SPLIT) continue;
      mma_bf16_16816(acc2[n], ah[0], ah[1], ah[2], ah[3], bl[2 * n], bl[2 * n + 1]);
      mma_bf16_16816(acc2[n], al[0], al[1], al[2], al[3], bh[2 * n], bh[2 * n + 1]);
    }
  }
  if (SPLIT) {
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[n][e] += acc2[n][e];
  }
}

// acc += A B for an A fragment given as hi / lo and a 16 x 16 matrix stored [n][k] as hi / lo.
__device__ __forceinline__ void frag_mat(float (&acc)[2][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], bool has_lo,
                                         uint32_t m_hi, uint32_t m_lo, uint32_t bo) {
  uint32_t bh[4], bl[4];
  ldsm_x4(bh, m_hi + bo);
  ldsm_x4(bl, m_lo + bo);
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    mma_bf16_16816(acc[n], ah[0], ah[1], ah[2], ah[3], bh[2 * n], bh[2 * n + 1]);
    mma_bf16_16816(acc[n], ah[0], ah[1], ah[2], ah[3], bl[2 * n], bl[2 * n + 1]);
    if (has_lo) mma_bf16_16816(acc[n], al[0], al[1], al[2], al[3], bh[2 * n], bh[2 * n + 1]);
  }
}

__device__ __forceinline__ void split_frag(const float (&x)[4], const float (&y)[4], uint32_t (&hi)[4], uint32_t (&lo)[4]) {
  split_bf16x2(x[0], x[1], hi[0], lo[0]);
  split_bf16x2(x[2], x[3], hi[1], lo[1]);
  split_bf16x2(y[0], y[1], hi[2], lo[2]);
  split_bf16x2(y[2], y[3], hi[3], lo[3]);
}

template <int MODE, int NK, int NV, bool VEC, int THREADS, int BLOCKS>  // NV = value columns / 64, rounded up
__global__ void __launch_bounds__(THREADS, BLOCKS) chunk_scan_kernel(const StateScan a, const SeqDesc* __restrict__ seqs, int dvp) {
  constexpr int DKP = 16 * NK, NP = DKP / 64, LD = DKP + 8;
  constexpr bool DELTA = MODE == kScanDelta;
  using L = Lay<DKP>;
  extern __shared__ __align__(128) uint8_t chunk_smem[];
  __shared__ float sh_tot[2][4][DELTA ? DKP : 1];   // producer groups: log-decay sums of each warp's four tokens
  __shared__ float sh_a1[2][kC][kC + 1];  // producer groups: U Ka^T, strictly lower, ...
  __shared__ float sh_inv[2][kC][kC + 1]; // ... and the diagonal blocks of the inverse, with the product between them
  __shared__ float sh_pow[kC + 1];
  const int buf_bytes = L::bytes(dvp), ldv = dvp + 8;
  const int n_cons = blockDim.x - kProducers;
  const int lane = threadIdx.x & 31;
  pdl_wait();
  const SeqDesc seq = seqs[blockIdx.y];
  const int h = blockIdx.x;
  const int n_chunks = (seq.len + kC - 1) / kC;
  if (!DELTA) {  // powers of the head's decay
    if (threadIdx.x <= kC) sh_pow[threadIdx.x] = powf(a.decay[h], static_cast<float>(threadIdx.x));
    __syncthreads();
  }

  if (static_cast<int>(threadIdx.x) >= n_cons) {
    // ---------------- producers: warp pw of a group takes tokens 4 pw .. 4 pw + 3 of a chunk, a lane NP channel pairs ----
    const int grp = (threadIdx.x - n_cons) / kGroup, pw = ((threadIdx.x - n_cons) >> 5) & 3;
    const bf16* proj = static_cast<const bf16*>(a.proj);
    const bf16* wzp = static_cast<const bf16*>(a.wz);
    const int hk = h * a.DK, hv = h * a.DV;
    float2 wb[NP], ab[NP];
    if (DELTA) {
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int c = 2 * lane + 64 * i;
        wb[i] = make_float2(c < a.DK ? a.w_bias[hk + c] : 0.0f, c + 1 < a.DK ? a.w_bias[hk + c + 1] : 0.0f);
        ab[i] = make_float2(c < a.DK ? a.a_bias[hk + c] : 0.0f, c + 1 < a.DK ? a.a_bias[hk + c + 1] : 0.0f);
      }
    }
    uint32_t rk[4][NP], rq[4][NP], rw[4][NP], ra[4][NP];  // raw projections of the chunk, bf16 pairs
    auto fetch = [&](int c) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = c * kC + 4 * pw + j;
        const bool in = t < seq.len;
        const size_t row = static_cast<size_t>(seq.row0) + (in ? t : 0);
        const bf16* pr = proj + row * a.ld + hk;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const int ch = 2 * lane + 64 * i;
          rk[j][i] = ld_pair<VEC>(pr + a.off_k, ch, a.DK);
          rq[j][i] = ld_pair<VEC>(pr + a.off_q, ch, a.DK);
          if (DELTA) {
            rw[j][i] = ld_pair<VEC>(wzp + row * a.ld_wz + hk, ch, a.DK);
            ra[j][i] = ld_pair<VEC>(pr + a.off_a, ch, a.DK);
          }
        }
      }
    };
    if (grp < n_chunks) fetch(grp);
    for (int c = grp; c < n_chunks; c += 2) {
      const int n = min(kC, seq.len - c * kC);
      uint8_t* sb = chunk_smem + grp * buf_bytes;
      const uint32_t sa = smem_u32(sb);
      uint32_t rv[4][NV];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = 4 * pw + j;
        const bf16* pr = proj + (static_cast<size_t>(seq.row0) + c * kC + (t < n ? t : 0)) * a.ld + a.off_v + hv;
#pragma unroll
        for (int i = 0; i < NV; ++i) rv[j][i] = ld_pair<VEC>(pr, 2 * lane + 64 * i, a.DV);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const int ch = 2 * lane + 64 * i, m = 4 * pw + j < n ? a.DK : 0;
          rk[j][i] = keep_pair(rk[j][i], ch, m);
          rq[j][i] = keep_pair(rq[j][i], ch, m);
        }
      float2 lw[4][NP];  // delta: running log decay over the warp's four tokens
      float inv[4];
      if (DELTA) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const bool in = 4 * pw + j < n;
          float ss = 0.0f;
#pragma unroll
          for (int i = 0; i < NP; ++i) {
            const float2 k = f2(rk[j][i]), wz = f2(rw[j][i]);
            ss = fmaf(k.x, k.x, fmaf(k.y, k.y, ss));
            lw[j][i] = in ? make_float2(-a.decay_coef * sigmoid_f(wz.x + wb[i].x), -a.decay_coef * sigmoid_f(wz.y + wb[i].y))
                          : make_float2(0.0f, 0.0f);
            if (j > 0) { lw[j][i].x += lw[j - 1][i].x; lw[j][i].y += lw[j - 1][i].y; }
          }
          inv[j] = ss;
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1)
#pragma unroll
          for (int j = 0; j < 4; ++j) inv[j] += __shfl_xor_sync(0xffffffffu, inv[j], o);
#pragma unroll
        for (int j = 0; j < 4; ++j) inv[j] = 1.0f / sqrtf(inv[j] + a.unit_eps);
#pragma unroll
        for (int i = 0; i < NP; ++i) *reinterpret_cast<float2*>(&sh_tot[grp][pw][DELTA ? 2 * lane + 64 * i : 0]) = lw[3][i];
      }
      if (c >= 2) buffer_sync<kBarEmpty>(grp, n_cons + kGroup);
      if (DELTA) {
        group_sync(grp);
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          const int ch = 2 * lane + 64 * i;
          float2 base = make_float2(0.0f, 0.0f);
#pragma unroll
          for (int q = 0; q < 3; ++q)
            if (q < pw) {
              const float2 o = *reinterpret_cast<const float2*>(&sh_tot[grp][q][DELTA ? ch : 0]);
              base.x += o.x; base.y += o.y;
            }
          float2 prev = make_float2(__expf(base.x), __expf(base.y));  // W_{t-1}
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float2 W = make_float2(__expf(base.x + lw[j][i].x), __expf(base.y + lw[j][i].y));
            const float2 iW = make_float2(__fdividef(1.0f, W.x), __fdividef(1.0f, W.y));
            const float2 k = f2(rk[j][i]), r = f2(rq[j][i]), az = f2(ra[j][i]);
            const float2 al = make_float2(sigmoid_f(az.x + ab[i].x), sigmoid_f(az.y + ab[i].y));
            const float2 u = make_float2(k.x * inv[j], k.y * inv[j]);
            const int off = ((4 * pw + j) * LD + ch) * 2;
            st_split(sb + L::tile(kU, 0), sb + L::tile(kU, 1), off, prev.x * u.x, prev.y * u.y);
            st_split(sb + L::tile(kR, 0), sb + L::tile(kR, 1), off, W.x * r.x, W.y * r.y);
            st_split(sb + L::tile(kKa, 0), sb + L::tile(kKa, 1), off, -al.x * u.x * iW.x, -al.y * u.y * iW.y);
            st_split(sb + L::tile(kKk, 0), sb + L::tile(kKk, 1), off, k.x * iW.x, k.y * iW.y);
            prev = W;
          }
          if (pw == 3) *reinterpret_cast<float2*>(sb + L::kScale + ch * 4) = prev;
        }
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int t = 4 * pw + j;
#pragma unroll
          for (int i = 0; i < NP; ++i) {
            const float2 qr = f2(rq[j][i]), kr = f2(rk[j][i]);
            const int off = (t * LD + 2 * lane + 64 * i) * 2;
            *reinterpret_cast<uint32_t*>(sb + L::tile(kR, 0) + off) = pack_bf16x2(silu_f(qr.x), silu_f(qr.y));
            *reinterpret_cast<uint32_t*>(sb + L::tile(kKk, 0) + off) = pack_bf16x2(silu_f(kr.x), silu_f(kr.y));
          }
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = 4 * pw + j;
        uint8_t* v_row = sb + L::kV + t * ldv * 2;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int x = 2 * lane + 64 * i;
          if (x >= dvp) continue;
          const uint32_t raw = keep_pair(rv[j][i], x, t < n ? a.DV : 0);
          if (DELTA) {
            *reinterpret_cast<uint32_t*>(v_row + 2 * x) = raw;
          } else {
            const float2 v = f2(raw);
            const uint32_t act = pack_bf16x2(silu_f(v.x), silu_f(v.y));
            const float w = t < n ? sh_pow[n - 1 - t] : 0.0f;
            *reinterpret_cast<uint32_t*>(v_row + 2 * x) = act;
            st_split(v_row + kC * ldv * 2, v_row + 2 * kC * ldv * 2, 2 * x, bf16_lo(act) * w, bf16_hi(act) * w);
          }
        }
      }
      if (c + 2 < n_chunks) fetch(c + 2);  // in flight while the matrices are built
      group_sync(grp);
      // the 16 x 16 matrices: warp 0 U Ka^T (and its inverse), 1 U Kk^T, 2 R Ka^T, 3 R Kk^T; decay: warp 3 q k^T alone
      const int g = lane >> 2, cc = lane & 3;
      if (DELTA || pw == 3) {
        float acc[2][4] = {};
        const int ta = DELTA && pw < 2 ? kU : kR, tb = DELTA && !(pw & 1) ? kKa : kKk;
        rows_product<NK, LD, DELTA>(acc, sa + L::tile(ta, 0), sa + L::tile(ta, 1), sa + L::tile(tb, 0), sa + L::tile(tb, 1), lane);
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int t = g + 8 * half, s = 8 * nb + 2 * cc;
            float x = acc[nb][2 * half], y = acc[nb][2 * half + 1];
            const int reach = DELTA && pw < 2 ? t - 1 : t;  // largest s that contributes
            if (!DELTA) {
              x *= sh_pow[s <= t ? t - s : 0];
              y *= sh_pow[s + 1 <= t ? t - s - 1 : 0];
            }
            x = s <= reach ? x : 0.0f;
            y = s + 1 <= reach ? y : 0.0f;
            if (DELTA && pw == 0) {
              sh_a1[grp][t][s] = x;
              sh_a1[grp][t][s + 1] = y;
            } else {
              const int m = DELTA ? (pw == 1 ? kA2 : (pw == 2 ? kB1 : kB2)) : kB2;
              st_split(sb + L::mat(m, 0), sb + L::mat(m, 1), (t * kMatLd + s) * 2, x, y);
            }
          }
        if (DELTA && pw == 0) {
          __syncwarp();
          // T = [T1 0; X T2] with the inverses T1, T2 of the two unit lower triangular 8 x 8 blocks (a half-warp each, a lane
          // per column, row by row) and X = T2 (A21 T1)
          const int blk = lane >> 4, col = lane & 7;
          float T[8];
#pragma unroll
          for (int t = 0; t < 8; ++t) {
            float v = t == col ? 1.0f : 0.0f, v2 = 0.0f;
#pragma unroll
            for (int s = 0; s < t; ++s) {
              const float m = sh_a1[grp][8 * blk + t][8 * blk + s];
              if (s & 1) v2 = fmaf(m, T[s], v2);
              else v = fmaf(m, T[s], v);
            }
            T[t] = v + v2;
          }
#pragma unroll
          for (int t = 0; t < 8; ++t) sh_inv[grp][8 * blk + t][8 * blk + col] = T[t];  // (two lanes, the same value)
          __syncwarp();
          const int xi = lane >> 2, xc = 2 * (lane & 3);
          float2 x = make_float2(0.0f, 0.0f);
#pragma unroll
          for (int s = 0; s < 8; ++s) {
            const float m = sh_a1[grp][8 + xi][s];
            x = make_float2(fmaf(m, sh_inv[grp][s][xc], x.x), fmaf(m, sh_inv[grp][s][xc + 1], x.y));
          }
          sh_inv[grp][8 + xi][xc] = x.x;
          sh_inv[grp][8 + xi][xc + 1] = x.y;
          __syncwarp();
          float2 y = make_float2(0.0f, 0.0f);
#pragma unroll
          for (int s = 0; s < 8; ++s) {
            const float m = sh_inv[grp][8 + xi][8 + s];
            y = make_float2(fmaf(m, sh_inv[grp][8 + s][xc], y.x), fmaf(m, sh_inv[grp][8 + s][xc + 1], y.y));
          }
          uint8_t *hi = sb + L::mat(kT, 0), *lo = sb + L::mat(kT, 1);
          st_split(hi, lo, (xi * kMatLd + xc) * 2, sh_inv[grp][xi][xc], sh_inv[grp][xi][xc + 1]);
          st_split(hi, lo, (xi * kMatLd + 8 + xc) * 2, 0.0f, 0.0f);
          st_split(hi, lo, ((8 + xi) * kMatLd + xc) * 2, y.x, y.y);
          st_split(hi, lo, ((8 + xi) * kMatLd + 8 + xc) * 2, sh_inv[grp][8 + xi][8 + xc], sh_inv[grp][8 + xi][8 + xc + 1]);
        }
      }
      buffer_arrive<kBarFull>(grp, n_cons + kGroup);
    }
    return;
  }

  // ---------------- consumers ----------------
  const int g = lane >> 2, cc = lane & 3;
  const int v0 = (threadIdx.x >> 5) * 16;
  float S[2 * NK][4];  // S^T: value columns v0 + g, v0 + g + 8; key channels 8 j + 2 cc, + 1
  float* state = a.state + (static_cast<size_t>(seq.slot) * a.H + h) * a.DK * a.DV;
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ch = 8 * j + 2 * cc + (e & 1), v = v0 + g + 8 * (e >> 1);
      S[j][e] = seq.pos > 0 && ch < a.DK && v < a.DV ? state[static_cast<size_t>(ch) * a.DV + v] : 0.0f;
    }
  const uint32_t row_b = static_cast<uint32_t>((lane & 7) + (lane >> 4) * 8), col_b = static_cast<uint32_t>((lane >> 3) & 1) * 8;
  const uint32_t bo = (row_b * LD + col_b) * 2, mo = (row_b * kMatLd + col_b) * 2;
  const uint32_t row_t = static_cast<uint32_t>((lane & 7) + ((lane >> 3) & 1) * 8);
  const uint32_t to = (row_t * LD + static_cast<uint32_t>(lane >> 4) * 8) * 2;
  const uint32_t vo = (row_b * static_cast<uint32_t>(ldv) + v0 + col_b) * 2;

  const bool in0 = v0 + g < a.DV, in1 = v0 + g + 8 < a.DV;
  const int ldo = static_cast<int>(a.ldo);
  float* orow = a.o + (static_cast<size_t>(seq.row0) + 2 * cc) * a.ldo + h * a.DV + v0 + g;

  for (int c = 0; c < n_chunks; ++c) {
    const int buf = c & 1, n = min(kC, seq.len - c * kC);
    const uint32_t sa = smem_u32(chunk_smem) + buf * buf_bytes;
    const float* scale = reinterpret_cast<const float*>(chunk_smem + buf * buf_bytes + L::kScale);
    buffer_sync<kBarFull>(buf, n_cons + kGroup);
    float O[2][4] = {}, P[2][4] = {}, O2[2][4] = {}, P2[2][4] = {};
#pragma unroll
    for (int k = 0; k < NK; ++k) {
      uint32_t sh[4], sl[4], bh[4], bl[4];
      split_frag(S[2 * k], S[2 * k + 1], sh, sl);
      if (DELTA) {
        ldsm_x4(bh, sa + L::tile(kU, 0) + bo + k * 32);
        ldsm_x4(bl, sa + L::tile(kU, 1) + bo + k * 32);
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
          mma_bf16_16816(P[nb], sh[0], sh[1], sh[2], sh[3], bh[2 * nb], bh[2 * nb + 1]);
          mma_bf16_16816(P2[nb], sh[0], sh[1], sh[2], sh[3], bl[2 * nb], bl[2 * nb + 1]);
          mma_bf16_16816(P2[nb], sl[0], sl[1], sl[2], sl[3], bh[2 * nb], bh[2 * nb + 1]);
        }
      }
      ldsm_x4(bh, sa + L::tile(kR, 0) + bo + k * 32);
      if (DELTA) ldsm_x4(bl, sa + L::tile(kR, 1) + bo + k * 32);
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) {
        mma_bf16_16816(O[nb], sh[0], sh[1], sh[2], sh[3], bh[2 * nb], bh[2 * nb + 1]);
        if (DELTA) mma_bf16_16816(O2[nb], sh[0], sh[1], sh[2], sh[3], bl[2 * nb], bl[2 * nb + 1]);
        mma_bf16_16816(O2[nb], sl[0], sl[1], sl[2], sl[3], bh[2 * nb], bh[2 * nb + 1]);
      }
    }
    if (!DELTA) {  // the state's decay up to token t = 8 nb + 2 cc + (e & 1)
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float d = sh_pow[8 * nb + 2 * cc + (e & 1) + 1];
          O[nb][e] *= d;
          O2[nb][e] *= d;
        }
    }
    uint32_t vh[4], vl[4] = {};
    ldsm_x4_trans(vh, sa + L::kV + vo);
    uint32_t ph[4], pl[4];
    if (DELTA) {
      frag_mat(P, vh, vl, false, sa + L::mat(kA2, 0), sa + L::mat(kA2, 1), mo);
#pragma unroll
      for (int nb = 0; nb < 2; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) P[nb][e] += P2[nb][e];
      split_frag(P[0], P[1], ph, pl);
      float Q[2][4] = {};
      frag_mat(Q, ph, pl, true, sa + L::mat(kT, 0), sa + L::mat(kT, 1), mo);
      split_frag(Q[0], Q[1], ph, pl);
      frag_mat(O, ph, pl, true, sa + L::mat(kB1, 0), sa + L::mat(kB1, 1), mo);
    }
    frag_mat(O2, vh, vl, false, sa + L::mat(kB2, 0), sa + L::mat(kB2, 1), mo);
    if (!DELTA) {  // from here on the values that enter the state: d^{n-1-s} v_s
      ldsm_x4_trans(vh, sa + L::kV + kC * ldv * 2 + vo);
      ldsm_x4_trans(vl, sa + L::kV + 2 * kC * ldv * 2 + vo);
    }
    // ---- output: token 8 nb + 2 cc + (e & 1), value column v0 + g + 8 (e >> 1) ----
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = 8 * nb + (e & 1);
        if (t + 2 * cc < n && ((e >> 1) ? in1 : in0)) orow[t * ldo + 8 * (e >> 1)] = O[nb][e] + O2[nb][e];
      }
    orow += kC * ldo;
    // ---- state ----
    const float dn = DELTA ? 1.0f : sh_pow[n];
#pragma unroll
    for (int j = 0; j < 2 * NK; j += 2) {
      uint32_t kh[4], kl[4];
      if (DELTA) {
        ldsm_x4_trans(kh, sa + L::tile(kKa, 0) + to + j * 16);
        ldsm_x4_trans(kl, sa + L::tile(kKa, 1) + to + j * 16);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma_bf16_16816(S[j + e], ph[0], ph[1], ph[2], ph[3], kh[2 * e], kh[2 * e + 1]);
          mma_bf16_16816(S[j + e], ph[0], ph[1], ph[2], ph[3], kl[2 * e], kl[2 * e + 1]);
          mma_bf16_16816(S[j + e], pl[0], pl[1], pl[2], pl[3], kh[2 * e], kh[2 * e + 1]);
        }
      } else {
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int f = 0; f < 4; ++f) S[j + e][f] *= dn;
      }
      ldsm_x4_trans(kh, sa + L::tile(kKk, 0) + to + j * 16);
      if (DELTA) ldsm_x4_trans(kl, sa + L::tile(kKk, 1) + to + j * 16);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mma_bf16_16816(S[j + e], vh[0], vh[1], vh[2], vh[3], kh[2 * e], kh[2 * e + 1]);
        if (DELTA) mma_bf16_16816(S[j + e], vh[0], vh[1], vh[2], vh[3], kl[2 * e], kl[2 * e + 1]);
        else mma_bf16_16816(S[j + e], vl[0], vl[1], vl[2], vl[3], kh[2 * e], kh[2 * e + 1]);
      }
      if (DELTA) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 w = *reinterpret_cast<const float2*>(scale + 8 * (j + e) + 2 * cc);
          S[j + e][0] *= w.x; S[j + e][1] *= w.y; S[j + e][2] *= w.x; S[j + e][3] *= w.y;
        }
      }
    }
    if (c + 2 < n_chunks) buffer_arrive<kBarEmpty>(buf, n_cons + kGroup);
  }
  pdl_trigger();
#pragma unroll
  for (int j = 0; j < 2 * NK; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int ch = 8 * j + 2 * cc + (e & 1), v = v0 + g + 8 * (e >> 1);
      if (ch < a.DK && v < a.DV) state[static_cast<size_t>(ch) * a.DV + v] = S[j][e];
    }
}

template <int MODE, int NK, int NV, bool VEC, int THREADS, int BLOCKS>
int launch_chunk(const StateScan& a, const SeqDesc* seqs, int n_seqs, int dvp, bool prepare_only, cudaStream_t st) {
  static std::atomic<unsigned long long> done{0};  // one bit per device; threads may race to set it
  int dev = 0;
  cudaGetDevice(&dev);
  const auto kernel = chunk_scan_kernel<MODE, NK, NV, VEC, THREADS, BLOCKS>;
  if (!(dev < 64 && (done.load(std::memory_order_acquire) >> dev) & 1ull)) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 2 * Lay<16 * NK>::bytes(64 * NV));
    if (e != cudaSuccess) return static_cast<int>(e);
    if (dev < 64) done.fetch_or(1ull << dev, std::memory_order_release);
  }
  if (prepare_only) return 0;
  launch_kernel(kernel, dim3(a.H, n_seqs), dim3(dvp * 2 + kProducers), 2 * Lay<16 * NK>::bytes(dvp), st, 1, a, seqs, dvp);
  return static_cast<int>(cudaGetLastError());
}

// Registers: a thread of the 64-channel kernel gets 80 with up to 64 value columns (two CTAs per SM), 96 above; of the
// 128-channel kernel 128 with up to 128 value columns, 96 above.
template <int MODE>
int dispatch_chunk(const StateScan& a, const SeqDesc* seqs, int n_seqs, bool prep, cudaStream_t st) {
  const bool vec = ((a.DK | a.DV | a.off_q | a.off_k | a.off_v) & 1) == 0 && (a.ld & 1) == 0 &&
                   (a.mode != kScanDelta || ((a.off_a & 1) == 0 && (a.ld_wz & 1) == 0));
  const int dvp = (a.DV + 15) / 16 * 16;
#define TEENY_CHUNK(NK, NV, T, B)                                                          \
  return vec ? launch_chunk<MODE, NK, NV, true, T, B>(a, seqs, n_seqs, dvp, prep, st)      \
             : launch_chunk<MODE, NK, NV, false, T, B>(a, seqs, n_seqs, dvp, prep, st)
  if (a.DK <= 64) {
    if (dvp <= 64) TEENY_CHUNK(4, 1, 384, 2);
    TEENY_CHUNK(4, 3, 640, 1);
  }
  if (dvp <= 128) TEENY_CHUNK(8, 2, 512, 1);
  TEENY_CHUNK(8, 3, 640, 1);
#undef TEENY_CHUNK
}

}  // namespace

bool chunk_scan_supports(const StateScan& a, int max_len) {
  // 1 / W_t must stay far from overflow within a chunk
  return !a.f32 && max_len >= kC && a.DK <= 128 && a.DV <= kMaxDV && (a.mode != kScanDelta || a.decay_coef * kC <= 40.0f);
}

int chunk_scan_prepare() {
  for (int odd = 0; odd < 2; ++odd)
    for (int dk : {64, 128})
      for (int dv : {64, 128, 192}) {
        StateScan a{};
        a.DK = dk; a.DV = dv; a.off_k = odd;
        int rc = dispatch_chunk<kScanDelta>(a, nullptr, 0, true, nullptr);
        if (!rc) rc = dispatch_chunk<kScanDecay>(a, nullptr, 0, true, nullptr);
        if (rc) return rc;
      }
  return 0;
}

int chunk_scan(const StateScan& a, const SeqDesc* seqs, int n_seqs, cudaStream_t st) {
  return a.mode == kScanDelta ? dispatch_chunk<kScanDelta>(a, seqs, n_seqs, false, st) : dispatch_chunk<kScanDecay>(a, seqs, n_seqs, false, st);
}

}  // namespace teeny
