// Latent attention: keys and values of all heads come from one small latent vector per token (plus one rotated key part that
// the heads share), so that is all the cache holds.  Two ways to attend:
//   expanded   per-head keys and values are made from the latents by one GEMM (hybrid_runner.cu) and go through the ordinary
//              attention kernels: long portions of prompts.
//   absorbed   the queries are taken into the latent space instead (head_linear with the key projection), attend over the
//              cached rows as ONE key / value head shared by all query heads, and the result is taken back out (head_linear
//              with the value projection): single tokens and short portions, where the cache is what has to be read.
// Kernels here
//   latent_prepare_kernel<T>          norms of the query latent and the latent, rotation of the shared key part, cache append
//   head_linear_mma_kernel<MT>        the small per-head products, bf16 (mma.sync; weights fetched ahead of the dependency wait)
//   head_linear_rows_kernel<T>        the same, anything
//   latent_attention_mma_kernel       absorbed attention, bf16 (mma.sync tiles over cp.async stages; the key range is split over
//                                     a cluster whose CTAs merge through distributed shared memory)
//   latent_attention_rows_kernel<T>   the same, anything: eight warps per (token, head)
#include <atomic>
#include <type_traits>

#include "common.cuh"
#include "kernels.h"
#include "mma.cuh"

namespace teeny {

namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

// eight consecutive elements, 16-byte aligned
__device__ __forceinline__ void ld8(const bf16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
  v[4] = bf16_lo(u.z); v[5] = bf16_hi(u.z); v[6] = bf16_lo(u.w); v[7] = bf16_hi(u.w);
}
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void st8(bf16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}
__device__ __forceinline__ void st8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

__host__ __device__ inline int pad8(int n) { return (n + 7) & ~7; }

constexpr int kPrepThreads = 128, kPrepVecs = 4;

// One CTA per (token, entry).  Columns between a part's size and the next multiple of 8 are zero in `proj` (zero weight rows)
// and stay zero.
template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prepare_kernel(const LatentPrepare a, const SeqDesc* __restrict__ seqs) {
  __shared__ float red[2][kPrepThreads / 32];
  const SeqDesc seq = seqs[blockIdx.y];  // written well before the kernel in front of this one
  const int i = blockIdx.x;
  pdl_wait();
  pdl_trigger();
  if (i >= seq.len) return;
  const size_t row = static_cast<size_t>(seq.row0) + i;
  const int pos = seq.pos + i, KR = pad8(a.rank), DL = KR + a.RD;
  const T* src = static_cast<const T*>(a.proj) + row * a.ld;
  const int nq = pad8(a.q_rank) / 8, nc = KR / 8;
  // the first vectors of both parts stay in registers; longer parts are read again (from L1)
  float v[kPrepVecs][8], sq = 0.0f, sc = 0.0f;
  auto part = [&](int x) { return x < nq ? src + a.off_q + 8 * x : src + a.off_c + 8 * (x - nq); };
#pragma unroll
  for (int t = 0; t < kPrepVecs; ++t) {
    const int x = threadIdx.x + t * kPrepThreads;
    if (x < nq + nc) {
      ld8(part(x), v[t]);
      float s = 0.0f;
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(v[t][e], v[t][e], s);
      (x < nq ? sq : sc) += s;
    }
  }
  for (int x = threadIdx.x + kPrepVecs * kPrepThreads; x < nq + nc; x += kPrepThreads) {
    float w[8], s = 0.0f;
    ld8(part(x), w);
#pragma unroll
    for (int e = 0; e < 8; ++e) s = fmaf(w[e], w[e], s);
    (x < nq ? sq : sc) += s;
  }
  T* lat = a.rows ? static_cast<T*>(a.rows) + row * DL : nullptr;
  T* cache = static_cast<T*>(a.cache) + (static_cast<size_t>(seq.slot) * a.max_len + pos) * DL;
  const int half = a.RD >> 1;
  for (int d = threadIdx.x; d < half; d += kPrepThreads) {
    float sn, cs;
    sincosf(static_cast<float>(pos) * a.inv_freq[d], &sn, &cs);
    sn *= a.rot_scale;
    cs *= a.rot_scale;
    const float x = ldf(src + a.off_r + d), y = ldf(src + a.off_r + d + half);
    const float p = x * cs - y * sn, q = y * cs + x * sn;
    stf(cache + KR + d, p);
    stf(cache + KR + half + d, q);
    if (lat) {
      stf(lat + KR + d, p);
      stf(lat + KR + half + d, q);
    }
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = sq;
    red[1][threadIdx.x >> 5] = sc;
  }
  __syncthreads();
  sq = sc = 0.0f;
#pragma unroll
  for (int w = 0; w < kPrepThreads / 32; ++w) {
    sq += red[0][w];
    sc += red[1][w];
  }
  const float rq = 1.0f / sqrtf(sq / static_cast<float>(a.q_rank) + a.eps), rc = 1.0f / sqrtf(sc / static_cast<float>(a.rank) + a.eps);
  auto emit = [&](int x, float (&w)[8]) {
    float g[8];
    const bool is_q = x < nq;
    ld8(is_q ? a.q_w + 8 * x : a.c_w + 8 * (x - nq), g);
    const float rr = is_q ? rq : rc;
#pragma unroll
    for (int e = 0; e < 8; ++e) w[e] = w[e] * rr * g[e];
    if (is_q) {
      st8(static_cast<T*>(a.cq) + row * a.ldcq + 8 * x, w);
    } else {
      st8(cache + 8 * (x - nq), w);
      if (lat) st8(lat + 8 * (x - nq), w);
    }
  };
#pragma unroll
  for (int t = 0; t < kPrepVecs; ++t) {
    const int x = threadIdx.x + t * kPrepThreads;
    if (x < nq + nc) emit(x, v[t]);
  }
  for (int x = threadIdx.x + kPrepVecs * kPrepThreads; x < nq + nc; x += kPrepThreads) {
    float w[8];
    ld8(part(x), w);
    emit(x, w);
  }
}

// ---------------------------------------------------------------------------------------------- per-head products
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void zero16(uint32_t dst) { asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};" ::"r"(dst), "r"(0u) : "memory"); }

// Rotated elements of head h of rows r0 .. r0 + n - 1 behind the product's columns; any block size.
template <typename T>
__device__ __forceinline__ void rotate_tail(const HeadLinear& a, int h, int r0, int n) {
  const int half = a.RD >> 1;
  const int base = a.seqs[0].row0;  // of row 0 of x and y
  for (int idx = threadIdx.x; idx < n * half; idx += blockDim.x) {
    const int r = r0 + idx / half, d = idx % half;
    int pos = 0;
    for (int s = 0; s < a.n_seqs; ++s) {
      const SeqDesc q = a.seqs[s];
      const int i = r + base - q.row0;
      if (i >= 0 && i < q.len) {
        pos = q.pos + i;
        break;
      }
    }
    float sn, cs;
    sincosf(static_cast<float>(pos) * a.inv_freq[d], &sn, &cs);
    sn *= a.rot_scale;
    cs *= a.rot_scale;
    const T* src = static_cast<const T*>(a.x) + r * a.ldx + h * a.x_head + a.rot_off;
    T* dst = static_cast<T*>(a.y) + r * a.ldy + h * a.y_head + a.N;
    const float x = ldf(src + d), y = ldf(src + d + half);
    stf(dst + d, x * cs - y * sn);
    stf(dst + d + half, y * cs + x * sn);
  }
}

// CTA = 32 output columns of one head for 16 MT rows.  MT = 1: the four warps split K and are summed through shared memory;
// MT = 4: each warp 16 rows.  The weights (no kernel writes them) are requested before the dependency wait.
constexpr int kHlCols = 32;
constexpr int hl_smem_bytes(int mt, int K) { return (kHlCols + 16 * mt) * ((K + 15) / 16 * 16 + 8) * 2; }

template <int MT>
__global__ void __launch_bounds__(128) head_linear_mma_kernel(const HeadLinear a) {
  extern __shared__ __align__(16) bf16 hl_smem[];
  const int KP = (a.K + 15) / 16 * 16, LD = KP + 8, CH = KP / 8;
  const int n0 = blockIdx.x * kHlCols, h = blockIdx.y, r0 = blockIdx.z * 16 * MT;
  const int rows = min(16 * MT, a.T - r0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  if (n0 >= a.N) {
    pdl_wait();
    pdl_trigger();
    rotate_tail<bf16>(a, h, r0, rows);
    return;
  }
  const uint32_t sw = smem_u32(hl_smem), sx = sw + kHlCols * LD * 2;
  const bf16* w = static_cast<const bf16*>(a.w) + (static_cast<size_t>(h) * a.N + n0) * a.K;
  for (int idx = threadIdx.x; idx < kHlCols * CH; idx += 128) {
    const int r = idx / CH, ch = idx % CH;
    const uint32_t dst = sw + static_cast<uint32_t>(r * LD + ch * 8) * 2;
    if (n0 + r < a.N && ch * 8 < a.K) cp_async16(dst, w + static_cast<size_t>(r) * a.K + ch * 8);
    else zero16(dst);
  }
  pdl_wait();
  const bf16* x = static_cast<const bf16*>(a.x) + static_cast<size_t>(r0) * a.ldx + h * a.x_head;
  for (int idx = threadIdx.x; idx < 16 * MT * CH; idx += 128) {
    const int r = idx / CH, ch = idx % CH;
    const uint32_t dst = sx + static_cast<uint32_t>(r * LD + ch * 8) * 2;
    if (r < rows && ch * 8 < a.K) cp_async16(dst, x + r * a.ldx + ch * 8);
    else zero16(dst);
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();
  pdl_trigger();
  float acc[4][4];
#pragma unroll
  for (int n = 0; n < 4; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.0f;
  const int row_x = (MT == 1 ? 0 : warp * 16) + (lane & 7) + ((lane >> 3) & 1) * 8;
  const uint32_t xa = sx + static_cast<uint32_t>(row_x * LD + (lane >> 4) * 8) * 2;
  const uint32_t wa = sw + static_cast<uint32_t>(((lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8) * 2;
  for (int k = MT == 1 ? warp : 0; k < KP / 16; k += MT == 1 ? 4 : 1) {
    uint32_t xf[4];
    ldsm_x4(xf, xa + k * 32);
#pragma unroll
    for (int n = 0; n < 4; n += 2) {
      uint32_t wf[4];
      ldsm_x4(wf, wa + static_cast<uint32_t>(n * 8 * LD) * 2 + k * 32);
      mma_bf16_16816(acc[n], xf[0], xf[1], xf[2], xf[3], wf[0], wf[1]);
      mma_bf16_16816(acc[n + 1], xf[0], xf[1], xf[2], xf[3], wf[2], wf[3]);
    }
  }
  bf16* y = static_cast<bf16*>(a.y) + static_cast<size_t>(r0) * a.ldy + h * a.y_head + n0;
  if constexpr (MT > 1) {
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = warp * 16 + g + 8 * e, d = 8 * n + 2 * c;
        if (r < rows && n0 + d < a.N) *reinterpret_cast<uint32_t*>(y + r * a.ldy + d) = pack_bf16x2(acc[n][2 * e], acc[n][2 * e + 1]);
      }
  } else {
    __shared__ float sum[4][16][kHlCols];
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) sum[warp][g + 8 * (e >> 1)][8 * n + 2 * c + (e & 1)] = acc[n][e];
    __syncthreads();
    for (int idx = threadIdx.x; idx < 16 * kHlCols / 2; idx += 128) {
      const int r = idx / (kHlCols / 2), d = idx % (kHlCols / 2) * 2;
      if (r >= rows || n0 + d >= a.N) continue;
      float v[2] = {0.0f, 0.0f};
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        v[0] += sum[q][r][d];
        v[1] += sum[q][r][d + 1];
      }
      *reinterpret_cast<uint32_t*>(y + r * a.ldy + d) = pack_bf16x2(v[0], v[1]);
    }
  }
}

template <typename T>
__global__ void head_linear_rows_kernel(const HeadLinear a) {
  pdl_wait();
  const int h = blockIdx.y, r = blockIdx.z;
  const int n = blockIdx.x * blockDim.x + threadIdx.x;
  if (a.RD > 0 && blockIdx.x == 0) rotate_tail<T>(a, h, r, 1);
  if (n >= a.N) return;
  const T* x = static_cast<const T*>(a.x) + r * a.ldx + h * a.x_head;
  const T* w = static_cast<const T*>(a.w) + (static_cast<size_t>(h) * a.N + n) * a.K;
  float s = 0.0f;
  for (int k = 0; k < a.K; ++k) s = fmaf(ldf(x + k), ldf(w + k), s);
  stf(static_cast<T*>(a.y) + r * a.ldy + h * a.y_head + n, s);
}

// ---------------------------------------------------------------------------------------------- absorbed attention
constexpr int kLatMax = 1024;  // largest cache row of the generic kernel

template <typename T>
__global__ void __launch_bounds__(256) latent_attention_rows_kernel(const LatentAttn a, const SeqDesc* __restrict__ seqs) {
  constexpr int NE = kLatMax / 32;
  __shared__ float sm_ml[8][2];
  __shared__ float sm_o[8][kLatMax];
  pdl_wait();
  pdl_trigger();
  const SeqDesc seq = seqs[blockIdx.y];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int i = blockIdx.x / a.H, h = blockIdx.x % a.H;
  if (i >= seq.len) return;
  const size_t row = static_cast<size_t>(seq.row0) + i;
  const T* qr = static_cast<const T*>(a.q) + row * a.ldq + h * a.D;
  const T* kr = static_cast<const T*>(a.cache) + static_cast<size_t>(seq.slot) * a.max_len * a.D;
  float qv[NE], acc[NE];
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const int d = lane + 32 * e;
    qv[e] = d < a.D ? ldf(qr + d) * a.scale : 0.0f;
    acc[e] = 0.0f;
  }
  float m = -INFINITY, l = 0.0f;
  for (int j = warp; j <= seq.pos + i; j += 8) {
    const T* kp = kr + static_cast<size_t>(j) * a.D;
    float dot = 0.0f;
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int d = lane + 32 * e;
      if (d < a.D) dot = fmaf(qv[e], ldf(kp + d), dot);
    }
    dot = warp_sum(dot);
    const float m_new = fmaxf(m, dot);
    const float corr = expf(m - m_new), p = expf(dot - m_new);
    l = fmaf(corr, l, p);
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int d = lane + 32 * e;
      if (d < a.DV) acc[e] = fmaf(corr, acc[e], p * ldf(kp + d));
    }
    m = m_new;
  }
  if (lane == 0) {
    sm_ml[warp][0] = m;
    sm_ml[warp][1] = l;
  }
#pragma unroll
  for (int e = 0; e < NE; ++e) sm_o[warp][lane + 32 * e] = acc[e];
  __syncthreads();
  float mm = -INFINITY;
#pragma unroll
  for (int w = 0; w < 8; ++w) mm = fmaxf(mm, sm_ml[w][0]);
  T* orow = static_cast<T*>(a.out) + row * a.ldo + h * a.DV;
  for (int d = threadIdx.x; d < a.DV; d += 256) {
    float o = 0.0f, ll = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {  // warps without keys hold -inf: factor 0
      const float sc = expf(sm_ml[w][0] - mm);
      ll = fmaf(sm_ml[w][1], sc, ll);
      o = fmaf(sm_o[w][d], sc, o);
    }
    stf(orow + d, o / ll);
  }
}

// CTA = 16 MT consecutive (token, head) rows of one entry x one share of the keys; the CTAs of a cluster hold the shares of
// one row tile.  Keys come in tiles of 64 cache rows through two cp.async stages.  Eight warps; per tile
//   scores   warp (kq, kh) multiplies a quarter of the row's dimensions (its queries stay in registers for the whole walk) for
//            32 of the keys; the four partial sums meet in shared memory, where each row belongs to 256 / rows threads that
//            keep its running maximum and sum and write the weights as bf16;
//   values   warp w owns 16 NV columns of the value and multiplies the weights with them, the same cache rows transposed on
//            the way out of shared memory.
// At the end the shares are scaled to the cluster's maximum and summed through distributed shared memory, every CTA a slice
// of the columns.  Columns between D and 64 NK are zero in shared memory.
constexpr int kLatKeys = 64;
constexpr int lat_ld(int nk) { return 64 * nk + 8; }
constexpr int kLatSLd = kLatKeys + 2, kLatPLd = kLatKeys + 8;
constexpr int lat_smem_bytes(int mt, int nk) {
  return 2 * kLatKeys * lat_ld(nk) * 2 + 4 * 16 * mt * kLatSLd * 4 + 16 * mt * kLatPLd * 2 + 3 * 16 * mt * 4;
}

__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float ld_cluster(uint32_t local_addr, uint32_t rank) {
  uint32_t r;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(r) : "memory");
  return v;
}
__device__ __forceinline__ float2 ld_cluster2(uint32_t local_addr, uint32_t rank) {
  uint32_t r;
  float2 v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(r) : "memory");
  return v;
}

template <int MT, int NK, int NV>
__global__ void __launch_bounds__(256) latent_attention_mma_kernel(const LatentAttn a, const SeqDesc* __restrict__ seqs) {
  constexpr int R = 16 * MT, LD = lat_ld(NK), CH = 8 * NK, TPR = 256 / R, KPT = kLatKeys / TPR;  // threads per row, keys per thread
  extern __shared__ __align__(16) uint8_t lat_smem[];
  bf16* stage0 = reinterpret_cast<bf16*>(lat_smem);
  float* sp = reinterpret_cast<float*>(lat_smem + 2 * kLatKeys * LD * 2);   // [4][R][kLatSLd] partial scores
  bf16* pb = reinterpret_cast<bf16*>(sp + 4 * R * kLatSLd);                 // [R][kLatPLd] weights
  float* row_f = reinterpret_cast<float*>(pb + R * kLatPLd);                // [3][R]: rescale factor of the tile; final maximum, sum
  const SeqDesc seq = seqs[blockIdx.z];  // written well before the kernel in front of this one
  const int row0 = blockIdx.y * R, n_rows = min(R, seq.len * a.H - row0);
  if (n_rows <= 0) {                     // the whole cluster
    pdl_wait();
    return;
  }
  const int splits = gridDim.x, split = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  const int L = seq.pos + (row0 + n_rows - 1) / a.H + 1;  // keys the tile's last row sees
  const int span = ((L + splits - 1) / splits + kLatKeys - 1) / kLatKeys * kLatKeys;
  const int key0 = split * span, key_end = min(L, key0 + span);
  const int n_tiles = key0 < key_end ? (key_end - key0 + kLatKeys - 1) / kLatKeys : 0;
  const bf16* cache = static_cast<const bf16*>(a.cache) + static_cast<size_t>(seq.slot) * a.max_len * a.D;
  const uint32_t st_a = smem_u32(stage0);

  for (int idx = threadIdx.x; idx < 2 * kLatKeys * (CH - a.D / 8); idx += 256) {  // columns that no copy fills
    const int r = idx / (CH - a.D / 8), ch = a.D / 8 + idx % (CH - a.D / 8);
    zero16(st_a + static_cast<uint32_t>(r * LD + ch * 8) * 2);
  }
  pdl_wait();
  auto load_tile = [&](int t) {
    const uint32_t dst0 = st_a + static_cast<uint32_t>((t & 1) * kLatKeys * LD) * 2;
    const int n = a.D / 8;
    for (int idx = threadIdx.x; idx < kLatKeys * n; idx += 256) {
      const int r = idx / n, ch = idx - r * n, j = key0 + t * kLatKeys + r;
      const uint32_t dst = dst0 + static_cast<uint32_t>(r * LD + ch * 8) * 2;
      if (j < key_end) cp_async16(dst, cache + static_cast<size_t>(j) * a.D + ch * 8);
      else zero16(dst);
    }
    cp_async_commit();
  };
  if (n_tiles > 0) load_tile(0);

  // query fragments of this warp's quarter of the dimensions
  const int kq = warp & 3, kh = warp >> 2;
  uint32_t qf[MT][NK][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = row0 + mt * 16 + g + 8 * e, tok = r / a.H, h = r - tok * a.H;
      const bool in = r < row0 + n_rows;
      const bf16* q = static_cast<const bf16*>(a.q) + (static_cast<size_t>(seq.row0) + (in ? tok : 0)) * a.ldq + (in ? h : 0) * a.D;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        const int d = (kq * NK + k) * 16 + 2 * c;
        qf[mt][k][e] = in && d < a.D ? *reinterpret_cast<const uint32_t*>(q + d) : 0u;
        qf[mt][k][2 + e] = in && d + 8 < a.D ? *reinterpret_cast<const uint32_t*>(q + d + 8) : 0u;
      }
    }
  float O[MT][2 * NV][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int n = 0; n < 2 * NV; ++n) O[mt][n][0] = O[mt][n][1] = O[mt][n][2] = O[mt][n][3] = 0.0f;
  // softmax: thread = (row sr, keys KPT * sub ..)
  const int sr = threadIdx.x / TPR, sub = threadIdx.x % TPR;
  const int s_pos = seq.pos + min(row0 + sr, row0 + n_rows - 1) / a.H;  // last key this row sees
  float m = -INFINITY, l = 0.0f;
  const float sc = a.scale * 1.4426950408889634f;
  const int v0 = warp * 16 * NV;  // value columns of this warp
  for (int t = 0; t < n_tiles; ++t) {
    if (t + 1 < n_tiles) {
      load_tile(t + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t kt = st_a + static_cast<uint32_t>((t & 1) * kLatKeys * LD) * 2;
    {
      float s[MT][4][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < 4; ++n) s[mt][n][0] = s[mt][n][1] = s[mt][n][2] = s[mt][n][3] = 0.0f;
      const uint32_t ka = kt + static_cast<uint32_t>((kh * 32 + (lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8 + kq * NK * 16) * 2;
#pragma unroll
      for (int k = 0; k < NK; ++k)
#pragma unroll
        for (int n = 0; n < 4; n += 2) {
          uint32_t b[4];
          ldsm_x4(b, ka + static_cast<uint32_t>(n * 8 * LD) * 2 + k * 32);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_bf16_16816(s[mt][n], qf[mt][k][0], qf[mt][k][1], qf[mt][k][2], qf[mt][k][3], b[0], b[1]);
            mma_bf16_16816(s[mt][n + 1], qf[mt][k][0], qf[mt][k][1], qf[mt][k][2], qf[mt][k][3], b[2], b[3]);
          }
        }
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int e = 0; e < 2; ++e)
            *reinterpret_cast<float2*>(sp + (kq * R + mt * 16 + g + 8 * e) * kLatSLd + kh * 32 + 8 * n + 2 * c) =
                make_float2(s[mt][n][2 * e], s[mt][n][2 * e + 1]);
    }
    __syncthreads();
    {
      float x[KPT], mx = m;
      const int j0 = key0 + t * kLatKeys + sub * KPT;
#pragma unroll
      for (int e = 0; e < KPT; e += 2) {
        float2 v = make_float2(0.0f, 0.0f);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float2 p = *reinterpret_cast<const float2*>(sp + (q * R + sr) * kLatSLd + sub * KPT + e);
          v.x += p.x;
          v.y += p.y;
        }
        x[e] = j0 + e <= s_pos && j0 + e < key_end ? v.x * sc : -INFINITY;
        x[e + 1] = j0 + e + 1 <= s_pos && j0 + e + 1 < key_end ? v.y * sc : -INFINITY;
        mx = fmaxf(mx, fmaxf(x[e], x[e + 1]));
      }
#pragma unroll
      for (int o = TPR >> 1; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float base = mx == -INFINITY ? 0.0f : mx;  // a row that has seen no key yet
      const float alpha = ex2(m - base);
      m = mx;
      l *= alpha;
#pragma unroll
      for (int e = 0; e < KPT; e += 2) {
        const float p0 = ex2(x[e] - base), p1 = ex2(x[e + 1] - base);
        l += p0 + p1;
        *reinterpret_cast<uint32_t*>(pb + sr * kLatPLd + sub * KPT + e) = pack_bf16x2(p0, p1);
      }
      if (sub == 0) row_f[sr] = alpha;
    }
    __syncthreads();
    if (v0 < a.DV) {
      float al[MT][2];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        al[mt][0] = row_f[mt * 16 + g];
        al[mt][1] = row_f[mt * 16 + g + 8];
#pragma unroll
        for (int n = 0; n < 2 * NV; ++n) {
          O[mt][n][0] *= al[mt][0]; O[mt][n][1] *= al[mt][0];
          O[mt][n][2] *= al[mt][1]; O[mt][n][3] *= al[mt][1];
        }
      }
      const uint32_t pa = smem_u32(pb) + static_cast<uint32_t>(((lane & 7) + ((lane >> 3) & 1) * 8) * kLatPLd + (lane >> 4) * 8) * 2;
      const uint32_t va = kt + static_cast<uint32_t>(((lane & 7) + ((lane >> 3) & 1) * 8) * LD + (lane >> 4) * 8 + v0) * 2;
#pragma unroll
      for (int k = 0; k < kLatKeys / 16; ++k) {
        uint32_t pf[MT][4];
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) ldsm_x4(pf[mt], pa + static_cast<uint32_t>(mt * 16 * kLatPLd + k * 16) * 2);
#pragma unroll
        for (int n = 0; n < NV; ++n) {
          uint32_t b[4];
          ldsm_x4_trans(b, va + static_cast<uint32_t>(k * 16 * LD + n * 16) * 2);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_bf16_16816(O[mt][2 * n], pf[mt][0], pf[mt][1], pf[mt][2], pf[mt][3], b[0], b[1]);
            mma_bf16_16816(O[mt][2 * n + 1], pf[mt][0], pf[mt][1], pf[mt][2], pf[mt][3], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();  // the stage, the scores and the weights may be written again
  }
  pdl_trigger();
  // ---- merge ----
#pragma unroll
  for (int o = TPR >> 1; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  if (sub == 0) {
    row_f[R + sr] = m;
    row_f[2 * R + sr] = l;
  }
  float* ob = reinterpret_cast<float*>(lat_smem);  // [R][16 NV * 8] this share's output, over the stages
  constexpr int OLD = 128 * NV + 2;
  static_assert(R * OLD * 4 <= 2 * kLatKeys * LD * 2, "the output fits into the stages");
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int n = 0; n < 2 * NV; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e)
        *reinterpret_cast<float2*>(ob + (mt * 16 + g + 8 * e) * OLD + v0 + 8 * n + 2 * c) = make_float2(O[mt][n][2 * e], O[mt][n][2 * e + 1]);
  if (splits > 1) cluster_sync();
  else __syncthreads();
  // this CTA's share of the columns, in pairs
  const int pairs = a.DV / 2, per = (pairs + splits - 1) / splits, p0 = split * per, p1 = min(pairs, p0 + per);
  const uint32_t ob_a = smem_u32(ob), rf_a = smem_u32(row_f);
  for (int r = warp; r < n_rows; r += 8) {
    float w = 0.0f, mm = -INFINITY;  // lane s: weight of share s (at most 32 shares)
    if (splits > 1) {
      const float ms = lane < splits ? ld_cluster(rf_a + (R + r) * 4, lane) : -INFINITY;
      const float ls = lane < splits ? ld_cluster(rf_a + (2 * R + r) * 4, lane) : 0.0f;
      mm = warp_max(ms);
      w = ex2(ms - mm);  // shares without keys hold -inf: 0
      w /= warp_sum(w * ls);
    } else {
      w = 1.0f / row_f[2 * R + r];
    }
    const int rr = row0 + r, tok = rr / a.H, h = rr - tok * a.H;
    bf16* orow = static_cast<bf16*>(a.out) + (static_cast<size_t>(seq.row0) + tok) * a.ldo + h * a.DV;
    for (int pp = p0; pp < p1; pp += 32) {  // (whole warps: shuffles)
      const int p = pp + lane;
      float2 o = make_float2(0.0f, 0.0f);
      for (int s = 0; s < splits; ++s) {
        const float ws = __shfl_sync(0xffffffffu, w, s);
        if (p >= p1) continue;
        const float2 v = splits > 1 ? ld_cluster2(ob_a + (r * OLD + 2 * p) * 4, s) : *reinterpret_cast<const float2*>(ob + r * OLD + 2 * p);
        o.x = fmaf(ws, v.x, o.x);
        o.y = fmaf(ws, v.y, o.y);
      }
      if (p < p1) *reinterpret_cast<uint32_t*>(orow + 2 * p) = pack_bf16x2(o.x, o.y);
    }
  }
  if (splits > 1) cluster_sync();  // no CTA leaves while others read its shared memory
}

// Size classes of the mma kernel: cache rows up to 64 NK elements (each a quarter of 16 NK), values up to 128 NV.
template <typename F>
int for_class(int d, int dv, F&& f) {
  if (d <= 192 && dv <= 128) return f(std::integral_constant<int, 3>(), std::integral_constant<int, 1>());
  if (d <= 320 && dv <= 256) return f(std::integral_constant<int, 5>(), std::integral_constant<int, 2>());
  if (d <= 576 && dv <= 512) return f(std::integral_constant<int, 9>(), std::integral_constant<int, 4>());
  return TEENY_ERR_BAD_ARG;
}

}  // namespace

int latent_prepare(const LatentPrepare& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  if (!a.proj || !a.q_w || !a.c_w || !a.cq || !a.cache || !seqs || n_seqs <= 0 || n_seqs > 65535 || max_len <= 0 || a.q_rank <= 0 ||
      a.rank <= 0 || a.RD < 0 || a.RD % 8 || (a.RD && !a.inv_freq) || a.max_len <= 0)
    return TEENY_ERR_BAD_ARG;
  const uintptr_t bases = reinterpret_cast<uintptr_t>(a.proj) | reinterpret_cast<uintptr_t>(a.cq) | reinterpret_cast<uintptr_t>(a.rows) |
                          reinterpret_cast<uintptr_t>(a.cache) | reinterpret_cast<uintptr_t>(a.q_w) | reinterpret_cast<uintptr_t>(a.c_w);
  if ((bases & 15) || ((a.ld | a.ldcq | a.off_q | a.off_c) & 7)) return TEENY_ERR_ALIGNMENT;
  const dim3 grid(max_len, n_seqs), block(kPrepThreads);
  if (a.f32) launch_kernel(latent_prepare_kernel<float>, grid, block, 0, st, 1, a, seqs);
  else launch_kernel(latent_prepare_kernel<bf16>, grid, block, 0, st, 1, a, seqs);
  return static_cast<int>(cudaGetLastError());
}

int head_linear(const HeadLinear& a, cudaStream_t st) {
  if (!a.x || !a.w || !a.y || a.H <= 0 || a.H > 65535 || a.N <= 0 || a.K <= 0 || a.T <= 0 || a.N % 8 || a.K % 8 || a.RD < 0 || a.RD % 2 ||
      (a.RD && (!a.inv_freq || !a.seqs || a.n_seqs <= 0)))
    return TEENY_ERR_BAD_ARG;
  {
    const int rc = latent_attention_prepare();
    if (rc) return rc;
  }
  const uintptr_t bases = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.w);
  const bool vec = !a.f32 && (bases & 15) == 0 && ((a.ldx | a.x_head) & 7) == 0 && (reinterpret_cast<uintptr_t>(a.y) & 3) == 0 &&
                   ((a.ldy | a.y_head) & 1) == 0 && a.K <= kLatMax;
  if (vec) {
    const int tail = a.RD > 0 ? 1 : 0;
    const int mt = a.T <= 16 ? 1 : 4, tiles = (a.T + 16 * mt - 1) / (16 * mt);
    if (tiles > 65535) return TEENY_ERR_BAD_ARG;
    const dim3 grid((a.N + kHlCols - 1) / kHlCols + tail, a.H, tiles);
    if (mt == 1) launch_kernel(head_linear_mma_kernel<1>, grid, dim3(128), hl_smem_bytes(1, a.K), st, 1, a);
    else launch_kernel(head_linear_mma_kernel<4>, grid, dim3(128), hl_smem_bytes(4, a.K), st, 1, a);
    return static_cast<int>(cudaGetLastError());
  }
  if (a.T > 65535) return TEENY_ERR_BAD_ARG;
  const dim3 grid((a.N + 127) / 128, a.H, a.T);
  if (a.f32) launch_kernel(head_linear_rows_kernel<float>, grid, dim3(128), 0, st, 1, a);
  else launch_kernel(head_linear_rows_kernel<bf16>, grid, dim3(128), 0, st, 1, a);
  return static_cast<int>(cudaGetLastError());
}

int latent_attention_prepare() {
  static std::atomic<unsigned long long> done{0};  // one bit per device; threads may race to set it
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 64 && (done.load(std::memory_order_acquire) >> dev) & 1ull) return 0;
  cudaError_t e = cudaFuncSetAttribute(head_linear_mma_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, hl_smem_bytes(1, kLatMax));
  if (e == cudaSuccess) e = cudaFuncSetAttribute(head_linear_mma_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, hl_smem_bytes(4, kLatMax));
  const int sizes[][2] = {{192, 128}, {320, 256}, {576, 512}};
  for (const auto& s : sizes)
    for_class(s[0], s[1], [&](auto nk, auto nv) {
      constexpr int NK = decltype(nk)::value, NV = decltype(nv)::value;
      if (e == cudaSuccess)
        e = cudaFuncSetAttribute(latent_attention_mma_kernel<1, NK, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, lat_smem_bytes(1, NK));
      if (e == cudaSuccess)
        e = cudaFuncSetAttribute(latent_attention_mma_kernel<2, NK, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, lat_smem_bytes(2, NK));
      return 0;
    });
  if (e != cudaSuccess) return static_cast<int>(e);
  if (dev < 64) done.fetch_or(1ull << dev, std::memory_order_release);
  return 0;
}

int latent_attention(const LatentAttn& a, const SeqDesc* seqs, int n_seqs, int longest, cudaStream_t st) {
  if (!a.q || !a.cache || !a.out || !seqs || n_seqs <= 0 || n_seqs > 65535 || longest <= 0 || a.H <= 0 || a.D <= 0 || a.D > kLatMax ||
      a.DV <= 0 || a.DV > a.D || a.max_len <= 0 || static_cast<long long>(longest) * a.H > 0x7fffffffLL)
    return TEENY_ERR_BAD_ARG;
  {
    const int rc = latent_attention_prepare();
    if (rc) return rc;
  }
  const uintptr_t bases = reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.cache) | reinterpret_cast<uintptr_t>(a.out);
  const bool vec = !a.f32 && a.D % 8 == 0 && a.DV % 8 == 0 && ((a.ldq | a.ldo) & 7) == 0 && (bases & 15) == 0;
  const int rows = longest * a.H, mt = rows <= 16 ? 1 : 2, tiles = (rows + 16 * mt - 1) / (16 * mt);
  if (vec && tiles <= 65535) {
    // shares of the keys: as many as still leave every SM at most about one CTA
    int splits = 1;
    const long long ctas = static_cast<long long>(tiles) * n_seqs;
    while (splits < 8 && ctas * splits * 2 <= sm_count() && splits * 2 * kLatKeys <= a.max_len) splits *= 2;
    const dim3 grid(splits, tiles, n_seqs);
    const int rc = for_class(a.D, a.DV, [&](auto nk, auto nv) {
      constexpr int NK = decltype(nk)::value, NV = decltype(nv)::value;
      if (mt == 1)
        launch_kernel(latent_attention_mma_kernel<1, NK, NV>, grid, dim3(256), lat_smem_bytes(1, NK), st, static_cast<unsigned>(splits), a, seqs);
      else
        launch_kernel(latent_attention_mma_kernel<2, NK, NV>, grid, dim3(256), lat_smem_bytes(2, NK), st, static_cast<unsigned>(splits), a, seqs);
      return static_cast<int>(cudaGetLastError());
    });
    if (rc != TEENY_ERR_BAD_ARG) return rc;
  }
  const dim3 grid(static_cast<unsigned>(rows), n_seqs);
  if (a.f32) launch_kernel(latent_attention_rows_kernel<float>, grid, dim3(256), 0, st, 1, a, seqs);
  else launch_kernel(latent_attention_rows_kernel<bf16>, grid, dim3(256), 0, st, 1, a, seqs);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace teeny
