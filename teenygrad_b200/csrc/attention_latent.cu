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
//   latent_attention_kernel<N>        absorbed attention, bf16 (tcgen05; the key range is split over CTAs), and
//   latent_merge_kernel               the sum over the shares of a split key range
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
    int e = min(r, a.n_seqs - 1);  // entries lie in row order, each with at least one row
    SeqDesc q = a.seqs[e];
    while (q.row0 - base > r) q = a.seqs[--e];
    const int pos = q.pos + r + base - q.row0;
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
  const size_t row = static_cast<size_t>(seq.row0) - a.row_base + i;
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

// Absorbed attention on the tensor cores (tcgen05).  CTA = N consecutive (token, head) rows of one entry x one share of its keys.
// The rows are the N side of both products (a few query heads waste
// nothing), and the cache rows, loaded once per 64-key tile, are the A operand of both.  M = 128 holds 64 keys twice: a slot of
// shared memory is 128 dimensions of the tile as two boxes [64 keys][64 d], one behind the other, which the two products read as
//   S^T [2 x 64 keys, 2 N] += [boxes] [Q of the first box's dimensions; Q of the second's]^T     (K-major)
//            the upper half of the lanes means something in the first N columns, the lower half in the others: their sum is S^T
//   O^T [128 values, N]    += [boxes]^T P^T                                                    (the same memory MN-major)
// so that two tiles are in shared memory at a time and no product is idle in half of its rows.
// Tensor memory: O^T in blocks of N columns per 128 values, two S^T buffers of 2 N columns.
//   warp 4   TMA producer: ring of 16 KB slots.  A slot is free again when its last product has completed (with P; for dimensions
//            behind the values with Q), so the loads follow the products slot by slot.  Starts before the dependency wait: only
//            the queries come from the kernel in front of this one.
//   warp 5   allocates tensor memory, loads the queries, issues the MMAs (one thread); S of tile t + 1 goes ahead of P V of tile t
//            where the ring holds two tiles.
//   warps 0-3  thread = tensor-memory lane: its lane's N partial scores, half of which it trades with the thread of the same key in
//            the other half (shared memory), so that each ends with N / 2 scores of its key; mask, weights against the rows'
//            running maxima (shared memory), sums in registers, weights as bf16 into shared memory ([row][key], the B operand).
//            The maxima only move when some score exceeds its row's by more than 2^8 (one vote per tile); then the tile's maxima
//            are reduced across the lanes and O^T is rescaled.
// At the end O^T over its row sums goes out as bf16 rows, one bulk store of N whole rows: to the output, or where the keys are
// split to a partial result beside its maxima and sums, which latent_merge_kernel weighs and adds.  (Shares of a cluster meeting in
// distributed shared memory were slower: the exchange of 64 KB per CTA took 5000 cycles, half as bf16, and clusters leave a
// third of the SMs idle.)
constexpr int kLatTile = 64, kLatSlot = 16384, kLatBox = 8192, kLatMaxSlots = 24, kLatThreads = 192;
constexpr float kLatGrow = 8.0f;  // log2 units

struct LatTcArgs {
  bf16* out;           // [rows, DV]
  bf16* part_o;        // split keys: [CTA][N][DV] and ...
  float2* part_ml;     // ... [CTA][N] maximum (log2 domain) and sum
  int row_base;        // step row that row 0 of q and out stands for
  int H, D, DV;
  int blocks;          // 128-dimension slots of a tile that hold values
  int tile_slots;      // slots of a tile
  int slots, ahead;    // of the ring; whether it holds two tiles
  uint32_t tmem_cols;
  float scale_log2;
  int* err;
};

struct LatSmem {  // byte offsets
  int q, p, swap, bars, stats, total;
};
__host__ __device__ inline LatSmem lat_smem(int n, int tile_slots, int slots) {
  LatSmem s;
  s.q = slots * kLatSlot;               // [boxes][n rows][64 d]
  s.p = s.q + 2 * tile_slots * n * 128; // [n rows][64 keys]
  s.swap = s.p + n * 128;               // partial scores between the lane halves: [n / 4][64 keys] float4
  s.bars = s.swap + n * 64 * 4;
  s.stats = s.bars + 8 * (2 * kLatMaxSlots + 8);
  s.total = s.stats + 4 * 8 * n + 1024;
  return s;
}

// `bytes` of this CTA's shared memory to global memory, by one thread, which then waits until they have been read.
__device__ __forceinline__ void bulk_store(void* dst, uint32_t src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(src), "r"(bytes) : "memory");
  asm volatile("cp.async.bulk.commit_group;\n\tcp.async.bulk.wait_group.read 0;" ::: "memory");
}
// whether `v` holds in any of the 128 softmax threads (barrier 1)
__device__ __forceinline__ bool any128(bool v) {
  uint32_t r;
  asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.u32 q, %1, 0;\n\tbar.red.or.pred p, 1, 128, q;\n\tselp.u32 %0, 1, 0, p;\n\t}"
               : "=r"(r) : "r"(static_cast<uint32_t>(v)) : "memory");
  return r != 0;
}
// N consecutive tensor-memory columns of this warp's lanes
template <int N>
__device__ __forceinline__ void tmem_ld_cols(uint32_t addr, float (&v)[N]) {
  if constexpr (N == 16) {
    uint32_t t[16];
    tmem_ld_32x16(addr, t);
    tmem_wait_ld();
#pragma unroll
    for (int e = 0; e < 16; ++e) v[e] = __uint_as_float(t[e]);
  } else {
    uint32_t t[N / 32][32];
#pragma unroll
    for (int i = 0; i < N / 32; ++i) tmem_ld_32x32(addr + 32 * i, t[i]);
    tmem_wait_ld();
#pragma unroll
    for (int i = 0; i < N / 32; ++i)
#pragma unroll
      for (int e = 0; e < 32; ++e) v[32 * i + e] = __uint_as_float(t[i][e]);
  }
}
// Two such blocks, side by side.
template <int N>
__device__ __forceinline__ void tmem_ld_cols2(uint32_t addr, float (&v)[2][N]) {
  if constexpr (N == 32) {
    uint32_t t[2][32];
    tmem_ld_32x32(addr, t[0]);
    tmem_ld_32x32(addr + 32, t[1]);
    tmem_wait_ld();
#pragma unroll
    for (int e = 0; e < 32; ++e) {
      v[0][e] = __uint_as_float(t[0][e]);
      v[1][e] = __uint_as_float(t[1][e]);
    }
  } else {
    tmem_ld_cols<N>(addr, v[0]);
    tmem_ld_cols<N>(addr + N, v[1]);
  }
}
template <int N>
__device__ __forceinline__ void tmem_st_cols(uint32_t addr, const float (&v)[N]) {
  if constexpr (N == 16) {
    uint32_t t[16];
#pragma unroll
    for (int e = 0; e < 16; ++e) t[e] = __float_as_uint(v[e]);
    tmem_st_32x16(addr, t);
  } else {
#pragma unroll
    for (int i = 0; i < N / 32; ++i) {
      uint32_t t[32];
#pragma unroll
      for (int e = 0; e < 32; ++e) t[e] = __float_as_uint(v[32 * i + e]);
      tmem_st_32x32(addr + 32 * i, t);
    }
  }
}
// Reduction of W columns (8, 16 or 32) over the warp's lanes, halving the columns a lane holds at every step; lane i ends with
// column i % W.
template <int W, bool MAX>
__device__ __forceinline__ float reduce_columns(float (&v)[W]) {
  const int lane = threadIdx.x & 31;
  auto op = [](float a, float b) { return MAX ? fmaxf(a, b) : a + b; };
#pragma unroll
  for (int w = 16; w >= W; w >>= 1)
#pragma unroll
    for (int i = 0; i < W; ++i) v[i] = op(v[i], __shfl_xor_sync(0xffffffffu, v[i], w));
#pragma unroll
  for (int w = W / 2; w > 0; w >>= 1)
#pragma unroll
    for (int i = 0; i < w; ++i) {
      const bool hi = (lane & w) != 0;
      const float keep = hi ? v[i + w] : v[i], send = hi ? v[i] : v[i + w];
      v[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, w));
    }
  return v[0];
}
// ... into dst[W] of this warp
template <int W, bool MAX>
__device__ __forceinline__ void reduce_to(const float (&v)[W], float* dst) {
  float t[W];
#pragma unroll
  for (int e = 0; e < W; ++e) t[e] = v[e];
  const float r = reduce_columns<W, MAX>(t);
  if ((threadIdx.x & 31) < W) dst[threadIdx.x & 31] = r;
}

// Whether the barrier's phase of this parity is complete, for the whole warp; does not wait.
__device__ __forceinline__ bool mbar_test_wait(uint32_t bar, uint32_t parity) {
  uint32_t done;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(done) : "r"(bar), "r"(parity) : "memory");
  return __all_sync(0xffffffffu, done != 0);
}
// Four K-steps of a product as straight-line code, the operands' addresses A_STEP and B_STEP (16-byte units) further at each.  The
// whole warp comes here and the one lane with `lead` issues: in uniform control flow descriptors and counters stay in uniform
// registers (a lone lane in a divergent branch issues a product only every ~100 cycles).
template <int A_STEP, int B_STEP>
__device__ __forceinline__ void umma_x4(uint32_t lead, uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate_first) {
  asm volatile(
      "{\n\t.reg .pred e, p, t;\n\t.reg .b64 x, y;\n\t"
      "setp.ne.b32 e, %5, 0;\n\t setp.ne.b32 p, %4, 0;\n\t setp.eq.b32 t, %3, %3;\n\t"
      "@e tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t"
      "add.u64 x, %1, %6;\n\t add.u64 y, %2, %9;\n\t @e tcgen05.mma.cta_group::1.kind::f16 [%0], x, y, %3, t;\n\t"
      "add.u64 x, %1, %7;\n\t add.u64 y, %2, %10;\n\t @e tcgen05.mma.cta_group::1.kind::f16 [%0], x, y, %3, t;\n\t"
      "add.u64 x, %1, %8;\n\t add.u64 y, %2, %11;\n\t @e tcgen05.mma.cta_group::1.kind::f16 [%0], x, y, %3, t;\n\t}"
      ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate_first), "r"(lead), "n"(A_STEP), "n"(2 * A_STEP), "n"(3 * A_STEP), "n"(B_STEP),
        "n"(2 * B_STEP), "n"(3 * B_STEP)
      : "memory");
}
// 128 dimensions of a tile into a slot: two boxes [64 keys][64 d].
__device__ __forceinline__ void load_slot(uint32_t lead, uint32_t dst, const CUtensorMap* m, uint32_t bar, int d, int key, int seq) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t.reg .b32 x, y;\n\t setp.ne.b32 e, %6, 0;\n\t add.u32 x, %0, %8;\n\t add.u32 y, %3, 64;\n\t"
      "@e mbarrier.arrive.expect_tx.shared::cta.b64 _, [%2], %7;\n\t"
      "@e cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];\n\t"
      "@e cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [x], [%1, {y, %4, %5}], [%2];\n\t}"
      ::"r"(dst), "l"(reinterpret_cast<uint64_t>(m)), "r"(bar), "r"(d), "r"(key), "r"(seq), "r"(lead), "n"(kLatSlot), "n"(kLatBox)
      : "memory");
}
__device__ __forceinline__ void load_queries(uint32_t lead, uint32_t dst, const CUtensorMap* m, uint32_t bar, int d, int row) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t setp.ne.b32 e, %5, 0;\n\t"
      "@e cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];\n\t}"
      ::"r"(dst), "l"(reinterpret_cast<uint64_t>(m)), "r"(bar), "r"(d), "r"(row), "r"(lead)
      : "memory");
}
__device__ __forceinline__ void umma_commit_lead(uint32_t lead, uint32_t bar) {
  asm volatile(
      "{\n\t.reg .pred e;\n\t setp.ne.b32 e, %1, 0;\n\t"
      "@e tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}"
      ::"r"(bar), "r"(lead)
      : "memory");
}

template <int N>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_attention_kernel(const __grid_constant__ CUtensorMap tmap_c, const __grid_constant__ CUtensorMap tmap_q, const LatTcArgs a,
                        const SeqDesc* __restrict__ seqs) {
  constexpr int HN = N / 2;  // rows whose weights a thread works out
  extern __shared__ uint8_t lat_raw[];
  const SeqDesc seq = seqs[blockIdx.z];  // written well before the kernel in front of this one
  const int row0 = blockIdx.y * N, n_rows = min(N, seq.len * a.H - row0);
  if (n_rows <= 0) {
    pdl_wait();
    return;
  }
  const uint32_t base = (smem_u32(lat_raw) + 1023u) & ~1023u;
  uint8_t* gen = lat_raw + (base - smem_u32(lat_raw));
  const LatSmem lay = lat_smem(N, a.tile_slots, a.slots);
  const uint32_t bar0 = base + lay.bars;
  auto full = [&](int i) { return bar0 + 8u * i; };
  auto empty = [&](int i) { return bar0 + 8u * (kLatMaxSlots + i); };
  const uint32_t misc = bar0 + 8u * 2 * kLatMaxSlots;
  const uint32_t q_full = misc, s_full = misc + 8, p_ready = misc + 24, pv_done = misc + 32, tmem_slot = misc + 40;  // two s_full
  float* m_sh = reinterpret_cast<float*>(gen + lay.stats);  // [N] running maxima, log2 domain
  float* alpha_sh = m_sh + N;                               // [N] factor of the last rescale; finally 1 / the row sums
  float* up_sh = alpha_sh + N;                              // [N] by how much the maxima just rose
  float* red = up_sh + N;                                   // [4][HN] of each warp
  int* lim = reinterpret_cast<int*>(red + 4 * N);           // [N] last key each row sees

  const int split = blockIdx.x, splits = gridDim.x;
  const int warp = threadIdx.x >> 5;
  const int L = seq.pos + (row0 + n_rows - 1) / a.H + 1;  // keys the tile's last row sees
  const int span = ((L + splits - 1) / splits + kLatTile - 1) / kLatTile * kLatTile;
  const int key0 = split * span, key_end = min(L, key0 + span);
  const int n_tiles = key0 < key_end ? (key_end - key0 + kLatTile - 1) / kLatTile : 0;

  if (threadIdx.x == 128) {
    tma_prefetch_desc(&tmap_c);
    tma_prefetch_desc(&tmap_q);
    for (int i = 0; i < a.slots; ++i) {
      mbar_init(full(i), 1);
      mbar_init(empty(i), 1);
    }
    mbar_init(q_full, 1);
    mbar_init(s_full, 1);
    mbar_init(s_full + 8, 1);
    mbar_init(p_ready, 128);
    mbar_init(pv_done, 1);
    mbar_fence_init();
  }
  if (warp == 5) {
    tmem_alloc(tmem_slot, a.tmem_cols);
    tmem_relinquish();
  }
  if (threadIdx.x < N) {
    lim[threadIdx.x] = seq.pos + min(row0 + static_cast<int>(threadIdx.x), row0 + n_rows - 1) / a.H;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(gen + lay.bars + 8 * 2 * kLatMaxSlots + 40);
  const uint32_t t_s = tmem + a.blocks * N;
  bool ok = true;

  if (warp == 4) {
    // ---------------- producer ----------------
    const uint32_t lead = elect_one() ? 1u : 0u;
    bool waited = false;
    int slot = 0, key = key0;
    uint32_t round = 0;
    for (int t = 0; ok && t < n_tiles; ++t, key += kLatTile)
      for (int p = 0; ok && p < a.tile_slots; ++p) {
        if (round > 0) {
          if (!waited) {  // the ring is full: the queries' kernel has to be done by now anyway
            pdl_wait();
            waited = true;
          }
          ok = mbar_wait(empty(slot), (round & 1) ^ 1, a.err, DEVERR_ATTN_PRODUCER);
          __syncwarp();
        }
        if (ok) load_slot(lead, base + slot * kLatSlot, &tmap_c, full(slot), 128 * p, key, seq.slot);
        if (++slot == a.slots) {
          slot = 0;
          ++round;
        }
      }
    if (!waited) pdl_wait();
    __syncwarp();
  } else if (warp == 5) {
    // ---------------- MMA issuer ----------------
    pdl_wait();
    if (n_tiles > 0) {
      const uint32_t lead = elect_one() ? 1u : 0u;
      if (lead) mbar_expect_tx(q_full, 2 * a.tile_slots * N * 128);
      __syncwarp();
      const int q_row = (seq.row0 - a.row_base) * a.H + row0;
      for (int b = 0; b < 2 * a.tile_slots; ++b) load_queries(lead, base + lay.q + b * N * 128, &tmap_q, q_full, 64 * b, q_row);
      constexpr uint32_t idesc_s = make_idesc_bf16(128, 2 * N, false, false), idesc_pv = make_idesc_bf16(128, N, true, false);
      const uint64_t q_desc = make_smem_desc_sw128(base + lay.q, 16, 1024), p_desc = make_smem_desc_sw128(base + lay.p, 16, 1024);
      // cache rows: K-major for the scores; MN-major (64 values contiguous per key, 8 keys 1 KB apart, the next 64 values a box on) for O
      const uint64_t c_desc = make_smem_desc_sw128(base, 16, 1024), v_desc = make_smem_desc_sw128(base, kLatBox, 1024);
      ok = mbar_wait(q_full, 0, a.err, DEVERR_ATTN_MMA);
      // Whichever product can go next: a slot of S as soon as it is loaded (S of a tile at most one ahead of P V, whose weights
      // show that its buffer has been read; not ahead at all in a ring of less than two tiles), else P V as soon as its weights are
      // there.
      int s_tile = 0, s_part = 0, s_slot = 0, v_tile = 0, v_slot = 0;
      uint32_t s_round = 0, spins = 0;
      uint64_t t0 = 0;
      while (ok && v_tile < n_tiles) {
        if (s_tile < n_tiles && s_tile <= v_tile + (a.ahead ? 1 : 0) && mbar_test_wait(full(s_slot), s_round & 1)) {
          tc_fence_after();
          // (32 bytes along the rows per step; dimensions beyond D are zero on both sides)
          umma_x4<2, 2>(lead, t_s + (s_tile & 1) * 2 * N, c_desc + static_cast<uint64_t>(s_slot * (kLatSlot >> 4)),
                        q_desc + static_cast<uint64_t>(s_part * 2 * N * 8), idesc_s, s_part > 0 ? 1u : 0u);
          if (s_part >= a.blocks) umma_commit_lead(lead, empty(s_slot));
          if (++s_part == a.tile_slots) {
            umma_commit_lead(lead, s_full + 8 * (s_tile & 1));
            s_part = 0;
            ++s_tile;
          }
          if (++s_slot == a.slots) {
            s_slot = 0;
            ++s_round;
          }
          spins = 0;
        } else if (mbar_test_wait(p_ready, v_tile & 1)) {
          tc_fence_after();
          for (int i = 0; i < a.tile_slots; ++i) {
            if (i < a.blocks) {  // 16 keys = 2 KB per step
              umma_x4<128, 2>(lead, tmem + i * N, v_desc + static_cast<uint64_t>(v_slot * (kLatSlot >> 4)), p_desc, idesc_pv, v_tile > 0 ? 1u : 0u);
              umma_commit_lead(lead, empty(v_slot));
            }
            if (++v_slot == a.slots) v_slot = 0;
          }
          umma_commit_lead(lead, pv_done);
          ++v_tile;
          spins = 0;
        } else if ((++spins & 0xff) == 0) {  // (the limits of mbar_wait)
          const uint64_t now = global_timer_ns();
          if (spins == 0x100) t0 = now;
          else if (*reinterpret_cast<volatile int*>(a.err) != 0) ok = false;
          else if (now - t0 > kWaitLimitNs) {
            atomicCAS(a.err, 0, static_cast<int>(DEVERR_ATTN_MMA));
            ok = false;
          }
        }
        ok = __all_sync(0xffffffffu, ok);
      }
    }
    __syncwarp();
  } else {
    // ---------------- softmax: thread = tensor-memory lane = (half, key of the tile) ----------------
    pdl_wait();
    const int r = threadIdx.x, key = r & 63, half = r >> 6;
    const int n0 = half * HN;  // first of the rows whose weights this thread works out
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    float4* swap = reinterpret_cast<float4*>(gen + lay.swap);
    const int min_lim = lim[0];  // rows are in token order
    float l[HN];
#pragma unroll
    for (int n = 0; n < HN; ++n) l[n] = 0.0f;
    uint8_t* pw = gen + lay.p + (key & 7) * 2 + n0 * 128;  // this key's column of the weights
    const int pc = key >> 3;
    for (int t = 0; t < n_tiles; ++t) {
      const int k0 = key0 + t * kLatTile, j = k0 + key;
      if (ok) ok = mbar_wait(s_full + 8 * (t & 1), (t >> 1) & 1, a.err, DEVERR_ATTN_SOFTMAX);
      __syncwarp();
      tc_fence_after();
      float s[HN];
      {
        float x[N];
        tmem_ld_cols<N>(t_s + lane_addr + (t & 1) * 2 * N + half * N, x);
        tc_fence_before();
        // the other half's rows to the thread of the same key there; mine from it (everyone's reads are behind the vote below)
#pragma unroll
        for (int n = 0; n < HN; n += 4) {
          const int give = half ? n : HN + n;
          swap[give / 4 * 64 + key] = half ? make_float4(x[n], x[n + 1], x[n + 2], x[n + 3])
                                           : make_float4(x[HN + n], x[HN + n + 1], x[HN + n + 2], x[HN + n + 3]);
        }
#pragma unroll
        for (int n = 0; n < HN; ++n) s[n] = half ? x[HN + n] : x[n];
      }
      named_barrier_sync(1, 128);
#pragma unroll
      for (int n = 0; n < HN; n += 4) {
        const float4 o = swap[(n0 + n) / 4 * 64 + key];
        s[n] += o.x;
        s[n + 1] += o.y;
        s[n + 2] += o.z;
        s[n + 3] += o.w;
      }
      if (k0 + kLatTile > key_end || k0 + kLatTile - 1 > min_lim) {
        const bool live = j < key_end;
#pragma unroll
        for (int n = 0; n < HN; ++n) s[n] = live && j <= lim[n0 + n] ? s[n] : -INFINITY;
        if (k0 + kLatTile > key_end && !live)
          // rows past the live length hold whatever the cache had; their weights are zero, but 0 * NaN is NaN inside the product
          for (int i = 0; i < a.blocks; ++i) {  // (in the last tile only)
            uint8_t* row = gen + ((t * a.tile_slots + i) % a.slots) * kLatSlot + half * kLatBox + key * 128;
#pragma unroll
            for (int c = 0; c < 8; ++c) *reinterpret_cast<uint4*>(row + ((c ^ (key & 7)) << 4)) = make_uint4(0, 0, 0, 0);
          }
      }
      if (t == 0) {
        // a first maximum: the score of the share's first key (a row that does not see it sees none); finite
        if (key == 0) {
#pragma unroll
          for (int n = 0; n < HN; ++n) m_sh[n0 + n] = fmaxf(s[n] * a.scale_log2, -1e30f);
        }
        named_barrier_sync(1, 128);
      }
      // scores relative to the running maxima
      bool grow = false;
#pragma unroll
      for (int n = 0; n < HN; n += 4) {
        const float4 m4 = *reinterpret_cast<const float4*>(m_sh + n0 + n);
        s[n] = fmaf(s[n], a.scale_log2, -m4.x);
        s[n + 1] = fmaf(s[n + 1], a.scale_log2, -m4.y);
        s[n + 2] = fmaf(s[n + 2], a.scale_log2, -m4.z);
        s[n + 3] = fmaf(s[n + 3], a.scale_log2, -m4.w);
        grow = grow || fmaxf(fmaxf(s[n], s[n + 1]), fmaxf(s[n + 2], s[n + 3])) > kLatGrow;
      }
      if (any128(grow)) {
        reduce_to<HN, true>(s, red + warp * HN);
        named_barrier_sync(1, 128);
        if (r < N) {
          const float* mine = red + (r / HN) * 2 * HN + r % HN;
          const float up = fmaxf(fmaxf(mine[0], mine[HN]), 0.0f);
          m_sh[r] += up;
          up_sh[r] = up;
          alpha_sh[r] = ex2(-up);
        }
        named_barrier_sync(1, 128);
        if (t > 0) {
          if (ok) ok = mbar_wait(pv_done, (t - 1) & 1, a.err, DEVERR_ATTN_SOFTMAX);  // O^T is final for the tiles before
          __syncwarp();
          tc_fence_after();
          for (int i = 0; i < a.blocks; ++i) {
            float o[N];
            tmem_ld_cols<N>(tmem + lane_addr + i * N, o);
#pragma unroll
            for (int n = 0; n < N; ++n) o[n] *= alpha_sh[n];
            tmem_st_cols<N>(tmem + lane_addr + i * N, o);
          }
          tmem_wait_st();
          tc_fence_before();
        }
#pragma unroll
        for (int n = 0; n < HN; ++n) {
          l[n] *= alpha_sh[n0 + n];
          s[n] -= up_sh[n0 + n];
        }
      }
      uint32_t pk[HN / 2];
#pragma unroll
      for (int n = 0; n < HN; n += 2) {
        const float p0 = ex2(s[n]), p1 = ex2(s[n + 1]);
        l[n] += p0;
        l[n + 1] += p1;
        pk[n / 2] = pack_bf16x2(p0, p1);
      }
      if (t > 0) {
        if (ok) ok = mbar_wait(pv_done, (t - 1) & 1, a.err, DEVERR_ATTN_SOFTMAX);  // the weights of the tile before have been read
      }
#pragma unroll
      for (int n = 0; n < HN; ++n)  // (n0 is a multiple of 8: row n0 + n has n's swizzle)
        *reinterpret_cast<uint16_t*>(pw + n * 128 + ((pc ^ (n & 7)) << 4)) = static_cast<uint16_t>(n & 1 ? pk[n / 2] >> 16 : pk[n / 2] & 0xffffu);
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(p_ready);
    }
    // ---- row sums, then O^T as rows over the slots ----
    reduce_to<HN, false>(l, red + warp * HN);
    named_barrier_sync(1, 128);
    if (r < N) {
      const float* part = red + (r / HN) * 2 * HN + r % HN;
      const float sum = part[0] + part[HN];
      alpha_sh[r] = sum > 0.0f ? 1.0f / sum : 0.0f;  // (no key of this share is visible to the row)
      if (splits > 1) {
        const size_t cta = (static_cast<size_t>(blockIdx.z) * gridDim.y + blockIdx.y) * splits + split;
        a.part_ml[cta * N + r] = make_float2(sum > 0.0f ? m_sh[r] : -INFINITY, sum);
      }
    }
    if (n_tiles > 0 && ok) ok = mbar_wait(pv_done, (n_tiles - 1) & 1, a.err, DEVERR_ATTN_SOFTMAX);
    __syncwarp();
    tc_fence_after();
    named_barrier_sync(1, 128);
    if (n_tiles > 0) {
      float w[N];
#pragma unroll
      for (int n = 0; n < N; n += 4) {
        const float4 w4 = *reinterpret_cast<const float4*>(alpha_sh + n);
        w[n] = w4.x; w[n + 1] = w4.y; w[n + 2] = w4.z; w[n + 3] = w4.w;
      }
      auto stage = [&](int i, const float (&o)[N]) {
        if (i * 128 + r < a.DV) {
          bf16* dst = reinterpret_cast<bf16*>(gen) + i * 128 + r;
#pragma unroll
          for (int n = 0; n < N; ++n) dst[n * a.DV] = __float2bfloat16_rn(o[n] * w[n]);
        }
      };
      int i = 0;
      for (; i + 2 <= a.blocks; i += 2) {  // two loads in flight
        float o[2][N];
        tmem_ld_cols2<N>(tmem + lane_addr + i * N, o);
        stage(i, o[0]);
        stage(i + 1, o[1]);
      }
      if (i < a.blocks) {
        float o[N];
        tmem_ld_cols<N>(tmem + lane_addr + i * N, o);
        stage(i, o);
      }
      fence_proxy_async_smem();
    }
    tc_fence_before();
  }
  pdl_trigger();
  __syncthreads();
  if (threadIdx.x == 0 && n_tiles > 0) {  // (a share without keys has weight zero: its rows are never read)
    bf16* dst = splits > 1 ? a.part_o + ((static_cast<size_t>(blockIdx.z) * gridDim.y + blockIdx.y) * splits + split) * N * a.DV
                           : a.out + ((static_cast<long long>(seq.row0) - a.row_base) * a.H + row0) * a.DV;
    bulk_store(dst, base, n_rows * a.DV * 2);
  }
  if (warp == 5) {
    if (*reinterpret_cast<volatile int*>(a.err) != 0) {  // a wait was given up: let copies and products in flight finish
      const uint64_t t0 = global_timer_ns();
      while (global_timer_ns() - t0 < 2000000ull) __nanosleep(1000);
    }
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, a.tmem_cols);
  }
}

// CTA = one row: thread = (eight columns, every `groups`-th share), so that a thread's few loads are all in flight together.
constexpr int kLatMaxSplits = 32;
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatTcArgs a, const SeqDesc* __restrict__ seqs, int N, int tiles, int splits) {
  __shared__ float weight[kLatMaxSplits];
  __shared__ float sum[128][9];
  const SeqDesc seq = seqs[blockIdx.y];
  const int row = blockIdx.x;
  pdl_wait();
  pdl_trigger();
  if (row >= seq.len * a.H) return;
  const int tile = row / N, r = row - tile * N;
  const size_t cta = (static_cast<size_t>(blockIdx.y) * tiles + tile) * splits;
  const int chunks = a.DV / 8, groups = 128 / chunks, chunk = threadIdx.x % chunks, group = threadIdx.x / chunks;  // (DV <= 1024)
  // the rows are on their way while the weights are worked out
  constexpr int kAhead = 8;
  const bf16* src = a.part_o + (cta * N + r) * a.DV + 8 * chunk;
  uint4 v[kAhead];
#pragma unroll
  for (int i = 0; i < kAhead; ++i)
    if (group < groups && group + i * groups < splits) v[i] = *reinterpret_cast<const uint4*>(src + static_cast<size_t>(group + i * groups) * N * a.DV);
  if (threadIdx.x < 32) {
    const int s = threadIdx.x;
    const float2 ml = s < splits ? a.part_ml[(cta + s) * N + r] : make_float2(-INFINITY, 0.0f);
    const float w = ml.y * ex2(ml.x - warp_max(ml.x));  // shares without a visible key: 0
    weight[s] = w / warp_sum(w);
  }
  __syncthreads();
  float o[8] = {};
  auto add = [&](int s, uint4 x) {
    const float w = weight[s];
    if (w > 0.0f) {  // (the rows of a share without keys are not even written)
      const uint32_t u[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        o[2 * e] = fmaf(w, bf16_lo(u[e]), o[2 * e]);
        o[2 * e + 1] = fmaf(w, bf16_hi(u[e]), o[2 * e + 1]);
      }
    }
  };
  if (group < groups) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (group + i * groups < splits) add(group + i * groups, v[i]);
    for (int s = group + kAhead * groups; s < splits; s += groups) add(s, *reinterpret_cast<const uint4*>(src + static_cast<size_t>(s) * N * a.DV));
  }
  if (groups > 1) {
#pragma unroll
    for (int e = 0; e < 8; ++e) sum[threadIdx.x][e] = o[e];
    __syncthreads();
    if (group == 0)
      for (int g = 1; g < groups; ++g)
#pragma unroll
        for (int e = 0; e < 8; ++e) o[e] += sum[g * chunks + chunk][e];
  }
  if (group == 0) st8(a.out + ((static_cast<long long>(seq.row0) - a.row_base) * a.H + row) * a.DV + 8 * chunk, o);
}

constexpr int kLatSmemLimit = 232448;

template <typename F>
int for_rows(int n, F&& f) {
  if (n <= 16) return f(std::integral_constant<int, 16>());
  if (n <= 32) return f(std::integral_constant<int, 32>());
  return f(std::integral_constant<int, 64>());
}

// Ring size for row tiles of n; false if the sizes do not fit.
bool plan_tc(int n, int d, int dv, LatTcArgs& a, int& smem) {
  a.blocks = (dv + 127) / 128;
  a.tile_slots = (d + 127) / 128;
  uint32_t cols = 32;
  while (static_cast<int>(cols) < (a.blocks + 4) * n) cols *= 2;
  a.tmem_cols = cols;
  if (cols > 512) return false;
  const int left = kLatSmemLimit - lat_smem(n, a.tile_slots, 0).total;
  a.slots = left > 0 ? left / kLatSlot : 0;
  if (a.slots > kLatMaxSlots) a.slots = kLatMaxSlots;
  if (a.slots > 3 * a.tile_slots) a.slots = 3 * a.tile_slots;
  const int rows = n * dv * 2;  // in the end over the slots
  if (a.slots * kLatSlot < rows) a.slots = (rows + kLatSlot - 1) / kLatSlot;
  a.ahead = a.slots >= 2 * a.tile_slots;
  if (a.slots < a.tile_slots || a.slots > kLatMaxSlots || (n > 32 && !a.ahead)) return false;
  smem = lat_smem(n, a.tile_slots, a.slots).total;
  return smem <= kLatSmemLimit;
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
  for (int n : {16, 32, 64})
    for_rows(n, [&](auto nn) {
      if (e == cudaSuccess)
        e = cudaFuncSetAttribute(latent_attention_kernel<decltype(nn)::value>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLatSmemLimit);
      return 0;
    });
  if (e != cudaSuccess) return static_cast<int>(e);
  if (dev < 64) done.fetch_or(1ull << dev, std::memory_order_release);
  return 0;
}

size_t latent_attention_scratch_bytes(int dv) {
  // as many partial results as rows of CTAs that a launch with a split key range has: at most two rounds of 64-row tiles
  return static_cast<size_t>(2 * sm_count()) * 64 * (static_cast<size_t>(dv) * 2 + 8) + 16;
}

int latent_attention(const LatentAttn& a, const SeqDesc* seqs, int n_seqs, int longest, cudaStream_t st) {
  if (!a.q || !a.cache || !a.out || !seqs || n_seqs <= 0 || n_seqs > 65535 || longest <= 0 || a.H <= 0 || a.D <= 0 || a.D > kLatMax ||
      a.DV <= 0 || a.DV > a.D || a.max_len <= 0 || static_cast<long long>(longest) * a.H > 0x7fffffffLL)
    return TEENY_ERR_BAD_ARG;
  {
    const int rc = latent_attention_prepare();
    if (rc) return rc;
  }
  const uintptr_t bases = reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.cache);
  const int rows = longest * a.H;
  if (!a.f32 && a.D % 8 == 0 && a.DV % 8 == 0 && (bases & 15) == 0 && (reinterpret_cast<uintptr_t>(a.out) & 15) == 0 &&
      a.ldq == static_cast<long long>(a.H) * a.D && a.ldo == static_cast<long long>(a.H) * a.DV) {
    LatTcArgs t{};
    int smem = 0, n = rows <= 16 ? 16 : (rows <= 32 ? 32 : 64);
    while (n >= 16 && !plan_tc(n, a.D, a.DV, t, smem)) n /= 2;
    const int tiles = n >= 16 ? (rows + n - 1) / n : 0;
    if (n >= 16 && tiles <= 65535) {
      t.out = static_cast<bf16*>(a.out);
      t.row_base = a.row_base;
      t.H = a.H; t.D = a.D; t.DV = a.DV;
      t.scale_log2 = a.scale * 1.4426950408889634f;
      t.err = device_error_word();
      if (!t.err) return TEENY_ERR_DRIVER;  // kernels report expired waits through this word: no launch without it
      CUtensorMap mc, mq;
      const uint64_t cd[3] = {static_cast<uint64_t>(a.D), static_cast<uint64_t>(a.max_len), static_cast<uint64_t>(a.slots)};
      const uint64_t cs[2] = {static_cast<uint64_t>(a.D) * 2, static_cast<uint64_t>(a.D) * 2 * a.max_len};
      const uint32_t cb[3] = {64, kLatTile, 1};
      int rc = encode_tensor_map_bf16(&mc, a.cache, 3, cd, cs, cb);
      if (rc) return rc;
      const uint64_t qd[2] = {static_cast<uint64_t>(a.D), static_cast<uint64_t>(a.q_rows) * a.H};
      const uint64_t qs[1] = {static_cast<uint64_t>(a.D) * 2};
      const uint32_t qb[2] = {64, static_cast<uint32_t>(n)};
      rc = encode_tensor_map_bf16(&mq, a.q, 2, qd, qs, qb);
      if (rc) return rc;
      // shares of the keys per row tile: fewest rounds of tiles, each CTA's start and end counted as four; as far as there is
      // scratch for the partial results
      const long long work = static_cast<long long>(tiles) * n_seqs;
      const int key_tiles = (a.max_len + kLatTile - 1) / kLatTile;
      int splits = 1;
      long long best = -1;
      for (int c = 1; c <= kLatMaxSplits && (c == 1 || (c <= key_tiles && a.scratch && work * c * n * (a.DV * 2 + 8) + 16 <= static_cast<long long>(a.scratch_bytes)));
           ++c) {
        const long long cost = ((work * c + sm_count() - 1) / sm_count()) * ((key_tiles + c - 1) / c + 4) + (c > 1 ? 3 : 0);
        if (best < 0 || cost < best) {
          best = cost;
          splits = c;
        }
      }
      t.part_ml = static_cast<float2*>(a.scratch);
      t.part_o = reinterpret_cast<bf16*>(static_cast<uint8_t*>(a.scratch) + (work * splits * n * 8 + 15) / 16 * 16);
      rc = for_rows(n, [&](auto nn) {
        constexpr int N = decltype(nn)::value;
        launch_kernel(latent_attention_kernel<N>, dim3(splits, tiles, n_seqs), dim3(kLatThreads), smem, st, 1, mc, mq, t, seqs);
        return static_cast<int>(cudaGetLastError());
      });
      if (rc || splits == 1) return rc;
      launch_kernel(latent_merge_kernel, dim3(rows, n_seqs), dim3(128), 0, st, 1, t, seqs, n, tiles, splits);
      return static_cast<int>(cudaGetLastError());
    }
  }
  const dim3 grid(static_cast<unsigned>(rows), n_seqs);
  if (a.f32) launch_kernel(latent_attention_rows_kernel<float>, grid, dim3(256), 0, st, 1, a, seqs);
  else launch_kernel(latent_attention_rows_kernel<bf16>, grid, dim3(256), 0, st, 1, a, seqs);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace teeny
