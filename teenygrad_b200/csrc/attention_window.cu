// Sliding-window grouped-query attention over a per-sequence ring cache, with the head norm / rotary kernel in front of
// it.  A window of W tokens needs only the last W keys of a sequence, so a sequence's cache is a ring of
// min(W, capacity) rows: position p lives in row p % ring.  A step reads keys older than its own first token from the
// ring and its own tokens' keys from the step's activations, and leaves its last `ring` keys in the ring afterwards,
// so portions may be cut anywhere and a long prompt never overwrites a key that one of its own queries still needs.
//
// A cache as long as a sequence can get is a ring that never wraps: a step's keys and values then go into it first
// (kKeysInRing) and every kernel reads all keys from there.
//
// window_attention chooses among
//   attention_prefill_bf16   whole prompts of one length, and long entries whose keys lie in order (a cache that never wraps, or
//                            all in k_new); keys up to 192, values up to 128 (tcgen05 on CTA pairs, attention_prefill.cu)
//   attention_decode_bf16    single tokens, head sizes up to 128 (TMA-streamed ring, attention_decode.cu)
//   window_attention_mma_kernel   any other bf16 step, head sizes up to 256 in multiples of 8 (mma.sync tiles, cp.async rows
//                            from ring and step): portions, unequal prompts, other head sizes
//   window_attention_rows_kernel<T>   anything, f32 included: one or eight warps per (token, query head)
#include <atomic>

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

constexpr int kMaxHead = 256;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ void rope_angle(const HeadNormRope& a, int pos, int d, float* sn, float* cs) {
  sincosf(static_cast<float>(pos) * a.inv_freq[d], &sn[d], &cs[d]);
  sn[d] *= a.rot_scale;
  cs[d] *= a.rot_scale;
}

// One CTA per (token, entry): the token's cos / sin once, then a warp per head (q heads, then k heads).
template <typename T>
__global__ void head_norm_rope_rows_kernel(const HeadNormRope a, const SeqDesc* __restrict__ seqs) {
  __shared__ float cs[kMaxHead / 2], sn[kMaxHead / 2];
  __shared__ float rowbuf[8][kMaxHead];
  pdl_wait();
  pdl_trigger();
  const SeqDesc seq = seqs[blockIdx.y];
  const int i = blockIdx.x;
  if (i >= seq.len) return;
  const size_t row = static_cast<size_t>(seq.row0) + i;
  const int half = a.rot_dims >> 1;
  for (int d = threadIdx.x; d < half; d += blockDim.x)
    rope_angle(a, seq.pos + i, d, sn, cs);
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int at = a.ring ? (seq.pos + i) % a.ring : 0;
  if (a.v) {
    const float lam = a.v_mode == kMixWith ? *a.mix : 0.0f;
    for (int c = threadIdx.x; c < a.Hkv * a.DV; c += blockDim.x) {
      float v = ldf(static_cast<const T*>(a.v) + row * a.ldv + c);
      T* first = static_cast<T*>(a.v_first) + row * a.ldvf + c;
      if (a.v_mode == kMixKeep) stf(first, v);
      else if (a.v_mode == kMixWith) v = (1.0f - lam) * v + lam * ldf(first);
      const int hd = c / a.DV;
      stf(static_cast<T*>(a.v_ring) + ((static_cast<size_t>(seq.slot) * a.Hkv + hd) * a.ring + at) * a.DV + (c - hd * a.DV), v);
    }
  }
  for (int u = warp; u < a.Hq + a.Hkv; u += warps) {
    const bool is_q = u < a.Hq;
    const int hd = is_q ? u : u - a.Hq;
    const T* src = is_q ? static_cast<const T*>(a.q) + row * a.ldq + hd * a.D : static_cast<const T*>(a.k_raw) + row * a.ldkr + hd * a.D;
    T* dst = is_q ? static_cast<T*>(a.q) + row * a.ldq + hd * a.D : (a.k_out ? static_cast<T*>(a.k_out) + row * a.ldk + hd * a.D : nullptr);
    // the rotated key (and, where the values are the raw keys, the value) straight into the ring as well
    const size_t rr0 = ((static_cast<size_t>(seq.slot) * a.Hkv + hd) * a.ring + at) * a.D;
    T* kring = !is_q && a.ring ? static_cast<T*>(a.k_ring) + rr0 : nullptr;
    T* vring = !is_q && a.ring && a.v_ring && !a.v ? static_cast<T*>(a.v_ring) + rr0 : nullptr;
    const float* w = is_q ? a.q_w : a.k_w;
    float* buf = rowbuf[warp];
    float sq = 0.0f;
    for (int d = lane; d < a.D; d += 32) {
      const float v = ldf(src + d);
      if (vring) stf(vring + d, v);
      buf[d] = v;
      sq = fmaf(v, v, sq);
    }
    sq = warp_sum(sq);
    if (w) {
      const float rr = 1.0f / sqrtf(sq / static_cast<float>(a.D) + a.eps);
      for (int d = lane; d < a.D; d += 32) buf[d] = buf[d] * rr * w[d];
    }
    __syncwarp();
    for (int d = lane; d < a.D; d += 32) {
      float v = buf[d];
      if (d < half) v = v * cs[d] - buf[d + half] * sn[d];
      else if (d < 2 * half) v = v * cs[d - half] + buf[d - half] * sn[d - half];
      if (dst) stf(dst + d, v);
      if (kring) stf(kring + d, v);
    }
    __syncwarp();
  }
}

// The same for bf16 heads of whole 16-byte vectors: `lph` (a power of two) lanes hold a head, eight elements each; the
// rotation partner of a lane is rot_dims / 16 lanes away.
constexpr int kRopeTasks = 4;  // (head, lane) tasks per thread whose loads are in flight together
template <bool PLAIN>  // normed heads and no values
__global__ void __launch_bounds__(256) head_norm_rope_vec_kernel(const HeadNormRope a, const SeqDesc* __restrict__ seqs, int lph) {
  __shared__ __align__(16) float cs[kMaxHead / 2], sn[kMaxHead / 2];
  const SeqDesc seq = seqs[blockIdx.y];  // written well before the kernel in front of this one
  const int i = blockIdx.x;
  const int half = a.rot_dims >> 1;
  if (i < seq.len)
    for (int d = threadIdx.x; d < half; d += blockDim.x)
      rope_angle(a, seq.pos + i, d, sn, cs);
  pdl_wait();
  pdl_trigger();
  if (i >= seq.len) return;
  const size_t row = static_cast<size_t>(seq.row0) + i;
  const bf16* qr = static_cast<const bf16*>(a.q) + row * a.ldq;
  const bf16* kr = static_cast<const bf16*>(a.k_raw) + row * a.ldkr;
  const int lane = threadIdx.x & 31, sub = lane & (lph - 1), d0 = sub * 8;
  const int per = 256 / lph, heads = a.Hq + a.Hkv, h0 = threadIdx.x / lph;
  const int step = half >> 3;
  const int at = a.ring ? (seq.pos + i) % a.ring : 0;
  if (!PLAIN && a.v) {
    const float lam = a.v_mode == kMixWith ? *a.mix : 0.0f, keep = 1.0f - lam;
    for (int c = threadIdx.x * 8; c < a.Hkv * a.DV; c += 256 * 8) {
      uint4 v = *reinterpret_cast<const uint4*>(static_cast<const bf16*>(a.v) + row * a.ldv + c);
      bf16* first = static_cast<bf16*>(a.v_first) + row * a.ldvf + c;
      if (a.v_mode == kMixKeep) *reinterpret_cast<uint4*>(first) = v;
      else if (a.v_mode == kMixWith) {
        const uint4 f = *reinterpret_cast<const uint4*>(first);
        auto mix = [&](uint32_t p, uint32_t q) {
          return pack_bf16x2(fmaf(lam, bf16_lo(q), keep * bf16_lo(p)), fmaf(lam, bf16_hi(q), keep * bf16_hi(p)));
        };
        v = make_uint4(mix(v.x, f.x), mix(v.y, f.y), mix(v.z, f.z), mix(v.w, f.w));
      }
      const int hd = c / a.DV;
      *reinterpret_cast<uint4*>(static_cast<bf16*>(a.v_ring) + ((static_cast<size_t>(seq.slot) * a.Hkv + hd) * a.ring + at) * a.DV + (c - hd * a.DV)) = v;
    }
  }
  const int partner = (lane - sub) + (sub < step ? sub + step : (sub < 2 * step ? sub - step : sub));
  // heads of q that are not normed change in place in their rotated dimensions only
  const bool in_k = d0 < a.D, in_q = PLAIN || a.q_w ? in_k : d0 < a.rot_dims;
  for (int base = 0; base < heads; base += per * kRopeTasks) {
    uint4 raw[kRopeTasks];
#pragma unroll
    for (int t = 0; t < kRopeTasks; ++t) {
      const int u = base + t * per + h0;
      raw[t] = make_uint4(0u, 0u, 0u, 0u);
      if (u < heads && (u < a.Hq ? in_q : in_k)) raw[t] = *reinterpret_cast<const uint4*>((u < a.Hq ? qr + u * a.D : kr + (u - a.Hq) * a.D) + d0);
    }
    if (base == 0) __syncthreads();  // the angles
#pragma unroll
    for (int t = 0; t < kRopeTasks; ++t) {
      const int u = base + t * per + h0;
      if (base + t * per >= heads) break;  // uniform over the CTA
      const bool is_q = u < a.Hq, in_head = is_q ? in_q : in_k;
      const uint32_t rw[4] = {raw[t].x, raw[t].y, raw[t].z, raw[t].w};
      float x[8], sq = 0.0f;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        x[2 * e] = bf16_lo(rw[e]);
        x[2 * e + 1] = bf16_hi(rw[e]);
        sq = fmaf(x[2 * e], x[2 * e], fmaf(x[2 * e + 1], x[2 * e + 1], sq));
      }
      for (int o = lph >> 1; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      const float* w = is_q ? a.q_w : a.k_w;
      if (w && in_head) {
        const float rr = 1.0f / sqrtf(sq / static_cast<float>(a.D) + a.eps);
        const float4 w0 = __ldg(reinterpret_cast<const float4*>(w + d0)), w1 = __ldg(reinterpret_cast<const float4*>(w + d0 + 4));
        x[0] *= rr * w0.x; x[1] *= rr * w0.y; x[2] *= rr * w0.z; x[3] *= rr * w0.w;
        x[4] *= rr * w1.x; x[5] *= rr * w1.y; x[6] *= rr * w1.z; x[7] *= rr * w1.w;
      }
      const int ca = (sub < step ? sub : sub - step) * 8;
      const float sign = sub < step ? -1.0f : 1.0f;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float y = __shfl_sync(0xffffffffu, x[e], partner);
        if (sub < 2 * step) x[e] = x[e] * cs[ca + e] + sign * y * sn[ca + e];
      }
      if (u >= heads || !in_head) continue;
      const uint4 out = make_uint4(pack_bf16x2(x[0], x[1]), pack_bf16x2(x[2], x[3]), pack_bf16x2(x[4], x[5]), pack_bf16x2(x[6], x[7]));
      if (is_q) {
        *reinterpret_cast<uint4*>(static_cast<bf16*>(a.q) + row * a.ldq + u * a.D + d0) = out;
      } else {
        const int hk = u - a.Hq;
        if (a.k_out) *reinterpret_cast<uint4*>(static_cast<bf16*>(a.k_out) + row * a.ldk + hk * a.D + d0) = out;
        if (a.ring) {
          const size_t r = ((static_cast<size_t>(seq.slot) * a.Hkv + hk) * a.ring + at) * a.D + d0;
          *reinterpret_cast<uint4*>(static_cast<bf16*>(a.k_ring) + r) = out;
          if (a.v_ring && !a.v) *reinterpret_cast<uint4*>(static_cast<bf16*>(a.v_ring) + r) = raw[t];
        }
      }
    }
  }
}

template <typename T>
__global__ void ring_append_kernel(const WindowAttn a, const SeqDesc* __restrict__ seqs) {
  pdl_wait();
  pdl_trigger();
  const SeqDesc seq = seqs[blockIdx.y];
  const int keep = min(seq.len, a.ring), i = seq.len - keep + blockIdx.x;
  if (static_cast<int>(blockIdx.x) >= keep) return;
  const size_t row = static_cast<size_t>(seq.row0) + i, dst = static_cast<size_t>(seq.slot) * a.Hkv;
  const int r = (seq.pos + i) % a.ring;
  for (int c = threadIdx.x; c < a.Hkv * a.D; c += blockDim.x)
    static_cast<T*>(a.k_ring)[((dst + c / a.D) * a.ring + r) * a.D + c % a.D] = static_cast<const T*>(a.k_new)[row * a.ldk + c];
  for (int c = threadIdx.x; c < a.Hkv * a.DV; c += blockDim.x)
    static_cast<T*>(a.v_ring)[((dst + c / a.DV) * a.ring + r) * a.DV + c % a.DV] = static_cast<const T*>(a.v_new)[row * a.ldv + c];
}

__device__ __forceinline__ bool from_new(const WindowAttn& a, const SeqDesc& seq, int j) {
  return a.keys == kKeysSplit ? j >= seq.pos : a.keys == kKeysInNew;
}

// WPU warps share a (token, query head): each takes every WPU-th key with an online softmax, merged through shared memory.
template <typename T, int WPU>
__global__ void __launch_bounds__(WPU > 1 ? 32 * WPU : 128) window_attention_rows_kernel(const WindowAttn a, const SeqDesc* __restrict__ seqs) {
  __shared__ float sm_ml[WPU][2];
  __shared__ float sm_o[WPU > 1 ? WPU : 1][kMaxHead];
  pdl_wait();
  pdl_trigger();
  const SeqDesc seq = seqs[blockIdx.y];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = WPU > 1 ? blockIdx.x : blockIdx.x * (blockDim.x >> 5) + warp;
  const int i = unit / a.Hq, h = unit % a.Hq;
  if (i >= seq.len) return;
  const int hk = h / (a.Hq / a.Hkv), pos = seq.pos + i;
  const size_t row = static_cast<size_t>(seq.row0) + i;
  const T* qr = static_cast<const T*>(a.q) + row * a.ldq + h * a.D;
  const T* kn = static_cast<const T*>(a.k_new) + static_cast<size_t>(seq.row0) * a.ldk + hk * a.D;
  const T* vn = static_cast<const T*>(a.v_new) + static_cast<size_t>(seq.row0) * a.ldv + hk * a.DV;
  const T* kr = static_cast<const T*>(a.k_ring) + (static_cast<size_t>(seq.slot) * a.Hkv + hk) * a.ring * a.D;
  const T* vr = static_cast<const T*>(a.v_ring) + (static_cast<size_t>(seq.slot) * a.Hkv + hk) * a.ring * a.DV;
  float qv[kMaxHead / 32], acc[kMaxHead / 32];
#pragma unroll
  for (int e = 0; e < kMaxHead / 32; ++e) {
    const int d = lane + 32 * e;
    qv[e] = d < a.D ? ldf(qr + d) * a.scale : 0.0f;
    acc[e] = 0.0f;
  }
  float m = -INFINITY, l = 0.0f;
  for (int j = max(0, pos - a.window + 1) + (WPU > 1 ? warp : 0); j <= pos; j += WPU) {
    const bool fresh = from_new(a, seq, j);
    const T* kp = fresh ? kn + static_cast<long long>(j - seq.pos) * a.ldk : kr + static_cast<size_t>(j % a.ring) * a.D;
    const T* vp = fresh ? vn + static_cast<long long>(j - seq.pos) * a.ldv : vr + static_cast<size_t>(j % a.ring) * a.DV;
    float dot = 0.0f;
#pragma unroll
    for (int e = 0; e < kMaxHead / 32; ++e) {
      const int d = lane + 32 * e;
      if (d < a.D) dot = fmaf(qv[e], ldf(kp + d), dot);
    }
    dot = warp_sum(dot);
    if (a.softcap > 0.0f) dot = a.softcap * tanhf(dot / a.softcap);
    const float m_new = fmaxf(m, dot);
    const float corr = expf(m - m_new), p = expf(dot - m_new);
    l = fmaf(corr, l, p);
#pragma unroll
    for (int e = 0; e < kMaxHead / 32; ++e) {
      const int d = lane + 32 * e;
      if (d < a.DV) acc[e] = fmaf(corr, acc[e], p * ldf(vp + d));
    }
    m = m_new;
  }
  T* orow = static_cast<T*>(a.out) + row * a.ldo + h * a.DV;
  const T* grow = a.gate ? static_cast<const T*>(a.gate) + row * a.ldg + h * a.DV : nullptr;
  if (WPU == 1) {
    if (a.sink) l += expf(a.sink[h] - m);
    const float inv = a.out_scale / l;
#pragma unroll
    for (int e = 0; e < kMaxHead / 32; ++e) {
      const int d = lane + 32 * e;
      if (d < a.DV) stf(orow + d, acc[e] * inv * (grow ? sigmoid_f(ldf(grow + d)) : 1.0f));
    }
    return;
  }
  if (lane == 0) {
    sm_ml[warp][0] = m;
    sm_ml[warp][1] = l;
  }
#pragma unroll
  for (int e = 0; e < kMaxHead / 32; ++e) sm_o[WPU > 1 ? warp : 0][lane + 32 * e] = acc[e];
  __syncthreads();
  float mm = -INFINITY, ll = 0.0f;
#pragma unroll
  for (int w = 0; w < WPU; ++w) mm = fmaxf(mm, sm_ml[w][0]);
  for (int d = threadIdx.x; d < a.DV; d += blockDim.x) {
    float o = 0.0f;
    ll = 0.0f;
#pragma unroll
    for (int w = 0; w < WPU; ++w) {  // warps without keys hold -inf: factor 0
      const float sc = expf(sm_ml[w][0] - mm);
      ll = fmaf(sm_ml[w][1], sc, ll);
      o = fmaf(sm_o[WPU > 1 ? w : 0][d], sc, o);
    }
    if (a.sink) ll += expf(a.sink[h] - mm);
    stf(orow + d, o / ll * a.out_scale * (grow ? sigmoid_f(ldf(grow + d)) : 1.0f));
  }
}

// ---- tensor-core tiles for bf16 steps of any shape ----
// CTA = 64 queries of one head of one entry, four warps of 16 rows; keys in tiles of 64 through a two-stage cp.async ring.
// Rows come by address (ring or step), so tiles start anywhere; columns beyond the head size and rows beyond the last key
// are zero.  S = Q K^T, online softmax in the fragments (log2 domain), O += P V with P packed straight from the S fragments.
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

constexpr int kPrefillLen = 128;  // shortest entry for the tcgen05 kernel
constexpr int kQRows = 64, kKeys = 64;
constexpr int mma_smem_bytes(int nd) { return (kQRows + 4 * kKeys) * (16 * nd + 8) * 2; }

template <int ND>  // padded head size / 16
__global__ void __launch_bounds__(128) window_attention_mma_kernel(const WindowAttn a, const SeqDesc* __restrict__ seqs) {
  constexpr int DP = 16 * ND, LD = DP + 8, CH = DP / 8;
  constexpr bool kHoldQ = ND <= 8;
  extern __shared__ __align__(16) bf16 wa_smem[];
  pdl_wait();
  const SeqDesc seq = seqs[blockIdx.z];
  const int i0 = blockIdx.x * kQRows;
  if (i0 >= seq.len) return;
  const int h = blockIdx.y, hk = h / (a.Hq / a.Hkv);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, c = lane & 3;
  bf16* sq = wa_smem;
  const uint32_t sq_a = smem_u32(sq);
  auto tile_addr = [&](int stage, int v) { return sq_a + (kQRows + (2 * stage + v) * kKeys) * LD * 2; };

  const bf16* kn = static_cast<const bf16*>(a.k_new) + static_cast<size_t>(seq.row0) * a.ldk + hk * a.D;
  const bf16* vn = static_cast<const bf16*>(a.v_new) + static_cast<size_t>(seq.row0) * a.ldv + hk * a.DV;
  const bf16* kr = static_cast<const bf16*>(a.k_ring) + (static_cast<size_t>(seq.slot) * a.Hkv + hk) * a.ring * a.D;
  const bf16* vr = static_cast<const bf16*>(a.v_ring) + (static_cast<size_t>(seq.slot) * a.Hkv + hk) * a.ring * a.DV;
  const bf16* qb = static_cast<const bf16*>(a.q) + static_cast<size_t>(seq.row0) * a.ldq + h * a.D;
  const int last_i = min(i0 + kQRows, seq.len) - 1;
  const int key_lo = max(0, seq.pos + i0 - a.window + 1), key_hi = seq.pos + last_i;  // keys any row of the tile sees
  const int n_tiles = (key_hi - key_lo) / kKeys + 1;

  auto zero16 = [&](uint32_t dst) { asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};" ::"r"(dst), "r"(0u) : "memory"); };
  auto load_tile = [&](int t) {
    const uint32_t kt = tile_addr(t & 1, 0), vt = tile_addr(t & 1, 1);
    for (int idx = threadIdx.x; idx < kKeys * CH; idx += 128) {
      const int r = idx / CH, ch = idx % CH, j = key_lo + t * kKeys + r;
      const uint32_t off = static_cast<uint32_t>(r * LD + ch * 8) * 2;
      const bool in = j <= key_hi, fresh = from_new(a, seq, j);
      if (in && ch * 8 < a.D)
        cp_async16(kt + off, (fresh ? kn + static_cast<long long>(j - seq.pos) * a.ldk : kr + static_cast<size_t>(j % a.ring) * a.D) + ch * 8);
      else zero16(kt + off);
      if (in && ch * 8 < a.DV)
        cp_async16(vt + off, (fresh ? vn + static_cast<long long>(j - seq.pos) * a.ldv : vr + static_cast<size_t>(j % a.ring) * a.DV) + ch * 8);
      else zero16(vt + off);
    }
    cp_async_commit();
  };
  for (int idx = threadIdx.x; idx < kQRows * CH; idx += 128) {
    const int r = idx / CH, ch = idx % CH;
    const uint32_t dst = sq_a + static_cast<uint32_t>(r * LD + ch * 8) * 2;
    if (i0 + r <= last_i && ch * 8 < a.D) cp_async16(dst, qb + static_cast<size_t>(i0 + r) * a.ldq + ch * 8);
    else zero16(dst);
  }
  load_tile(0);

  const uint32_t qa_addr = sq_a + static_cast<uint32_t>((warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + (lane >> 4) * 8) * 2;
  const uint32_t ko = static_cast<uint32_t>(((lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8) * 2;
  const uint32_t vo = static_cast<uint32_t>(((lane & 7) + ((lane >> 3) & 1) * 8) * LD + (lane >> 4) * 8) * 2;
  uint32_t qf[kHoldQ ? ND : 1][4];
  float O[2 * ND][4];
#pragma unroll
  for (int n = 0; n < 2 * ND; ++n) O[n][0] = O[n][1] = O[n][2] = O[n][3] = 0.0f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
  const float sc = a.scale * kLog2e;
  const bool capped = a.softcap > 0.0f;
  const float two_y = capped ? 2.0f * sc / a.softcap : 0.0f, cap_l2 = a.softcap * kLog2e;
  const int p_lo = seq.pos + i0 + warp * 16;  // position of the warp's first row; rows g and g + 8
  for (int t = 0; t < n_tiles; ++t) {
    if (t + 1 < n_tiles) {
      load_tile(t + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (kHoldQ && t == 0) {
#pragma unroll
      for (int k = 0; k < ND; ++k) ldsm_x4(qf[kHoldQ ? k : 0], qa_addr + k * 32);
    }
    const int j0 = key_lo + t * kKeys;
    if (j0 <= p_lo + 15 && j0 + kKeys > p_lo - a.window + 1) {  // some row of the warp sees some key of the tile
      const uint32_t kt = tile_addr(t & 1, 0), vt = tile_addr(t & 1, 1);
      float s[kKeys / 8][4];
#pragma unroll
      for (int n = 0; n < kKeys / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.0f;
#pragma unroll
      for (int k = 0; k < ND; ++k) {
        uint32_t q[4];
        if (kHoldQ) {
#pragma unroll
          for (int e = 0; e < 4; ++e) q[e] = qf[kHoldQ ? k : 0][e];
        } else {
          ldsm_x4(q, qa_addr + k * 32);
        }
#pragma unroll
        for (int n = 0; n < kKeys / 8; n += 2) {
          uint32_t b[4];
          ldsm_x4(b, kt + ko + static_cast<uint32_t>(n * 8 * LD) * 2 + k * 32);
          mma_bf16_16816(s[n], q[0], q[1], q[2], q[3], b[0], b[1]);
          mma_bf16_16816(s[n + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
        }
      }
      const bool mask = j0 + kKeys - 1 > p_lo || j0 < p_lo + 16 - a.window;
      float mx[2] = {m[0], m[1]};
#pragma unroll
      for (int n = 0; n < kKeys / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int p = p_lo + g + 8 * (e >> 1), j = j0 + 8 * n + 2 * c + (e & 1);
          const float x = capped ? softcap_log2(s[n][e], two_y, cap_l2) : s[n][e] * sc;
          s[n][e] = mask && (j > p || j <= p - a.window) ? -INFINITY : x;
          mx[e >> 1] = fmaxf(mx[e >> 1], s[n][e]);
        }
      float alpha[2], base[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        base[r] = mx[r] == -INFINITY ? 0.0f : mx[r];  // a row that has seen no key yet
        alpha[r] = ex2(m[r] - base[r]);
        m[r] = mx[r];
        l[r] *= alpha[r];
      }
#pragma unroll
      for (int n = 0; n < 2 * ND; ++n) {
        O[n][0] *= alpha[0]; O[n][1] *= alpha[0]; O[n][2] *= alpha[1]; O[n][3] *= alpha[1];
      }
#pragma unroll
      for (int k = 0; k < kKeys / 16; ++k) {
        uint32_t pf[4];
#pragma unroll
        for (int f = 0; f < 2; ++f) {
          float* x = s[2 * k + f];
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = ex2(x[e] - base[e >> 1]);
          l[0] += x[0] + x[1];
          l[1] += x[2] + x[3];
          pf[2 * f] = pack_bf16x2(x[0], x[1]);
          pf[2 * f + 1] = pack_bf16x2(x[2], x[3]);
        }
#pragma unroll
        for (int n = 0; n < 2 * ND; n += 2) {
          uint32_t b[4];
          ldsm_x4_trans(b, vt + vo + static_cast<uint32_t>(k * 16 * LD + n * 8) * 2);
          mma_bf16_16816(O[n], pf[0], pf[1], pf[2], pf[3], b[0], b[1]);
          mma_bf16_16816(O[n + 1], pf[0], pf[1], pf[2], pf[3], b[2], b[3]);
        }
      }
    }
    __syncthreads();  // the stage is free for the tile after the next
  }
  pdl_trigger();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int i = i0 + warp * 16 + g + 8 * r;
    if (i > last_i) continue;
    if (a.sink) l[r] += ex2(fmaf(a.sink[h], kLog2e, -m[r]));
    const float inv = a.out_scale / l[r];
    const size_t row = static_cast<size_t>(seq.row0) + i;
    bf16* orow = static_cast<bf16*>(a.out) + row * a.ldo + h * a.DV;
    const bf16* grow = a.gate ? static_cast<const bf16*>(a.gate) + row * a.ldg + h * a.DV : nullptr;
#pragma unroll
    for (int n = 0; n < 2 * ND; ++n) {
      const int d = 8 * n + 2 * c;
      if (d >= a.DV) continue;
      float o0 = O[n][2 * r] * inv, o1 = O[n][2 * r + 1] * inv;
      if (grow) {
        const uint32_t g2 = *reinterpret_cast<const uint32_t*>(grow + d);
        o0 *= sigmoid_f(bf16_lo(g2));
        o1 *= sigmoid_f(bf16_hi(g2));
      }
      *reinterpret_cast<uint32_t*>(orow + d) = pack_bf16x2(o0, o1);
    }
  }
}

bool valid(const WindowAttn& a, const SeqDesc* seqs, int n_seqs, int max_len) {
  return (a.keys == kKeysInRing || (a.k_new && a.v_new)) && (a.keys == kKeysInNew || (a.k_ring && a.v_ring)) && seqs && n_seqs > 0 && n_seqs <= 65535 && max_len > 0 && a.ring > 0 &&
         a.window > 0 && a.Hq > 0 && a.Hkv > 0 && a.Hq % a.Hkv == 0 && a.D > 0 && a.D <= kMaxHead && a.DV > 0 && a.DV <= kMaxHead;
}

}  // namespace

int head_norm_rope_rows(const HeadNormRope& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  if (!a.q || (a.Hkv > 0 && (!a.k_raw || (!a.k_out && !a.ring))) || !seqs || n_seqs <= 0 || n_seqs > 65535 || max_len <= 0 || a.D <= 0 ||
      a.D > kMaxHead || a.rot_dims < 0 || a.rot_dims > a.D || (a.rot_dims & 1) || (a.rot_dims && !a.inv_freq) || a.ring < 0 ||
      (a.ring && !a.k_ring))
    return TEENY_ERR_BAD_ARG;
  if (a.v && (!a.ring || !a.v_ring || a.DV <= 0 || (a.v_mode != kMixNone && !a.v_first) || (a.v_mode == kMixWith && !a.mix)))
    return TEENY_ERR_BAD_ARG;
  const dim3 grid(max_len, n_seqs), block(256);
  const uintptr_t bases = reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k_raw) | reinterpret_cast<uintptr_t>(a.k_out) |
                          reinterpret_cast<uintptr_t>(a.k_ring) | reinterpret_cast<uintptr_t>(a.v_ring) | reinterpret_cast<uintptr_t>(a.q_w) |
                          reinterpret_cast<uintptr_t>(a.k_w) | reinterpret_cast<uintptr_t>(a.v) | reinterpret_cast<uintptr_t>(a.v_first);
  if (!a.f32 && a.D % 8 == 0 && a.DV % 8 == 0 && a.rot_dims % 16 == 0 && ((a.ldq | a.ldkr | a.ldk | a.ldv | a.ldvf) & 7) == 0 && (bases & 15) == 0) {
    int lph = 1;
    while (lph * 8 < (a.Hkv == 0 && !a.q_w ? a.rot_dims : a.D)) lph *= 2;
    if (a.q_w && !a.v) launch_kernel(head_norm_rope_vec_kernel<true>, grid, block, 0, st, 1, a, seqs, lph);
    else launch_kernel(head_norm_rope_vec_kernel<false>, grid, block, 0, st, 1, a, seqs, lph);
    return static_cast<int>(cudaGetLastError());
  }
  if (a.f32) launch_kernel(head_norm_rope_rows_kernel<float>, grid, block, 0, st, 1, a, seqs);
  else launch_kernel(head_norm_rope_rows_kernel<bf16>, grid, block, 0, st, 1, a, seqs);
  return static_cast<int>(cudaGetLastError());
}

int window_attention_prepare() {
  static std::atomic<unsigned long long> done{0};  // one bit per device; threads may race to set it
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 64 && (done.load(std::memory_order_acquire) >> dev) & 1ull) return 0;
  cudaError_t e = cudaFuncSetAttribute(window_attention_mma_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, mma_smem_bytes(4));
  if (e == cudaSuccess) e = cudaFuncSetAttribute(window_attention_mma_kernel<8>, cudaFuncAttributeMaxDynamicSharedMemorySize, mma_smem_bytes(8));
  if (e == cudaSuccess) e = cudaFuncSetAttribute(window_attention_mma_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, mma_smem_bytes(16));
  if (e != cudaSuccess) return static_cast<int>(e);
  int rc = attention_prefill_prepare();
  if (rc == 0) rc = attention_decode_prepare();
  if (rc == 0 && dev < 64) done.fetch_or(1ull << dev, std::memory_order_release);
  return rc;
}

int window_attention(const WindowAttn& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  if (!valid(a, seqs, n_seqs, max_len) || !a.q || !a.out) return TEENY_ERR_BAD_ARG;
  {
    const int rc = window_attention_prepare();
    if (rc) return rc;
  }
  const int G = a.Hq / a.Hkv;
  // 16-byte rows everywhere
  const uintptr_t bases = reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.k_new) | reinterpret_cast<uintptr_t>(a.v_new) |
                          reinterpret_cast<uintptr_t>(a.k_ring) | reinterpret_cast<uintptr_t>(a.v_ring) | reinterpret_cast<uintptr_t>(a.out);
  const bool rows16 = !a.f32 && a.D % 8 == 0 && a.DV % 8 == 0 && ((a.ldq | a.ldk | a.ldv | a.ldo | a.ldg) & 7) == 0 && (bases & 15) == 0;
  const int head = a.D > a.DV ? a.D : a.DV;
  AttnShape s{};
  s.Hq = a.Hq; s.Hkv = a.Hkv; s.D = a.D; s.DV = a.DV; s.scale = a.scale; s.out_scale = a.out_scale;
  s.softcap = a.softcap; s.sink = a.sink;
  s.q_sb = a.ldq; s.q_sh = a.D; s.q_ss = a.ldq;
  s.o_sb = a.ldo; s.o_sh = a.DV; s.o_ss = a.ldo;
  // the ring as a tensor [slot, kv head, row, d]
  s.k_ss = a.D; s.k_sh = static_cast<long long>(a.ring) * a.D; s.k_sb = s.k_sh * a.Hkv;
  s.v_ss = a.DV; s.v_sh = static_cast<long long>(a.ring) * a.DV; s.v_sb = s.v_sh * a.Hkv;
  if (rows16 && max_len == 1 && a.keys == kKeysInRing && head <= 128 && (G == 1 || G == 2 || G == 4 || G == 8) && a.scratch &&
      a.scratch_bytes >= attention_decode_scratch_bytes(n_seqs, a.Hq, head <= 64 ? 64 : 128, a.ring)) {
    s.B = n_seqs; s.Sq = 1; s.Skv = a.ring;
    s.gate = static_cast<const bf16*>(a.gate); s.gate_sb = a.ldg;
    const DecodeRing ring{seqs, a.slots};
    // (the kernel before this one, head_norm_rope_rows, wrote q and each sequence's newest ring row)
    return attention_decode_bf16(static_cast<const bf16*>(a.q), static_cast<const bf16*>(a.k_ring), static_cast<const bf16*>(a.v_ring),
                                 static_cast<bf16*>(a.out), s, 0, nullptr, a.scratch, a.scratch_bytes, st, 1, nullptr, a.counters, &ring);
  }
  const bool prefill = rows16 && a.D <= 192 && a.DV <= 128 && a.scale > 0.0f;
  if (prefill && a.keys == kKeysInRing && a.host && a.window >= a.ring && max_len >= kPrefillLen) {
    // Entries of equal length and position in neighbouring slots make one launch over the cache; short ones in between go
    // to the other kernels together.
    WindowAttn rest = a;
    rest.host = nullptr;
    for (int e = 0; e < n_seqs;) {
      const SeqDesc f = a.host[e];
      int n = 1;
      if (f.len < kPrefillLen) {
        int most = f.len;
        for (; e + n < n_seqs && a.host[e + n].len < kPrefillLen; ++n) most = a.host[e + n].len > most ? a.host[e + n].len : most;
        const int rc = window_attention(rest, seqs + e, n, most, st);
        if (rc) return rc;
      } else {
        while (e + n < n_seqs && a.host[e + n].len == f.len && a.host[e + n].pos == f.pos && a.host[e + n].slot == f.slot + n &&
               a.host[e + n].row0 == f.row0 + n * f.len)
          ++n;
        s.B = n; s.Sq = f.len; s.Skv = f.pos + f.len; s.causal = 1;
        s.q_sb = f.len * a.ldq; s.o_sb = f.len * a.ldo;
        bf16* out = static_cast<bf16*>(a.out) + static_cast<size_t>(f.row0) * a.ldo;
        if (a.gate) {
          s.gate = static_cast<const bf16*>(a.gate) + static_cast<size_t>(f.row0) * a.ldg;
          s.gate_sb = f.len * a.ldg;
          s.gate_ss = a.ldg;
        }
        const int rc = attention_prefill_bf16(static_cast<const bf16*>(a.q) + static_cast<size_t>(f.row0) * a.ldq,
                                              static_cast<const bf16*>(a.k_ring) + static_cast<size_t>(f.slot) * s.k_sb,
                                              static_cast<const bf16*>(a.v_ring) + static_cast<size_t>(f.slot) * s.v_sb, out, nullptr, s, st);
        if (rc) return rc;
      }
      e += n;
    }
    return 0;
  }
  // whole prompts of one length, or one entry with its keys all in k_new
  const bool alone = a.keys == kKeysInNew && a.host && n_seqs == 1;
  if (prefill && ((a.uniform_fresh && a.keys != kKeysInRing) || alone) && max_len >= kPrefillLen) {
    const long long first = alone ? a.host->row0 : 0, pos = alone ? a.host->pos : 0;
    s.B = n_seqs; s.Sq = max_len; s.Skv = max_len + static_cast<int>(pos); s.causal = 1;
    s.window = a.window < s.Skv ? a.window : 0;
    s.q_sb = max_len * a.ldq; s.o_sb = max_len * a.ldo;
    s.k_sb = max_len * a.ldk; s.k_sh = a.D; s.k_ss = a.ldk;
    s.v_sb = max_len * a.ldv; s.v_sh = a.DV; s.v_ss = a.ldv;
    bf16* out = static_cast<bf16*>(a.out) + first * a.ldo;
    if (a.gate) {
      s.gate = static_cast<const bf16*>(a.gate) + first * a.ldg;
      s.gate_sb = max_len * a.ldg;
      s.gate_ss = a.ldg;
    }
    return attention_prefill_bf16(static_cast<const bf16*>(a.q) + first * a.ldq, static_cast<const bf16*>(a.k_new) + (first - pos) * a.ldk,
                                  static_cast<const bf16*>(a.v_new) + (first - pos) * a.ldv, out, nullptr, s, st);
  }
  if (rows16 && max_len >= 8) {
    const dim3 grid((max_len + kQRows - 1) / kQRows, a.Hq, n_seqs), block(128);
    if (head <= 64) launch_kernel(window_attention_mma_kernel<4>, grid, block, mma_smem_bytes(4), st, 1, a, seqs);
    else if (head <= 128) launch_kernel(window_attention_mma_kernel<8>, grid, block, mma_smem_bytes(8), st, 1, a, seqs);
    else launch_kernel(window_attention_mma_kernel<16>, grid, block, mma_smem_bytes(16), st, 1, a, seqs);
    return static_cast<int>(cudaGetLastError());
  }
  const long long units = static_cast<long long>(max_len) * a.Hq;
  if (max_len <= 16 && a.window > 32) {  // few rows: eight warps each
    const dim3 grid(static_cast<unsigned>(units), n_seqs), block(256);
    if (a.f32) launch_kernel(window_attention_rows_kernel<float, 8>, grid, block, 0, st, 1, a, seqs);
    else launch_kernel(window_attention_rows_kernel<bf16, 8>, grid, block, 0, st, 1, a, seqs);
  } else {
    const dim3 grid(static_cast<unsigned>((units + 3) / 4), n_seqs), block(128);
    if (a.f32) launch_kernel(window_attention_rows_kernel<float, 1>, grid, block, 0, st, 1, a, seqs);
    else launch_kernel(window_attention_rows_kernel<bf16, 1>, grid, block, 0, st, 1, a, seqs);
  }
  return static_cast<int>(cudaGetLastError());
}

int ring_append(const WindowAttn& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  if (!valid(a, seqs, n_seqs, max_len)) return TEENY_ERR_BAD_ARG;
  const dim3 grid(max_len < a.ring ? max_len : a.ring, n_seqs), block(128);
  if (a.f32) launch_kernel(ring_append_kernel<float>, grid, block, 0, st, 1, a, seqs);
  else launch_kernel(ring_append_kernel<bf16>, grid, block, 0, st, 1, a, seqs);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace teeny
