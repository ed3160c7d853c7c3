// Sliding-window grouped-query attention over a per-sequence ring cache, with the head norm / rotary kernel in front of
// it.  A window of W tokens needs only the last W keys of a sequence, so a sequence's cache is a ring of
// min(W, capacity) rows: position p lives in row p % ring.  A step reads keys older than its own first token from the
// ring and its own tokens' keys from the step's activations, and leaves its last `ring` keys in the ring afterwards,
// so portions may be cut anywhere and a long prompt never overwrites a key that one of its own queries still needs.
//
// window_attention_rows_kernel<T>: one warp per (token, query head), any head size up to 256, f32 or bf16 storage, f32
// arithmetic.
#include <atomic>

#include "common.cuh"
#include "kernels.h"

namespace teeny {

namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<bf16>(const bf16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

constexpr int kMaxHead = 256;

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
    sincosf(static_cast<float>(seq.pos + i) * a.inv_freq[d], &sn[d], &cs[d]);
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  for (int u = warp; u < a.Hq + a.Hkv; u += warps) {
    const bool is_q = u < a.Hq;
    const int hd = is_q ? u : u - a.Hq;
    const T* src = is_q ? static_cast<const T*>(a.q) + row * a.ldq + hd * a.D : static_cast<const T*>(a.k_raw) + row * a.ldkr + hd * a.D;
    T* dst = is_q ? static_cast<T*>(a.q) + row * a.ldq + hd * a.D : static_cast<T*>(a.k_out) + row * a.ldk + hd * a.D;
    const float* w = is_q ? a.q_w : a.k_w;
    float* buf = rowbuf[warp];
    float sq = 0.0f;
    for (int d = lane; d < a.D; d += 32) {
      const float v = ldf(src + d);
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
      stf(dst + d, v);
    }
    __syncwarp();
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

template <typename T>
__global__ void window_attention_rows_kernel(const WindowAttn a, const SeqDesc* __restrict__ seqs) {
  pdl_wait();
  pdl_trigger();
  const SeqDesc seq = seqs[blockIdx.y];
  const int unit = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
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
  for (int j = max(0, pos - a.window + 1); j <= pos; ++j) {
    const bool fresh = j >= seq.pos;
    const T* kp = fresh ? kn + static_cast<size_t>(j - seq.pos) * a.ldk : kr + static_cast<size_t>(j % a.ring) * a.D;
    const T* vp = fresh ? vn + static_cast<size_t>(j - seq.pos) * a.ldv : vr + static_cast<size_t>(j % a.ring) * a.DV;
    float dot = 0.0f;
#pragma unroll
    for (int e = 0; e < kMaxHead / 32; ++e) {
      const int d = lane + 32 * e;
      if (d < a.D) dot = fmaf(qv[e], ldf(kp + d), dot);
    }
    dot = warp_sum(dot);
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
  const float inv = a.out_scale / l;
#pragma unroll
  for (int e = 0; e < kMaxHead / 32; ++e) {
    const int d = lane + 32 * e;
    if (d < a.DV) stf(orow + d, acc[e] * inv);
  }
}

bool valid(const WindowAttn& a, const SeqDesc* seqs, int n_seqs, int max_len) {
  return a.k_new && a.v_new && a.k_ring && a.v_ring && seqs && n_seqs > 0 && n_seqs <= 65535 && max_len > 0 && a.ring > 0 &&
         a.window > 0 && a.Hq > 0 && a.Hkv > 0 && a.Hq % a.Hkv == 0 && a.D > 0 && a.D <= kMaxHead && a.DV > 0 && a.DV <= kMaxHead;
}

}  // namespace

int head_norm_rope_rows(const HeadNormRope& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  if (!a.q || !a.k_raw || !a.k_out || !seqs || n_seqs <= 0 || n_seqs > 65535 || max_len <= 0 || a.D <= 0 || a.D > kMaxHead ||
      a.rot_dims < 0 || a.rot_dims > a.D || (a.rot_dims & 1) || (a.rot_dims && !a.inv_freq))
    return TEENY_ERR_BAD_ARG;
  const dim3 grid(max_len, n_seqs), block(256);
  if (a.f32) launch_kernel(head_norm_rope_rows_kernel<float>, grid, block, 0, st, 1, a, seqs);
  else launch_kernel(head_norm_rope_rows_kernel<bf16>, grid, block, 0, st, 1, a, seqs);
  return static_cast<int>(cudaGetLastError());
}

int window_attention_prepare() { return 0; }

int window_attention(const WindowAttn& a, const SeqDesc* seqs, int n_seqs, int max_len, cudaStream_t st) {
  if (!valid(a, seqs, n_seqs, max_len) || !a.q || !a.out) return TEENY_ERR_BAD_ARG;
  const long long units = static_cast<long long>(max_len) * a.Hq;
  const dim3 grid(static_cast<unsigned>((units + 3) / 4), n_seqs), block(128);
  if (a.f32) launch_kernel(window_attention_rows_kernel<float>, grid, block, 0, st, 1, a, seqs);
  else launch_kernel(window_attention_rows_kernel<bf16>, grid, block, 0, st, 1, a, seqs);
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
