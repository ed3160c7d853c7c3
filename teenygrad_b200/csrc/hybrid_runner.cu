// Hybrid decoder runner (include/teeny_hybrid.h): the executor that strings the recurrent, windowed-attention and GEMM
// kernels into steps over state slots, with graph replay of the decode step.  Generation state, token selection and
// graph capture are those of every runner (decoder_base.h).
//
// Per layer (T tokens of any number of sequences; x is the f32 residual stream):
//   y = rms_norm(x [+= previous delta])                 residual add + norm (the delta normed and scaled first, with POST_NORM)
//   proj = y W_in^T                                     one tcgen05 GEMM for all inputs of all branches
//   per branch, into its columns of `mix`:
//     attention   windowed: q, k <- head norm + rotary; attention over ring and own tokens; ring update
//                 full: q, k <- rotary, v <- mixed values, k and v into the cache; attention over the cache * gate
//     latent      norms + rotary + cache append; q = c_q W_uq^T; long portions: keys and values from the latents by one GEMM,
//                 attention; the rest: queries into the latent space, attention over the cache, values out of it
//     delta       low = tanh(W_1 h); wz = low W_low^T; state scan; per-head norm * gate
//     decay       state scan; norm over all heads * gate
//     min-gru     element-wise scan * gate
//   delta = mix W_out^T
//   y = rms_norm(x += delta); act = act(y Wg^T) * (y Wu^T) in the GEMM's epilogue; delta = act W_down^T
// then the final norm on the rows that want logits and the LM head.
#include <cstring>
#include <new>
#include <vector>

#include "../../include/teeny_b200.h"
#include "../../include/teeny_hybrid.h"
#include "decoder_base.h"

namespace teeny {

namespace {

inline int pad8(int n) { return (n + 7) / 8 * 8; }
inline int pad64(int n) { return (n + 63) / 64 * 64; }

// A branch with its place in the layer's fused input rows and output columns.
struct Branch {
  teeny_hybrid_branch c;
  int in[6] = {};   // column of each input part in `proj`
  int n_in = 0;     // input rows (padded)
  int out_col = 0, n_out = 0;
  size_t state = 0, v_ring = 0;  // workspace offsets: matrix / vector state, or the key ring; the value ring
  int ring = 0;
  const float *q_norm = nullptr, *k_norm = nullptr, *o_norm = nullptr, *decay_bias = nullptr, *rate_bias = nullptr;
  const float *z_bias = nullptr, *x_bias = nullptr, *decay = nullptr, *inv_freq = nullptr;
  const void* low = nullptr;
  const float *sink = nullptr, *value_mix = nullptr;
  const void *uq = nullptr, *expand = nullptr, *absorb = nullptr, *value_up = nullptr;
  int v_mode = kMixNone;
  bool full() const { return c.kind == TEENY_HYBRID_ATTENTION && c.window == 0; }
  int head() const { return c.rot_dims + c.dim; }     // LATENT: a head of q or of the expanded keys
  int latent() const { return pad8(c.rank); }
  int row() const { return latent() + c.rot_dims; }   // LATENT: a cache row
  bool keys_are_values() const { return (c.flags & TEENY_HYBRID_KEYS_ARE_VALUES) != 0; }
};

struct Layer {
  std::vector<Branch> branches;
  int n_in = 0, n_out = 0, ff = 0, act = 0, flags = 0;
  const float *norm1 = nullptr, *norm2 = nullptr, *norm1_post = nullptr, *norm2_post = nullptr;
  const void *in_bias = nullptr, *w_in = nullptr, *w_out = nullptr, *gate_up = nullptr, *down = nullptr;
};

struct Plan {
  std::vector<Layer> layers;
  size_t x, y, proj, mix, delta, act, gu, o32, low, wz, kbuf, yrows, logits, logits16;
  size_t attn_scratch, attn_counters, attn_scratch_bytes;
  size_t v_first, cq, lat_q, lat_rows, lat_kv, lat_qa, lat_oa, lat_scratch, lat_scratch_bytes;  // value mixing; latent attention
  int v_first_ld, cq_ld, lat_q_ld, lat_row_ld, lat_kv_ld, lat_qa_ld, lat_oa_ld;
  int absorb_rows;  // most rows of one absorbed run
  size_t seqs, rows, sample_u, best_val, next_ids, cur_ids, history, state, total;
  size_t slot_bytes;
  int proj_ld, mix_ld, act_ld, o_ld, low_ld, wz_ld, k_ld, vocab_ld, width_ld;
};

bool valid_branch(const teeny_hybrid_branch& b) {
  switch (b.kind) {
    case TEENY_HYBRID_ATTENTION:
      return b.heads > 0 && b.kv_heads > 0 && b.heads % b.kv_heads == 0 && b.dim > 0 && b.dim <= 256 && b.vdim > 0 && b.vdim <= 256 &&
             b.window >= 0 && b.rot_dims >= 0 && b.rot_dims <= b.dim && b.rot_dims % 2 == 0 &&
             (!(b.flags & TEENY_HYBRID_KEYS_ARE_VALUES) || (b.vdim == b.dim && !(b.flags & TEENY_HYBRID_OUT_GATE))) &&
             (!(b.flags & TEENY_HYBRID_VALUE_MIX) || (b.window == 0 && !(b.flags & TEENY_HYBRID_KEYS_ARE_VALUES))) && b.softcap >= 0.0f;
    case TEENY_HYBRID_LATENT:
      return b.heads > 0 && b.dim > 0 && b.dim % 8 == 0 && b.vdim > 0 && b.vdim % 8 == 0 && b.vdim <= 256 && b.rot_dims >= 0 &&
             b.rot_dims % 8 == 0 && b.dim + b.rot_dims <= 256 && b.rank > 0 && b.q_rank > 0 && pad8(b.rank) + b.rot_dims <= 1024;
    case TEENY_HYBRID_DELTA:
      return b.heads > 0 && b.dim > 0 && b.vdim == b.dim && b.rank > 0 && state_scan_supports(b.dim, b.vdim);
    case TEENY_HYBRID_DECAY:
      return b.heads > 0 && b.dim > 0 && b.vdim > 0 && state_scan_supports(b.dim, b.vdim);
    case TEENY_HYBRID_MIN_GRU:
      return b.dim > 0;
    default:
      return false;
  }
}

bool make_plan(const teeny_hybrid_config& c, const teeny_hybrid_layer* layers, const teeny_hybrid_branch* branches, Plan& p) {
  if (c.num_layers <= 0 || c.num_branches <= 0 || c.width <= 0 || c.vocab <= 0 || c.max_batch <= 0 || c.max_batch > 1024 ||
      c.max_len <= 0 || c.max_tokens < c.max_batch || c.max_rows < c.max_batch || c.max_new_tokens < 0 || !layers || !branches)
    return false;
  p.layers.assign(c.num_layers, Layer());
  p.proj_ld = p.mix_ld = p.o_ld = p.low_ld = p.wz_ld = p.k_ld = 8;
  p.act_ld = 64;
  p.v_first_ld = p.cq_ld = p.lat_q_ld = p.lat_row_ld = p.lat_kv_ld = p.lat_qa_ld = p.lat_oa_ld = 0;
  p.lat_scratch_bytes = 0;
  int mixed_values = 0;  // columns of the first branch that mixes values
  p.attn_scratch_bytes = 0;
  int kv_heads = 1;
  const size_t es = c.f32 ? 4 : 2;
  const size_t T = c.max_tokens, Bm = c.max_batch;
  size_t o = 0;
  auto take = [&](size_t bytes) { const size_t at = o; o += align_up(bytes); return at; };
  p.slot_bytes = 0;
  auto up = [](int& have, int want) { if (want > have) have = want; };
  for (int l = 0; l < c.num_layers; ++l) {
    const teeny_hybrid_layer& lc = layers[l];
    if (lc.num_branches <= 0 || lc.first_branch < 0 || lc.first_branch + lc.num_branches > c.num_branches || lc.ff < 0) return false;
    if (lc.ff > 0 && lc.act != TEENY_HYBRID_ACT_SILU && lc.act != TEENY_HYBRID_ACT_GELU_TANH) return false;
    Layer& L = p.layers[l];
    L.ff = pad64(lc.ff);
    L.act = lc.act;
    L.flags = lc.flags;
    up(p.act_ld, L.ff);
    for (int i = 0; i < lc.num_branches; ++i) {
      Branch b;
      b.c = branches[lc.first_branch + i];
      if (!valid_branch(b.c)) return false;
      const int H = b.c.heads, D = b.c.dim, V = b.c.vdim;
      int sizes[6], n = 0;
      switch (b.c.kind) {
        case TEENY_HYBRID_ATTENTION:
          sizes[n++] = H * D; sizes[n++] = b.c.kv_heads * D;
          if (!b.keys_are_values()) sizes[n++] = b.c.kv_heads * V;
          if (b.c.flags & TEENY_HYBRID_OUT_GATE) sizes[n++] = H * V;
          if (b.c.flags & TEENY_HYBRID_VALUE_MIX) {
            b.v_mode = mixed_values ? kMixWith : kMixKeep;
            if (mixed_values && mixed_values != b.c.kv_heads * V) return false;
            mixed_values = b.c.kv_heads * V;
            p.v_first_ld = pad8(mixed_values);
          }
          b.n_out = H * V;
          b.ring = b.c.window > 0 && b.c.window < c.max_len ? b.c.window : c.max_len;
          b.state = take(Bm * b.c.kv_heads * static_cast<size_t>(b.ring) * D * es);
          b.v_ring = take(Bm * b.c.kv_heads * static_cast<size_t>(b.ring) * V * es);
          p.slot_bytes += b.c.kv_heads * static_cast<size_t>(b.ring) * (D + V) * es;
          up(p.k_ld, pad8(b.c.kv_heads * D));
          up(kv_heads, b.c.kv_heads);
          if (!c.f32) {
            const size_t need = attention_decode_scratch_bytes(c.max_batch, H, D <= 64 && V <= 64 ? 64 : 128, b.ring);
            if (need > p.attn_scratch_bytes) p.attn_scratch_bytes = need;
          }
          break;
        case TEENY_HYBRID_LATENT:
          sizes[n++] = b.c.q_rank; sizes[n++] = b.c.rank; sizes[n++] = b.c.rot_dims;
          b.n_out = H * V;
          b.state = take(Bm * c.max_len * b.row() * es);
          p.slot_bytes += static_cast<size_t>(c.max_len) * b.row() * es;
          up(p.cq_ld, pad8(b.c.q_rank));
          up(p.lat_q_ld, H * b.head());
          up(p.lat_row_ld, b.row());
          up(p.lat_kv_ld, H * (b.head() + V));
          up(p.lat_qa_ld, H * b.row());
          up(p.lat_oa_ld, H * b.latent());
          if (!c.f32) {
            const size_t need = latent_attention_scratch_bytes(b.latent());
            if (need > p.lat_scratch_bytes) p.lat_scratch_bytes = need;
          }
          break;
        case TEENY_HYBRID_DELTA:
          for (; n < 5; ++n) sizes[n] = H * D;
          sizes[n++] = b.c.rank;
          b.n_out = H * V;
          up(p.low_ld, pad8(b.c.rank));
          up(p.wz_ld, pad8(H * D));
          break;
        case TEENY_HYBRID_DECAY:
          sizes[n++] = H * D; sizes[n++] = H * D; sizes[n++] = H * V; sizes[n++] = H * V;
          b.n_out = H * V;
          break;
        default:
          for (; n < 3; ++n) sizes[n] = D;
          b.n_out = D;
          b.state = take(Bm * D * 4);
          p.slot_bytes += static_cast<size_t>(D) * 4;
      }
      if (b.c.kind == TEENY_HYBRID_DELTA || b.c.kind == TEENY_HYBRID_DECAY) {
        const size_t per = static_cast<size_t>(H) * D * V * 4;
        b.state = take(Bm * per);
        p.slot_bytes += per;
        up(p.o_ld, pad8(H * V));
      }
      for (int k = 0; k < n; ++k) {
        b.in[k] = L.n_in;
        L.n_in += pad8(sizes[k]);
        b.n_in += pad8(sizes[k]);
      }
      b.out_col = L.n_out;
      L.n_out += pad8(b.n_out);
      L.branches.push_back(b);
    }
    up(p.proj_ld, L.n_in);
    up(p.mix_ld, L.n_out);
  }
  p.width_ld = pad8(c.width);
  p.vocab_ld = pad8(c.vocab);
  p.x = take(T * c.width * 4);
  p.y = take(T * p.width_ld * es);
  p.proj = take(T * p.proj_ld * es);
  p.mix = take(T * p.mix_ld * es);
  p.delta = take(T * p.width_ld * es);
  p.act = take(T * p.act_ld * es);
  p.gu = take(c.f32 ? T * 2 * p.act_ld * es : 0);
  p.o32 = take(T * p.o_ld * 4);
  p.low = take(T * p.low_ld * es);
  p.wz = take(T * p.wz_ld * es);
  p.kbuf = take(T * p.k_ld * es);
  p.v_first = take(T * p.v_first_ld * es);
  p.cq = take(T * p.cq_ld * es);
  p.lat_q = take(T * p.lat_q_ld * es);
  p.lat_rows = take(T * p.lat_row_ld * es);
  p.lat_kv = take((T > static_cast<size_t>(c.max_len) ? T : c.max_len) * p.lat_kv_ld * es);
  p.absorb_rows = c.max_tokens < 2048 ? c.max_tokens : (c.max_batch > 2048 ? c.max_batch : 2048);
  p.lat_qa = take(static_cast<size_t>(p.absorb_rows) * p.lat_qa_ld * es);
  p.lat_oa = take(static_cast<size_t>(p.absorb_rows) * p.lat_oa_ld * es);
  p.lat_scratch = take(p.lat_scratch_bytes);
  p.yrows = take(static_cast<size_t>(c.max_rows) * p.width_ld * es);
  p.logits = take(static_cast<size_t>(c.max_rows) * p.vocab_ld * es);
  p.logits16 = take(c.f32 ? Bm * p.vocab_ld * 2 : 0);
  p.attn_scratch = take(p.attn_scratch_bytes);
  p.attn_counters = take(Bm * kv_heads * 4);
  p.seqs = take(Bm * sizeof(SeqDesc));
  p.rows = take(static_cast<size_t>(c.max_rows) * 4);
  p.sample_u = take(Bm * 4);
  p.best_val = take(Bm * 4);
  p.next_ids = take(Bm * 4);
  p.cur_ids = take(Bm * 4);
  p.history = take(Bm * 4 * static_cast<size_t>(c.max_new_tokens > 0 ? c.max_new_tokens : 1));
  p.state = take(16);
  p.total = o;
  return true;
}

}  // namespace

}  // namespace teeny

using namespace teeny;

struct teeny_hybrid : DecoderBase {
  teeny_hybrid_config cfg;
  Plan p;
  const void *embed = nullptr, *lm_head = nullptr;
  const float* final_norm = nullptr;
  std::vector<SeqDesc> last;  // the entries of the last step
  int last_rows = 0;
  bool pending_delta = false;
  const float* pending_post = nullptr;  // norm behind the pending sublayer, or null
  bool checked = false;       // every weight is there

  SeqDesc* seqs() const { return at<SeqDesc>(p.seqs); }
};

namespace {

// y[M, N] = x[M, K] W^T (+ bias), in the model's element type; glu: act(gate) * up with N counting both.
int linear(teeny_hybrid* m, const void* x, int ldx, const void* w, int ldw, void* y, int ldy, int M, int N, int K, cudaStream_t st,
           int glu = 0, const void* bias = nullptr) {
  if (m->cfg.f32) {
    float* out = glu ? m->at<float>(m->p.gu) : static_cast<float*>(y);
    const int ldo = glu ? N : ldy;
    TEENY_TRY(gemm_f32(static_cast<const float*>(x), ldx, 1, static_cast<const float*>(w), 1, ldw, static_cast<const float*>(bias), out, ldo, 1, M, N, K, st));
    return glu ? glu_interleaved_f32(out, ldo, static_cast<float*>(y), ldy, M, N / 2, glu, st) : 0;
  }
  return gemm_bf16(static_cast<const bf16*>(x), ldx, static_cast<const bf16*>(w), ldw, false, static_cast<const bf16*>(bias), static_cast<bf16*>(y), ldy, M, N,
                   K, nullptr, 0, st, glu);
}

struct StepShape {
  int T, n, max_len;  // tokens, entries, longest entry
  bool uniform_fresh; // whole prompts of one length from position 0
  const SeqDesc* host; // the entries; null in decode (single tokens, positions on the device)
};

// Address of column `col` of row 0 of an activation buffer in the model's element type.
void* column(const teeny_hybrid* m, size_t buf, int col) {
  return m->at<uint8_t>(buf) + static_cast<size_t>(col) * (m->cfg.f32 ? 4 : 2);
}

// Element (row, column) of a buffer with `ld` columns; row may be negative (kernels add the entries' row numbers).
void* element(const teeny_hybrid* m, size_t buf, long long row, long long ld, long long col = 0) {
  return m->at<uint8_t>(buf) + (row * ld + col) * (m->cfg.f32 ? 4 : 2);
}

// Attention over a cache that never wraps: everything new goes into the cache first.
int run_full_attention(teeny_hybrid* m, const Layer& L, const Branch& b, const StepShape& s, cudaStream_t st) {
  const Plan& p = m->p;
  const teeny_hybrid_branch& c = b.c;
  HeadNormRope r{};
  r.f32 = m->cfg.f32;
  r.q = column(m, p.proj, b.in[0]);
  r.k_raw = column(m, p.proj, b.in[1]);
  r.ldq = r.ldkr = r.ldv = L.n_in;
  r.q_w = b.q_norm; r.k_w = b.k_norm; r.inv_freq = b.inv_freq;
  r.Hq = c.heads; r.Hkv = c.kv_heads; r.D = c.dim; r.rot_dims = c.rot_dims;
  r.eps = m->cfg.eps;
  r.rot_scale = c.rot_scale;
  r.k_ring = m->at<void>(b.state);
  r.v_ring = m->at<void>(b.v_ring);
  r.ring = b.ring;
  if (!b.keys_are_values()) {
    r.v = column(m, p.proj, b.in[2]);
    r.DV = c.vdim;
    r.v_mode = b.v_mode;
    r.v_first = m->at<void>(p.v_first);
    r.ldvf = p.v_first_ld;
    r.mix = b.value_mix;
  }
  TEENY_TRY(head_norm_rope_rows(r, m->seqs(), s.n, s.max_len, st));
  WindowAttn a{};
  a.f32 = m->cfg.f32;
  a.q = r.q; a.ldq = L.n_in;
  a.k_ring = r.k_ring;
  a.v_ring = r.v_ring;
  a.ring = a.window = b.ring;
  a.out = column(m, p.mix, b.out_col);
  a.ldo = L.n_out;
  a.Hq = c.heads; a.Hkv = c.kv_heads; a.D = c.dim; a.DV = c.vdim;
  a.scale = c.score_scale; a.out_scale = c.out_scale;
  a.slots = m->cfg.max_batch;
  a.keys = kKeysInRing;
  a.scratch = m->at<void>(p.attn_scratch);
  a.scratch_bytes = p.attn_scratch_bytes;
  a.counters = m->at<unsigned>(p.attn_counters);
  a.softcap = c.softcap;
  a.sink = b.sink;
  if (c.flags & TEENY_HYBRID_OUT_GATE) {
    a.gate = column(m, p.proj, b.in[3]);
    a.ldg = L.n_in;
  }
  a.host = s.host;
  return window_attention(a, m->seqs(), s.n, s.max_len, st);
}

constexpr int kExpandLen = 64;  // entries from here on have their keys and values made from the latents

// Entries e0 .. e0 + n - 1 (rows r0 .. r0 + rows - 1) in the latent space.
int run_latent_absorbed(teeny_hybrid* m, const Layer& L, const Branch& b, int e0, int n, int r0, int rows, int longest, cudaStream_t st) {
  const Plan& p = m->p;
  const teeny_hybrid_branch& c = b.c;
  const int H = c.heads, D = b.head(), KR = b.latent(), DL = b.row();
  const SeqDesc* seqs = m->seqs() + e0;
  HeadLinear in{};
  in.f32 = m->cfg.f32;
  in.x = element(m, p.lat_q, r0, H * D, c.rot_dims);
  in.ldx = H * D; in.x_head = D;
  in.w = b.absorb;
  in.y = m->at<void>(p.lat_qa);
  in.ldy = H * DL; in.y_head = DL;
  in.H = H; in.N = KR; in.K = c.dim; in.T = rows;
  in.RD = c.rot_dims; in.rot_off = -c.rot_dims;
  in.inv_freq = b.inv_freq; in.rot_scale = c.rot_scale;
  in.seqs = seqs; in.n_seqs = n;
  TEENY_TRY(head_linear(in, st));
  LatentAttn a{};
  a.f32 = m->cfg.f32;
  a.q = in.y; a.ldq = H * DL;
  a.q_rows = rows; a.row_base = r0;
  a.cache = m->at<void>(b.state);
  a.slots = m->cfg.max_batch;
  a.max_len = m->cfg.max_len;
  a.out = m->at<void>(p.lat_oa); a.ldo = H * KR;
  a.H = H; a.D = DL; a.DV = KR;
  a.scale = c.score_scale;
  a.scratch = m->at<void>(p.lat_scratch);
  a.scratch_bytes = p.lat_scratch_bytes;
  TEENY_TRY(latent_attention(a, seqs, n, longest, st));
  HeadLinear out{};
  out.f32 = m->cfg.f32;
  out.x = m->at<void>(p.lat_oa);
  out.ldx = H * KR; out.x_head = KR;
  out.w = b.value_up;
  out.y = element(m, p.mix, r0, L.n_out, b.out_col);
  out.ldy = L.n_out; out.y_head = c.vdim;
  out.H = H; out.N = c.vdim; out.K = KR; out.T = rows;
  return head_linear(out, st);
}

// Entries e0 .. e0 + n - 1, whole prompts so far (their latents in the step's rows) or one entry with a past (in the cache).
int run_latent_expanded(teeny_hybrid* m, const Layer& L, const Branch& b, const StepShape& s, int e0, int n, int rows, int longest,
                        bool uniform, cudaStream_t st) {
  const Plan& p = m->p;
  const teeny_hybrid_branch& c = b.c;
  const int H = c.heads, D = b.head(), DL = b.row(), ld = H * (D + c.vdim);
  const SeqDesc* seqs = m->seqs() + e0;
  const SeqDesc first = s.host[e0];
  HeadNormRope r{};
  r.f32 = m->cfg.f32;
  r.q = m->at<void>(p.lat_q); r.ldq = H * D;
  r.inv_freq = b.inv_freq;
  r.Hq = H; r.D = D; r.rot_dims = c.rot_dims;
  r.rot_scale = c.rot_scale;
  if (c.rot_dims) TEENY_TRY(head_norm_rope_rows(r, seqs, n, longest, st));
  const void* latents = first.pos == 0 ? element(m, p.lat_rows, first.row0, DL)
                                       : element(m, b.state, static_cast<long long>(first.slot) * m->cfg.max_len, DL);
  TEENY_TRY(linear(m, latents, DL, b.expand, DL, m->at<void>(p.lat_kv), ld, first.pos + rows, ld, DL, st));
  WindowAttn a{};
  a.f32 = m->cfg.f32;
  a.q = r.q; a.ldq = H * D;
  a.k_new = element(m, p.lat_kv, first.pos - first.row0, ld);  // row of the entry's first token
  a.v_new = element(m, p.lat_kv, first.pos - first.row0, ld, H * D);
  a.ldk = a.ldv = ld;
  a.ring = a.window = m->cfg.max_len;
  a.out = column(m, p.mix, b.out_col);
  a.ldo = L.n_out;
  a.Hq = a.Hkv = H; a.D = D; a.DV = c.vdim;
  a.scale = c.score_scale; a.out_scale = c.out_scale;
  a.slots = m->cfg.max_batch;
  a.keys = kKeysInNew;
  a.host = s.host + e0;
  a.uniform_fresh = uniform && first.row0 == 0;
  return window_attention(a, seqs, n, longest, st);
}

int run_latent(teeny_hybrid* m, const Layer& L, const Branch& b, const StepShape& s, cudaStream_t st) {
  const Plan& p = m->p;
  const teeny_hybrid_branch& c = b.c;
  LatentPrepare a{};
  a.f32 = m->cfg.f32;
  a.proj = m->at<void>(p.proj);
  a.ld = L.n_in;
  a.off_q = b.in[0]; a.off_c = b.in[1]; a.off_r = b.in[2];
  a.q_rank = c.q_rank; a.rank = c.rank; a.RD = c.rot_dims;
  a.q_w = b.q_norm; a.c_w = b.k_norm; a.inv_freq = b.inv_freq;
  a.eps = m->cfg.eps; a.rot_scale = c.rot_scale;
  a.cq = m->at<void>(p.cq); a.ldcq = p.cq_ld;
  a.rows = s.host ? m->at<void>(p.lat_rows) : nullptr;
  a.cache = m->at<void>(b.state);
  a.max_len = m->cfg.max_len;
  TEENY_TRY(latent_prepare(a, m->seqs(), s.n, s.max_len, st));
  const int nq = c.heads * b.head();
  TEENY_TRY(linear(m, a.cq, p.cq_ld, b.uq, pad8(c.q_rank), m->at<void>(p.lat_q), nq, s.T, nq, c.q_rank, st));
  if (!s.host) return run_latent_absorbed(m, L, b, 0, s.n, 0, s.T, 1, st);
  // runs of entries that go the same way
  for (int e = 0; e < s.n;) {
    const SeqDesc f = s.host[e];
    int n = 1, rows = f.len, longest = f.len;
    auto take = [&](const SeqDesc& q) { ++n; rows += q.len; longest = q.len > longest ? q.len : longest; };
    if (f.len < kExpandLen) {
      while (e + n < s.n && s.host[e + n].len < kExpandLen && rows + s.host[e + n].len <= p.absorb_rows) take(s.host[e + n]);
      TEENY_TRY(run_latent_absorbed(m, L, b, e, n, f.row0, rows, longest, st));
    } else {
      bool uniform = f.pos == 0;
      if (f.pos == 0)
        while (e + n < s.n && s.host[e + n].len >= kExpandLen && s.host[e + n].pos == 0) {
          uniform = uniform && s.host[e + n].len == f.len;
          take(s.host[e + n]);
        }
      TEENY_TRY(run_latent_expanded(m, L, b, s, e, n, rows, longest, uniform, st));
    }
    e += n;
  }
  return 0;
}

int run_attention(teeny_hybrid* m, const Layer& L, const Branch& b, const StepShape& s, cudaStream_t st) {
  const Plan& p = m->p;
  const teeny_hybrid_branch& c = b.c;
  HeadNormRope r{};
  r.f32 = m->cfg.f32;
  r.q = column(m, p.proj, b.in[0]);
  r.ldq = L.n_in;
  r.k_raw = column(m, p.proj, b.in[1]);
  r.ldkr = L.n_in;
  r.k_out = m->at<void>(p.kbuf);
  r.ldk = p.k_ld;
  r.q_w = b.q_norm; r.k_w = b.k_norm; r.inv_freq = b.inv_freq;
  r.Hq = c.heads; r.Hkv = c.kv_heads; r.D = c.dim; r.rot_dims = c.rot_dims;
  r.eps = m->cfg.eps;
  r.rot_scale = c.rot_scale;
  const bool single = s.max_len == 1 && b.keys_are_values();  // decode: the new key goes into the ring on the way
  if (single) {
    r.k_ring = m->at<void>(b.state);
    r.v_ring = m->at<void>(b.v_ring);
    r.ring = b.ring;
  }
  TEENY_TRY(head_norm_rope_rows(r, m->seqs(), s.n, s.max_len, st));
  WindowAttn a{};
  a.f32 = m->cfg.f32;
  a.q = r.q; a.ldq = L.n_in;
  a.k_new = r.k_out; a.ldk = p.k_ld;
  a.v_new = column(m, p.proj, b.keys_are_values() ? b.in[1] : b.in[2]);
  a.ldv = L.n_in;
  a.k_ring = m->at<void>(b.state);
  a.v_ring = m->at<void>(b.v_ring);
  a.ring = b.ring; a.window = c.window;
  a.out = column(m, p.mix, b.out_col);
  a.ldo = L.n_out;
  a.Hq = c.heads; a.Hkv = c.kv_heads; a.D = c.dim; a.DV = c.vdim;
  a.scale = c.score_scale; a.out_scale = c.out_scale;
  a.softcap = c.softcap;
  a.sink = b.sink;
  if (c.flags & TEENY_HYBRID_OUT_GATE) {
    a.gate = column(m, p.proj, b.in[3]);
    a.ldg = L.n_in;
  }
  a.slots = m->cfg.max_batch;
  a.uniform_fresh = s.uniform_fresh;
  a.keys = single ? kKeysInRing : kKeysSplit;
  a.scratch = m->at<void>(p.attn_scratch);
  a.scratch_bytes = p.attn_scratch_bytes;
  a.counters = m->at<unsigned>(p.attn_counters);
  TEENY_TRY(window_attention(a, m->seqs(), s.n, s.max_len, st));
  return single ? 0 : ring_append(a, m->seqs(), s.n, s.max_len, st);
}

int run_matrix_state(teeny_hybrid* m, const Layer& L, const Branch& b, const StepShape& s, cudaStream_t st) {
  const Plan& p = m->p;
  const teeny_hybrid_branch& c = b.c;
  const bool delta = c.kind == TEENY_HYBRID_DELTA;
  const int n = c.heads * c.dim;
  StateScan a{};
  a.mode = delta ? kScanDelta : kScanDecay;
  a.f32 = m->cfg.f32;
  a.proj = m->at<void>(p.proj);
  a.ld = L.n_in;
  a.off_q = b.in[0]; a.off_k = b.in[1]; a.off_v = b.in[2];
  a.state = m->at<float>(b.state);
  a.o = m->at<float>(p.o32);
  a.ldo = p.o_ld;
  a.H = c.heads; a.DK = c.dim; a.DV = c.vdim;
  if (delta) {
    TEENY_TRY(tanh_rows(column(m, p.proj, b.in[5]), L.n_in, m->at<void>(p.low), p.low_ld, s.T, c.rank, m->cfg.f32, st));
    TEENY_TRY(linear(m, m->at<void>(p.low), p.low_ld, b.low, pad8(c.rank), m->at<void>(p.wz), p.wz_ld, s.T, n, c.rank, st));
    a.off_a = b.in[3];
    a.wz = m->at<void>(p.wz);
    a.ld_wz = p.wz_ld;
    a.w_bias = b.decay_bias; a.a_bias = b.rate_bias;
    a.decay_coef = c.decay_coef; a.unit_eps = c.unit_eps;
    a.norm_w = b.o_norm;
    a.off_g = b.in[4];
    a.out = column(m, p.mix, b.out_col);
    a.ldout = L.n_out;
    a.norm_eps = m->cfg.eps;
    a.out_scale = c.out_scale;
  } else {
    a.decay = b.decay;
  }
  bool normed = false;
  TEENY_TRY(state_scan(a, m->seqs(), s.n, s.max_len, st, &normed));
  if (normed) return 0;
  return gated_rms_norm(a.o, a.ldo, column(m, p.proj, b.in[delta ? 4 : 3]), L.n_in, b.o_norm, column(m, p.mix, b.out_col), L.n_out,
                        s.T, b.n_out, delta ? c.vdim : b.n_out, m->cfg.eps, c.out_scale, m->cfg.f32 != 0, st);
}

int run_min_gru(teeny_hybrid* m, const Layer& L, const Branch& b, const StepShape& s, cudaStream_t st) {
  MinGru a{};
  a.f32 = m->cfg.f32;
  a.proj = m->at<void>(m->p.proj);
  a.ld = L.n_in;
  a.off_z = b.in[0]; a.off_x = b.in[1]; a.off_g = b.in[2];
  a.z_bias = b.z_bias; a.x_bias = b.x_bias;
  a.state = m->at<float>(b.state);
  a.out = column(m, m->p.mix, b.out_col);
  a.ldout = L.n_out;
  a.W = b.c.dim;
  a.scale = b.c.out_scale;
  return min_gru(a, m->seqs(), s.n, s.max_len, st);
}

// residual += pending sublayer output (normed and scaled, where the layer does that); y = norm(residual)
int norm(teeny_hybrid* m, const float* w, int T, cudaStream_t st) {
  const Plan& p = m->p;
  const void* d = m->pending_delta ? m->at<void>(p.delta) : nullptr;
  m->pending_delta = false;
  return residual_rms_norm(m->at<float>(p.x), d, p.width_ld, m->at<void>(p.y), p.width_ld, w, T, m->cfg.width, m->cfg.eps, nullptr,
                           m->cfg.f32 != 0, st, m->pending_post, m->cfg.residual_mult);
}

int run_layers(teeny_hybrid* m, const int* ids, const StepShape& s, cudaStream_t st) {
  const Plan& p = m->p;
  const int d = m->cfg.width;
  void *y = m->at<void>(p.y), *delta = m->at<void>(p.delta), *act = m->at<void>(p.act);
  TEENY_TRY(embedding_scaled(ids, m->embed, m->at<float>(p.x), s.T, d, m->cfg.vocab, m->cfg.embed_scale, m->cfg.f32 != 0, st));
  m->pending_delta = false;
  for (const Layer& L : p.layers) {
    TEENY_TRY(norm(m, L.norm1, s.T, st));
    TEENY_TRY(linear(m, y, p.width_ld, L.w_in, p.width_ld, m->at<void>(p.proj), L.n_in, s.T, L.n_in, d, st, 0, L.in_bias));
    for (const Branch& b : L.branches) {
      if (b.full()) TEENY_TRY(run_full_attention(m, L, b, s, st));
      else if (b.c.kind == TEENY_HYBRID_ATTENTION) TEENY_TRY(run_attention(m, L, b, s, st));
      else if (b.c.kind == TEENY_HYBRID_LATENT) TEENY_TRY(run_latent(m, L, b, s, st));
      else if (b.c.kind == TEENY_HYBRID_MIN_GRU) TEENY_TRY(run_min_gru(m, L, b, s, st));
      else TEENY_TRY(run_matrix_state(m, L, b, s, st));
    }
    TEENY_TRY(linear(m, m->at<void>(p.mix), L.n_out, L.w_out, L.n_out, delta, p.width_ld, s.T, d, L.n_out, st));
    m->pending_delta = true;
    m->pending_post = L.norm1_post;
    if (L.ff) {
      TEENY_TRY(norm(m, L.norm2, s.T, st));
      TEENY_TRY(linear(m, y, p.width_ld, L.gate_up, p.width_ld, act, L.ff, s.T, 2 * L.ff, d, st, L.act));
      TEENY_TRY(linear(m, act, L.ff, L.down, L.ff, delta, p.width_ld, s.T, d, L.ff, st));
      m->pending_delta = true;
      m->pending_post = L.norm2_post;
    }
  }
  return 0;
}

// Final norm and LM head on the rows that want logits: `rows` (device row numbers), or the first n rows when null.
int run_head(teeny_hybrid* m, const int* rows, int n, cudaStream_t st) {
  const Plan& p = m->p;
  void* y = m->at<void>(p.yrows);
  TEENY_TRY(residual_rms_norm(m->at<float>(p.x), m->at<void>(p.delta), p.width_ld, y, p.width_ld, m->final_norm, n, m->cfg.width,
                              m->cfg.eps, rows, m->cfg.f32 != 0, st, m->pending_post, m->cfg.residual_mult));
  return linear(m, y, p.width_ld, m->lm_head, p.width_ld, m->at<void>(p.logits), p.vocab_ld, n, m->cfg.vocab, m->cfg.width, st);
}

// Tokens of the first n rows of logits into next_ids.
int pick(teeny_hybrid* m, int n, const int* step_dev, cudaStream_t st) {
  const Plan& p = m->p;
  int* next = m->at<int>(p.next_ids);
  float *u = m->at<float>(p.sample_u), *best = m->at<float>(p.best_val);
  if (!m->cfg.f32) return select_tokens(m, m->at<bf16>(p.logits), p.vocab_ld, n, m->cfg.vocab, step_dev, u, best, next, st);
  if (m->sample_temperature <= 0.0f) return argmax_f32(m->at<float>(p.logits), p.vocab_ld, best, next, n, m->cfg.vocab, st);
  TEENY_TRY(f32_to_bf16(m->at<float>(p.logits), m->at<bf16>(p.logits16), static_cast<long long>(n) * p.vocab_ld, st));
  return select_tokens(m, m->at<bf16>(p.logits16), p.vocab_ld, n, m->cfg.vocab, step_dev, u, best, next, st);
}

int record(teeny_hybrid* m, int n, cudaStream_t st) {
  const Plan& p = m->p;
  return finish_step(m->at<int>(p.next_ids), m->at<int>(p.cur_ids), m->at<int>(p.history), m->at<int>(p.state), n,
                     m->cfg.max_new_tokens, nullptr, m->seqs(), st);
}

int decode_body(teeny_hybrid* m, int n, cudaStream_t st) {
  PdlScope pdl;
  TEENY_TRY(run_layers(m, m->at<int>(m->p.cur_ids), StepShape{n, n, 1, false, nullptr}, st));
  TEENY_TRY(run_head(m, nullptr, n, st));
  TEENY_TRY(pick(m, n, m->at<int>(m->p.state) + 2, st));
  return record(m, n, st);
}

int check_ready(teeny_hybrid* m) {
  if (m->checked) return 0;
  if (!m->embed || !m->final_norm || !m->lm_head) return TEENY_ERR_BAD_ARG;
  for (const Layer& L : m->p.layers) {
    if (!L.norm1 || !L.w_in || !L.w_out || (L.ff && (!L.norm2 || !L.gate_up || !L.down))) return TEENY_ERR_BAD_ARG;
    if ((L.flags & TEENY_HYBRID_IN_BIAS) && !L.in_bias) return TEENY_ERR_BAD_ARG;
    if ((L.flags & TEENY_HYBRID_POST_NORM) && (!L.norm1_post || (L.ff && !L.norm2_post))) return TEENY_ERR_BAD_ARG;
    for (const Branch& b : L.branches) {
      bool ok = true;
      switch (b.c.kind) {
        case TEENY_HYBRID_ATTENTION:
          ok = (!(b.c.flags & TEENY_HYBRID_QK_NORM) || (b.q_norm && b.k_norm)) && (!b.c.rot_dims || b.inv_freq) &&
               (!(b.c.flags & TEENY_HYBRID_SINK) || b.sink) && (b.v_mode != kMixWith || b.value_mix);
          break;
        case TEENY_HYBRID_LATENT:
          ok = b.q_norm && b.k_norm && b.uq && b.expand && b.absorb && b.value_up && (!b.c.rot_dims || b.inv_freq);
          break;
        case TEENY_HYBRID_DELTA: ok = b.o_norm && b.low && b.decay_bias && b.rate_bias; break;
        case TEENY_HYBRID_DECAY: ok = b.o_norm && b.decay; break;
        default: ok = b.z_bias && b.x_bias;
      }
      if (!ok) return TEENY_ERR_BAD_ARG;
    }
  }
  m->checked = true;
  return 0;
}

}  // namespace

extern "C" {

size_t teeny_hybrid_workspace_bytes(const teeny_hybrid_config* cfg, const teeny_hybrid_layer* layers, const teeny_hybrid_branch* branches) {
  Plan p;
  return cfg && make_plan(*cfg, layers, branches, p) ? p.total : 0;
}

size_t teeny_hybrid_slot_bytes(const teeny_hybrid_config* cfg, const teeny_hybrid_layer* layers, const teeny_hybrid_branch* branches) {
  Plan p;
  return cfg && make_plan(*cfg, layers, branches, p) ? p.slot_bytes : 0;
}

int teeny_hybrid_create(const teeny_hybrid_config* cfg, const teeny_hybrid_layer* layers, const teeny_hybrid_branch* branches,
                        void* workspace, size_t workspace_bytes, teeny_stream_t stream, teeny_hybrid** out) {
  if (!cfg || !workspace || !out) return TEENY_ERR_BAD_ARG;
  if (reinterpret_cast<uintptr_t>(workspace) & 255) return TEENY_ERR_ALIGNMENT;
  teeny_hybrid* m = new (std::nothrow) teeny_hybrid();
  if (!m) return TEENY_ERR_BAD_ARG;
  int rc = make_plan(*cfg, layers, branches, m->p) ? 0 : TEENY_ERR_BAD_ARG;
  if (rc == 0 && workspace_bytes < m->p.total) rc = TEENY_ERR_SCRATCH;
  // function attributes (dynamic shared memory) are set once per device here, outside any stream capture
  if (rc == 0) rc = gemm_bf16_prepare();
  if (rc == 0) rc = gemm_bf16_2cta_prepare();
  if (rc == 0) rc = state_scan_prepare();
  if (rc == 0) rc = window_attention_prepare();
  if (rc == 0) rc = latent_attention_prepare();
  m->cfg = *cfg;
  m->ws = static_cast<uint8_t*>(workspace);
  // Arrival counters start at zero, and everything starts finite: padding columns are multiplied by zero weights.  (Rings and
  // states of fresh slots are never read.)
  if (rc == 0) rc = static_cast<int>(cudaMemsetAsync(workspace, 0, m->p.total, reinterpret_cast<cudaStream_t>(stream)));
  if (rc != 0) {
    delete m;
    return rc;
  }
  *out = m;
  return 0;
}

void teeny_hybrid_destroy(teeny_hybrid* m) {
  if (!m) return;
  destroy_base(m);
  delete m;
}

int teeny_hybrid_set_weight(teeny_hybrid* m, int layer, int branch, int which, const void* ptr) {
  if (!m || !ptr) return TEENY_ERR_BAD_ARG;
  if (reinterpret_cast<uintptr_t>(ptr) & 15) return TEENY_ERR_ALIGNMENT;
  const float* f = static_cast<const float*>(ptr);
  m->checked = false;
  switch (which) {
    case TEENY_HYBRID_W_EMBED: m->embed = ptr; return 0;
    case TEENY_HYBRID_W_FINAL_NORM: m->final_norm = f; return 0;
    case TEENY_HYBRID_W_LM_HEAD: m->lm_head = ptr; return 0;
    default: break;
  }
  if (layer < 0 || layer >= m->cfg.num_layers) return TEENY_ERR_BAD_ARG;
  Layer& L = m->p.layers[layer];
  switch (which) {
    case TEENY_HYBRID_W_NORM1: L.norm1 = f; return 0;
    case TEENY_HYBRID_W_NORM2: L.norm2 = f; return 0;
    case TEENY_HYBRID_W_IN: L.w_in = ptr; return 0;
    case TEENY_HYBRID_W_OUT: L.w_out = ptr; return 0;
    case TEENY_HYBRID_W_GATE_UP: L.gate_up = ptr; return 0;
    case TEENY_HYBRID_W_DOWN: L.down = ptr; return 0;
    case TEENY_HYBRID_W_IN_BIAS: L.in_bias = ptr; return 0;
    case TEENY_HYBRID_W_NORM1_POST: L.norm1_post = f; return 0;
    case TEENY_HYBRID_W_NORM2_POST: L.norm2_post = f; return 0;
    default: break;
  }
  if (branch < 0 || branch >= static_cast<int>(L.branches.size())) return TEENY_ERR_BAD_ARG;
  Branch& b = L.branches[branch];
  switch (which) {
    case TEENY_HYBRID_W_Q_NORM: b.q_norm = f; return 0;
    case TEENY_HYBRID_W_K_NORM: b.k_norm = f; return 0;
    case TEENY_HYBRID_W_O_NORM: b.o_norm = f; return 0;
    case TEENY_HYBRID_W_LOW: b.low = ptr; return 0;
    case TEENY_HYBRID_W_DECAY_BIAS: b.decay_bias = f; return 0;
    case TEENY_HYBRID_W_RATE_BIAS: b.rate_bias = f; return 0;
    case TEENY_HYBRID_W_Z_BIAS: b.z_bias = f; return 0;
    case TEENY_HYBRID_W_X_BIAS: b.x_bias = f; return 0;
    case TEENY_HYBRID_W_DECAY: b.decay = f; return 0;
    case TEENY_HYBRID_W_INV_FREQ: b.inv_freq = f; return 0;
    case TEENY_HYBRID_W_SINK: b.sink = f; return 0;
    case TEENY_HYBRID_W_VALUE_MIX: b.value_mix = f; return 0;
    case TEENY_HYBRID_W_UQ: b.uq = ptr; return 0;
    case TEENY_HYBRID_W_EXPAND: b.expand = ptr; return 0;
    case TEENY_HYBRID_W_ABSORB: b.absorb = ptr; return 0;
    case TEENY_HYBRID_W_VALUE_UP: b.value_up = ptr; return 0;
    default: return TEENY_ERR_BAD_ARG;
  }
}

int teeny_hybrid_step(teeny_hybrid* m, const int* ids, const int* slots, const int* positions, const int* lens, int n,
                      const int* rows, int n_rows, teeny_stream_t stream) {
  if (!m || !ids || !slots || !positions || !lens || n <= 0 || n > m->cfg.max_batch || n_rows < 0 || n_rows > m->cfg.max_rows ||
      (n_rows > 0 && !rows))
    return TEENY_ERR_BAD_ARG;
  TEENY_TRY(check_ready(m));
  std::vector<SeqDesc> seqs(n);
  std::vector<char> used(m->cfg.max_batch, 0);
  StepShape s{0, n, 0, true, nullptr};
  for (int e = 0; e < n; ++e) {
    if (slots[e] < 0 || slots[e] >= m->cfg.max_batch || used[slots[e]] || positions[e] < 0 || lens[e] <= 0 ||
        positions[e] > m->cfg.max_len - lens[e] || lens[e] > m->cfg.max_tokens - s.T)
      return TEENY_ERR_BAD_ARG;
    used[slots[e]] = 1;
    seqs[e] = SeqDesc{slots[e], positions[e], s.T, lens[e]};
    s.T += lens[e];
    if (lens[e] > s.max_len) s.max_len = lens[e];
    s.uniform_fresh = s.uniform_fresh && positions[e] == 0 && lens[e] == lens[0];
  }
  s.host = seqs.data();
  for (int r = 0; r < n_rows; ++r)
    if (rows[r] < 0 || rows[r] >= s.T) return TEENY_ERR_BAD_ARG;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  // pageable host memory: the runtime has taken its copy when the call returns
  cudaError_t e = cudaMemcpyAsync(m->seqs(), seqs.data(), n * sizeof(SeqDesc), cudaMemcpyHostToDevice, st);
  if (e == cudaSuccess && n_rows)
    e = cudaMemcpyAsync(m->at<int>(m->p.rows), rows, static_cast<size_t>(n_rows) * 4, cudaMemcpyHostToDevice, st);
  if (e != cudaSuccess) return static_cast<int>(e);
  PdlScope pdl;
  TEENY_TRY(run_layers(m, ids, s, st));
  if (n_rows) TEENY_TRY(run_head(m, m->at<int>(m->p.rows), n_rows, st));
  m->last = seqs;
  m->last_rows = n_rows;
  m->batch = 0;  // a generation starts with teeny_hybrid_begin
  return 0;
}

int teeny_hybrid_begin(teeny_hybrid* m, teeny_stream_t stream) {
  if (!m || m->last.empty() || m->last_rows != static_cast<int>(m->last.size())) return TEENY_ERR_BAD_ARG;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const int n = m->last_rows;
  int most = 0;
  for (const SeqDesc& s : m->last) most = s.pos + s.len > most ? s.pos + s.len : most;
  TEENY_TRY(pick(m, n, nullptr, st));
  TEENY_TRY(set_generation_state(m->at<int>(m->p.state), m->last[0].pos + m->last[0].len - 1, m->last[0].pos + m->last[0].len, 0, st));
  TEENY_TRY(record(m, n, st));
  m->last.clear();
  m->batch = n;
  m->next_pos = most;
  return 0;
}

int teeny_hybrid_decode(teeny_hybrid* m, teeny_stream_t stream) {
  if (!m || m->batch <= 0 || m->next_pos >= m->cfg.max_len) return TEENY_ERR_BAD_ARG;
  const int rc = decode_body(m, m->batch, reinterpret_cast<cudaStream_t>(stream));
  if (rc == 0) ++m->next_pos;
  return rc;
}

int teeny_hybrid_set_sampling(teeny_hybrid* m, float temperature, int top_k, float top_p, unsigned long long seed) {
  return m ? set_sampling(m, temperature, top_k, top_p, seed) : static_cast<int>(TEENY_ERR_BAD_ARG);
}

int teeny_hybrid_capture_decode(teeny_hybrid* m, teeny_stream_t stream) {
  (void)stream;
  if (!m) return TEENY_ERR_BAD_ARG;
  return capture_step(m, [m](cudaStream_t st) { return decode_body(m, m->batch, st); });
}

int teeny_hybrid_decode_replay(teeny_hybrid* m, teeny_stream_t stream) {
  if (!m) return TEENY_ERR_BAD_ARG;
  return replay_step(m, m->cfg.max_len, reinterpret_cast<cudaStream_t>(stream));
}

void* teeny_hybrid_buffer(teeny_hybrid* m, int which) {
  if (!m) return nullptr;
  switch (which) {
    case TEENY_HYBRID_BUF_LOGITS: return m->ws + m->p.logits;
    case TEENY_HYBRID_BUF_NEXT_IDS: return m->ws + m->p.cur_ids;
    case TEENY_HYBRID_BUF_HISTORY: return m->ws + m->p.history;
    case TEENY_HYBRID_BUF_STATE: return m->ws + m->p.state;
    case TEENY_HYBRID_BUF_RESIDUAL: return m->ws + m->p.x;
    case TEENY_HYBRID_BUF_LAST_DELTA: return m->ws + m->p.delta;
    default: return nullptr;
  }
}

// ---- the kernels on their own ----
int teeny_state_scan(int mode, int f32, const void* proj, long long ld, int off_q, int off_k, int off_v, int off_a, const void* wz,
                     long long ld_wz, const float* w_bias, const float* a_bias, const float* decay, float decay_coef,
                     float unit_eps, float* state, float* o, long long ldo, int heads, int dk, int dv, const int* seqs,
                     int n_seqs, int max_len, teeny_stream_t stream) {
  if (mode != kScanDelta && mode != kScanDecay) return TEENY_ERR_BAD_ARG;
  TEENY_TRY(state_scan_prepare());
  StateScan a{};
  a.mode = mode; a.f32 = f32;
  a.proj = proj; a.ld = ld;
  a.off_q = off_q; a.off_k = off_k; a.off_v = off_v; a.off_a = off_a;
  a.wz = wz; a.ld_wz = ld_wz;
  a.w_bias = w_bias; a.a_bias = a_bias; a.decay = decay;
  a.decay_coef = decay_coef; a.unit_eps = unit_eps;
  a.state = state;
  a.o = o; a.ldo = ldo;
  a.H = heads; a.DK = dk; a.DV = dv;
  return state_scan(a, reinterpret_cast<const SeqDesc*>(seqs), n_seqs, max_len, reinterpret_cast<cudaStream_t>(stream));
}

int teeny_gated_rms_norm(int f32, const float* o, long long ldo, const void* gate, long long ldg, const float* weight, void* out,
                         long long ldout, int rows, int cols, int group_size, float eps, float scale, teeny_stream_t stream) {
  return gated_rms_norm(o, ldo, gate, ldg, weight, out, ldout, rows, cols, group_size, eps, scale, f32 != 0,
                        reinterpret_cast<cudaStream_t>(stream));
}

int teeny_min_gru(int f32, const void* proj, long long ld, int off_z, int off_x, int off_g, const float* z_bias, const float* x_bias,
                  float* state, void* out, long long ldout, int width, float scale, const int* seqs, int n_seqs, int max_len,
                  teeny_stream_t stream) {
  const MinGru a{f32, proj, ld, off_z, off_x, off_g, z_bias, x_bias, state, out, ldout, width, scale};
  return min_gru(a, reinterpret_cast<const SeqDesc*>(seqs), n_seqs, max_len, reinterpret_cast<cudaStream_t>(stream));
}

int teeny_head_norm_rope(int f32, void* q, long long ldq, const void* k_raw, long long ldkr, void* k_out, long long ldk,
                         const float* q_weight, const float* k_weight, const float* inv_freq, int heads, int kv_heads, int dim,
                         int rot_dims, float eps, const int* seqs, int n_seqs, int max_len, teeny_stream_t stream) {
  HeadNormRope a{};
  a.f32 = f32;
  a.q = q; a.ldq = ldq;
  a.k_raw = k_raw; a.ldkr = ldkr;
  a.k_out = k_out; a.ldk = ldk;
  a.q_w = q_weight; a.k_w = k_weight; a.inv_freq = inv_freq;
  a.Hq = heads; a.Hkv = kv_heads; a.D = dim; a.rot_dims = rot_dims;
  a.eps = eps;
  a.rot_scale = 1.0f;
  return head_norm_rope_rows(a, reinterpret_cast<const SeqDesc*>(seqs), n_seqs, max_len, reinterpret_cast<cudaStream_t>(stream));
}

int teeny_window_attention(int f32, const void* q, long long ldq, const void* k_new, long long ldk, const void* v_new, long long ldv,
                           void* k_ring, void* v_ring, int slots, int ring, int window, void* out, long long ldo, int heads,
                           int kv_heads, int dim, int vdim, float score_scale, float out_scale, int uniform_fresh,
                           const int* seqs, int n_seqs, int max_len, teeny_stream_t stream) {
  if (slots <= 0) return TEENY_ERR_BAD_ARG;
  WindowAttn a{};
  a.f32 = f32;
  a.q = q; a.ldq = ldq;
  a.k_new = k_new; a.ldk = ldk;
  a.v_new = v_new; a.ldv = ldv;
  a.k_ring = k_ring; a.v_ring = v_ring;
  a.ring = ring; a.window = window;
  a.out = out; a.ldo = ldo;
  a.Hq = heads; a.Hkv = kv_heads; a.D = dim; a.DV = vdim;
  a.scale = score_scale; a.out_scale = out_scale;
  a.slots = slots;
  a.uniform_fresh = uniform_fresh;
  const SeqDesc* sq = reinterpret_cast<const SeqDesc*>(seqs);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  TEENY_TRY(window_attention(a, sq, n_seqs, max_len, st));
  return ring_append(a, sq, n_seqs, max_len, st);
}

int teeny_residual_rms_norm(int f32, float* x, const void* delta, long long ldd, void* y, long long ldy, const float* weight, int rows,
                            int n, float eps, const float* post, float mult, teeny_stream_t stream) {
  return residual_rms_norm(x, delta, ldd, y, ldy, weight, rows, n, eps, nullptr, f32 != 0, reinterpret_cast<cudaStream_t>(stream), post, mult);
}

int teeny_rope_cache(int f32, void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv, void* k_cache,
                     void* v_cache, int max_cached, const float* inv_freq, float rot_scale, int heads, int kv_heads, int dim, int vdim,
                     int rot_dims, int mix_mode, void* v_first, const float* mix, const int* seqs, int n_seqs, int max_len,
                     teeny_stream_t stream) {
  if (!k || !v || !k_cache || !v_cache || max_cached <= 0 || kv_heads <= 0 || mix_mode < kMixNone || mix_mode > kMixWith) return TEENY_ERR_BAD_ARG;
  HeadNormRope a{};
  a.f32 = f32;
  a.q = q; a.ldq = ldq;
  a.k_raw = k; a.ldkr = ldk;
  a.inv_freq = inv_freq; a.rot_scale = rot_scale;
  a.Hq = heads; a.Hkv = kv_heads; a.D = dim; a.rot_dims = rot_dims;
  a.k_ring = k_cache; a.v_ring = v_cache; a.ring = max_cached;
  a.v = v; a.ldv = ldv; a.DV = vdim;
  a.v_mode = mix_mode; a.v_first = v_first; a.ldvf = static_cast<long long>(kv_heads) * vdim; a.mix = mix;
  return head_norm_rope_rows(a, reinterpret_cast<const SeqDesc*>(seqs), n_seqs, max_len, reinterpret_cast<cudaStream_t>(stream));
}

int teeny_cached_attention(int f32, const void* q, long long ldq, void* k_cache, void* v_cache, int slots, int max_cached, void* out,
                           long long ldo, int heads, int kv_heads, int dim, int vdim, float score_scale, float softcap,
                           const float* sink, const void* gate, long long ldg, void* scratch, size_t scratch_bytes,
                           unsigned* counters, const int* seqs, const int* host_seqs, int n_seqs, int max_len, teeny_stream_t stream) {
  if (slots <= 0) return TEENY_ERR_BAD_ARG;
  WindowAttn a{};
  a.f32 = f32;
  a.q = q; a.ldq = ldq;
  a.k_ring = k_cache; a.v_ring = v_cache;
  a.ring = a.window = max_cached;
  a.out = out; a.ldo = ldo;
  a.Hq = heads; a.Hkv = kv_heads; a.D = dim; a.DV = vdim;
  a.scale = score_scale; a.out_scale = 1.0f;
  a.slots = slots;
  a.keys = kKeysInRing;
  a.scratch = counters ? scratch : nullptr;
  a.scratch_bytes = scratch_bytes;
  a.counters = counters;
  a.softcap = softcap; a.sink = sink;
  a.gate = gate; a.ldg = ldg;
  a.host = reinterpret_cast<const SeqDesc*>(host_seqs);
  return window_attention(a, reinterpret_cast<const SeqDesc*>(seqs), n_seqs, max_len, reinterpret_cast<cudaStream_t>(stream));
}

int teeny_latent_prepare(int f32, const void* proj, long long ld, int off_q, int off_c, int off_r, int q_rank, int rank, int rot_dims,
                         const float* q_weight, const float* c_weight, const float* inv_freq, float eps, float rot_scale, void* cq,
                         long long ldcq, void* latents, void* cache, int max_cached, const int* seqs, int n_seqs, int max_len,
                         teeny_stream_t stream) {
  const LatentPrepare a{f32, proj, ld, off_q, off_c, off_r, q_rank, rank, rot_dims, q_weight, c_weight, inv_freq, eps, rot_scale,
                        cq, ldcq, latents, cache, max_cached};
  return latent_prepare(a, reinterpret_cast<const SeqDesc*>(seqs), n_seqs, max_len, reinterpret_cast<cudaStream_t>(stream));
}

int teeny_head_linear(int f32, const void* x, long long ldx, long long x_head, const void* w, void* y, long long ldy, long long y_head,
                      int heads, int n, int k, int rows, int rot_dims, int rot_off, const float* inv_freq, float rot_scale, const int* seqs,
                      int n_seqs, teeny_stream_t stream) {
  const HeadLinear a{f32, x, ldx, x_head, w, y, ldy, y_head, heads, n, k, rows, rot_dims, rot_off, inv_freq, rot_scale,
                     reinterpret_cast<const SeqDesc*>(seqs), n_seqs};
  return head_linear(a, reinterpret_cast<cudaStream_t>(stream));
}

size_t teeny_latent_attention_scratch_bytes(int vdim) { return vdim > 0 ? latent_attention_scratch_bytes(vdim) : 0; }

int teeny_latent_attention(int f32, const void* q, long long ldq, int rows, const void* cache, int slots, int max_cached, void* out,
                           long long ldo, int heads, int dim, int vdim, float score_scale, void* scratch, size_t scratch_bytes,
                           const int* seqs, int n_seqs, int max_len, teeny_stream_t stream) {
  const LatentAttn a{f32, q, ldq, rows, 0, cache, slots, max_cached, out, ldo, heads, dim, vdim, score_scale, scratch, scratch_bytes};
  return latent_attention(a, reinterpret_cast<const SeqDesc*>(seqs), n_seqs, max_len, reinterpret_cast<cudaStream_t>(stream));
}

}  // extern "C"
