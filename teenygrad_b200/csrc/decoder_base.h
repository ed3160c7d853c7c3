// What the model runners of this library share: the generation state that lives in device memory, token selection
// behind the LM head, and recording / replaying one decode step as a CUDA graph.  A runner derives its handle from
// DecoderBase and supplies the layer loop.
#pragma once

#include <functional>

#include "common.cuh"
#include "kernels.h"

namespace teeny {

#define TEENY_TRY(expr)                  \
  do {                                   \
    const int rc_ = (expr);              \
    if (rc_ != 0) return rc_;            \
  } while (0)

inline size_t align_up(size_t v, size_t a = 256) { return (v + a - 1) / a * a; }

// While alive, this thread's launches carry the programmatic-dependent-launch attribute, so each kernel's set-up
// (and the decode GEMMs' first weight tiles) overlaps the tail of the kernel before it.
struct PdlScope {
  PdlScope() { pdl_set_enabled(true); }
  ~PdlScope() { pdl_set_enabled(false); }
};

struct DecoderBase {
  uint8_t* ws = nullptr;
  int batch = 0;     // sequences of the running generation (set by prefill)
  int next_pos = 0;  // host mirror: largest position the next decode step appends at
  cudaGraphExec_t graph_exec = nullptr;
  cudaStream_t capture_stream = nullptr;
  int graph_batch = 0;
  unsigned long long graph_kernels = 0;  // kernels recorded in graph_exec (launch accounting)
  // token selection: greedy unless a temperature > 0 was set
  float sample_temperature = 0.0f, sample_top_p = 1.0f;
  int sample_top_k = 1;
  unsigned long long sample_seed = 0;

  template <typename T> T* at(size_t o) const { return reinterpret_cast<T*>(ws + o); }
};

// Device state of a generation: state[0] = position of the next token to append, state[1] = live length during that
// step, state[2] = tokens generated so far.
int set_generation_state(int* state, int pos, int len, int steps, cudaStream_t st);
// Records next_ids as the step's tokens (cur_ids, history[step]) and advances `state`; also the tensor-parallel epoch
// and, for runners with per-sequence descriptors, every sequence's descriptor to {slot, pos + len, own row, 1}.
int finish_step(const int* next_ids, int* cur_ids, int* history, int* state, int B, int max_steps, unsigned* tp_epoch,
                SeqDesc* seqs, cudaStream_t st);
// Greedy or sampled token of every row of bf16 logits (single GPU): token t of a generation draws u from (seed, t, row);
// step_dev = device count of tokens generated so far, null for the first token.
int select_tokens(const DecoderBase* m, const bf16* logits, long long ld, int rows, int vocab, const int* step_dev, float* u,
                  float* best_val, int* next, cudaStream_t st);
int set_sampling(DecoderBase* m, float temperature, int top_k, float top_p, unsigned long long seed);
void drop_graph(DecoderBase* m);
// Records `body` (one decode step for m->batch sequences) on a stream of its own / launches the recorded step.
int capture_step(DecoderBase* m, const std::function<int(cudaStream_t)>& body);
int replay_step(DecoderBase* m, int max_len, cudaStream_t st);
void destroy_base(DecoderBase* m);

}  // namespace teeny
