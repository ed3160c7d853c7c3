// Generation state, token selection and graph capture shared by the model runners (decoder_base.h).
//
// capture_step / replay_step stand where the reference's executor has capture_graph and CudaGraphModel::run
// (drivers/teeny-cuda/src/model/mod.rs:1245, 1799).
#include "decoder_base.h"

namespace teeny {

namespace {

__global__ void finish_step_kernel(const int* __restrict__ next_ids, int* __restrict__ cur_ids,
                                   int* __restrict__ history, int* __restrict__ state, int B, int max_steps,
                                   unsigned* __restrict__ tp_epoch, SeqDesc* __restrict__ seqs) {
  pdl_wait();
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  const int step = state[2];
  if (b < B) {
    const int id = next_ids[b];
    cur_ids[b] = id;
    if (step < max_steps) history[static_cast<size_t>(step) * B + b] = id;
    if (seqs) {
      SeqDesc s = seqs[b];
      s.pos += s.len;
      s.row0 = b;
      s.len = 1;
      seqs[b] = s;
    }
  }
  __syncthreads();  // single block: every thread has read `step`
  if (b == 0) {
    state[0] += 1;
    state[1] += 1;
    state[2] = step + 1;
    if (tp_epoch) *tp_epoch += 1u;  // the pushes of the next step carry new stamps
  }
}

__global__ void set_state_kernel(int* state, int pos, int len, int steps) {
  pdl_wait();
  state[0] = pos;
  state[1] = len;
  state[2] = steps;
}

}  // namespace

int set_generation_state(int* state, int pos, int len, int steps, cudaStream_t st) {
  return launch_kernel(set_state_kernel, dim3(1), dim3(1), 0, st, 1, state, pos, len, steps);
}

int finish_step(const int* next_ids, int* cur_ids, int* history, int* state, int B, int max_steps, unsigned* tp_epoch,
                SeqDesc* seqs, cudaStream_t st) {
  if (B <= 0 || B > 1024) return TEENY_ERR_BAD_ARG;
  launch_kernel(finish_step_kernel, dim3(1), dim3(1024), 0, st, 1, next_ids, cur_ids, history, state, B, max_steps, tp_epoch,
                seqs);
  return static_cast<int>(cudaGetLastError());
}

int select_tokens(const DecoderBase* m, const bf16* logits, long long ld, int rows, int vocab, const int* step_dev, float* u,
                  float* best_val, int* next, cudaStream_t st) {
  if (m->sample_temperature > 0.0f) {
    TEENY_TRY(sampling_uniform(m->sample_seed, 0, step_dev, u, rows, st));
    return sample_top_k_top_p_bf16(logits, ld, rows, vocab, m->sample_temperature, m->sample_top_k, m->sample_top_p, u, next,
                                   nullptr, st);
  }
  return argmax_bf16(logits, ld, best_val, next, rows, vocab, 0, st);
}

void drop_graph(DecoderBase* m) {
  if (m->graph_exec) cudaGraphExecDestroy(m->graph_exec);
  m->graph_exec = nullptr;
}

int set_sampling(DecoderBase* m, float temperature, int top_k, float top_p, unsigned long long seed) {
  if (temperature > 0.0f) {
    if (top_k < 1 || top_k > 1024 || !(top_p > 0.0f) || top_p > 1.0f) return TEENY_ERR_BAD_ARG;
    m->sample_temperature = temperature; m->sample_top_k = top_k; m->sample_top_p = top_p; m->sample_seed = seed;
  } else {
    m->sample_temperature = 0.0f;
  }
  drop_graph(m);  // the captured step has the old selection baked in
  return TEENY_OK;
}

int capture_step(DecoderBase* m, const std::function<int(cudaStream_t)>& body) {
  if (m->batch <= 0) return TEENY_ERR_BAD_ARG;
  drop_graph(m);
  cudaError_t e = cudaSuccess;
  // recording needs a non-default stream of its own; the graph is replayed on the caller's stream
  if (!m->capture_stream) e = cudaStreamCreateWithFlags(&m->capture_stream, cudaStreamNonBlocking);
  if (e != cudaSuccess) return static_cast<int>(e);
  e = cudaStreamBeginCapture(m->capture_stream, cudaStreamCaptureModeThreadLocal);
  if (e != cudaSuccess) return static_cast<int>(e);
  const unsigned long long launches_before = launches_so_far();
  const int rc = body(m->capture_stream);
  m->graph_kernels = launches_so_far() - launches_before;
  cudaGraph_t graph = nullptr;
  e = cudaStreamEndCapture(m->capture_stream, &graph);
  if (rc != 0) {
    if (graph) cudaGraphDestroy(graph);
    return rc;
  }
  if (e != cudaSuccess) return static_cast<int>(e);
  e = cudaGraphInstantiate(&m->graph_exec, graph, 0);
  cudaGraphDestroy(graph);
  if (e != cudaSuccess) {
    m->graph_exec = nullptr;
    return static_cast<int>(e);
  }
  m->graph_batch = m->batch;
  return 0;
}

int replay_step(DecoderBase* m, int max_len, cudaStream_t st) {
  if (!m->graph_exec || m->graph_batch != m->batch) return TEENY_ERR_BAD_ARG;
  if (m->next_pos >= max_len) return TEENY_ERR_BAD_ARG;  // cache full
  const int rc = static_cast<int>(cudaGraphLaunch(m->graph_exec, st));
  if (rc == 0) {
    ++m->next_pos;
    count_launches(m->graph_kernels);
  }
  return rc;
}

void destroy_base(DecoderBase* m) {
  drop_graph(m);
  if (m->capture_stream) cudaStreamDestroy(m->capture_stream);
}

}  // namespace teeny
