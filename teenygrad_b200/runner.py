"""What the model runners share on the host side: the C handle over one device workspace, buffer views, weight upload,
token selection and the decode loop with CUDA-graph replay.  A runner class sets ``PREFIX`` (its C entry points are
``{PREFIX}_decode`` and so on) and adds the parts that depend on the model: weights, prefill."""
import ctypes as C

import torch

from ._lib import lib, check

BUF_LOGITS, BUF_NEXT_IDS, BUF_HISTORY, BUF_STATE = range(4)  # the same numbers in every runner's header


def stream():
    return C.c_void_p(torch.cuda.current_stream().cuda_stream)


class DecoderRunner:
    PREFIX = None
    _h = None

    def _call(self, name, *args):
        name = f"{self.PREFIX}_{name}"
        check(getattr(lib, name)(*args), name)

    def _init_runner(self, nbytes, max_len, max_new_tokens, device):
        self.device = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
        self.max_len, self.max_new_tokens = max_len, max_new_tokens
        self.workspace = torch.empty(nbytes, dtype=torch.uint8, device=self.device)
        self._weights = []  # keeps device tensors alive
        self._captured = False
        self.batch = 0

    def __del__(self):
        h = self._h
        if h and lib is not None:  # at interpreter shutdown the module globals may already be gone
            getattr(lib, f"{self.PREFIX}_destroy")(h)
            self._h = None

    def _upload(self, t):
        """Device address of a contiguous copy of ``t`` that lives as long as the runner."""
        t = t.to(self.device).contiguous()
        self._weights.append(t)
        return C.c_void_p(t.data_ptr())

    def _set_batch(self, n):
        if n != self.batch:
            self._captured = False  # the recorded decode step has the batch baked in; everything else is a fixed address
        self.batch = n

    # ---- buffers ----
    def _view(self, which, shape, dtype):
        ptr = getattr(lib, f"{self.PREFIX}_buffer")(self._h, which)
        off = ptr - self.workspace.data_ptr()
        n = int(torch.tensor(shape).prod()) * torch.empty(0, dtype=dtype).element_size()
        return self.workspace[off:off + n].view(dtype).view(*shape)

    def next_ids(self):
        return self._view(BUF_NEXT_IDS, (self.batch,), torch.int32)

    def history(self):
        return self._view(BUF_HISTORY, (self.max_new_tokens, self.batch), torch.int32)

    def state(self):
        return self._view(BUF_STATE, (3,), torch.int32)

    # ---- execution ----
    @staticmethod
    def device_error():
        """Synchronises and returns (and clears) the device error word: 0 unless a kernel gave up on a wait."""
        return lib.teeny_device_error(1)

    def set_sampling(self, temperature, top_k=50, top_p=1.0, seed=0):
        """Token selection for the following generations: ``temperature <= 0`` is greedy; otherwise temperature /
        top-k / top-p sampling with u for token t and row r a stateless hash of (seed, t, r)."""
        self._call("set_sampling", self._h, float(temperature), int(top_k), float(top_p), int(seed))
        self._captured = False

    def decode_step(self, graph=False):
        if graph:
            if not self._captured:
                self._call("capture_decode", self._h, stream())
                self._captured = True
            self._call("decode_replay", self._h, stream())
        else:
            self._call("decode", self._h, stream())

    def _decode_loop(self, max_new_tokens, use_graph):
        """The tokens after the first (which the prefill picked): int32 [batch, max_new_tokens] on the device, no host
        sync inside."""
        for _ in range(max_new_tokens - 1):
            self.decode_step(graph=use_graph)
        return self.history()[:max_new_tokens].t()
