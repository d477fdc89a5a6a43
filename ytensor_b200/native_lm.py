"""Language models whose passes run inside the library (ytcuda_lm_*): the handle, its calls, and how checkpoint tensors are
padded to the sizes the kernels want and uploaded. A model adds its configuration and its weights (duzozen.py,
derupel.py). torch is used for device memory only."""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import _lib
from ._lib import check, lib
from .causal_lm import CausalLM

MLP_NONE, MLP_DENSE, MLP_MOE = 0, 1, 2


def up_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def up8(n: int) -> int:
    return up_to(n, 8)


class Checkpoint:
    """Tensors of a checkpoint on the device, checked against the shapes a configuration states and padded with zeros.
    weights: name -> numpy array (uint16: bf16 bits, or float32) or torch tensor; anything with __getitem__."""

    def __init__(self, weights, shapes, device):
        import torch
        self.torch, self.weights, self.shapes, self.device = torch, weights, shapes, device

    def get(self, name, dtype):
        torch = self.torch
        a = self.weights[name]
        if not isinstance(a, torch.Tensor):
            a = np.array(a)  # (an own, writable copy)
            a = torch.from_numpy(a.view(np.int16)).view(torch.bfloat16) if a.dtype == np.uint16 else torch.from_numpy(a)
        if tuple(a.shape) != self.shapes[name]:
            raise ValueError(f"{name}: shape {tuple(a.shape)} does not fit the configuration ({self.shapes[name]})")
        return a.to(self.device).to(dtype)

    def mat(self, name, rows=0, cols=0):
        """bf16, padded to at least rows x cols."""
        a = self.get(name, self.torch.bfloat16)
        return self.torch.nn.functional.pad(a, (0, max(0, cols - a.shape[1]), 0, max(0, rows - a.shape[0])))

    def vec(self, name, size=0):
        """fp32, padded to at least `size`."""
        a = self.get(name, self.torch.float32).reshape(-1)
        return self.torch.nn.functional.pad(a, (0, max(0, size - a.shape[0])))

    def heads_out(self, name, n, d, dp, cols):
        """Rows of n heads of d dimensions -> [n * dp, cols]."""
        a = self.get(name, self.torch.bfloat16)
        a = a.reshape(n, d, a.shape[1])
        return self.torch.nn.functional.pad(a, (0, cols - a.shape[2], 0, dp - d)).reshape(n * dp, cols)

    def heads_in(self, name, n, d, dp, rows):
        """Columns of n heads of d dimensions -> [rows, n * dp]."""
        a = self.get(name, self.torch.bfloat16)
        a = a.reshape(a.shape[0], n, d)
        return self.torch.nn.functional.pad(a, (0, dp - d, 0, 0, 0, rows - a.shape[0])).reshape(rows, n * dp)

    def gate_up(self, prefix, ff_p, cols):
        """Gate and up rows in turns: [2 * ff_p, cols]."""
        return self.torch.stack([self.mat(prefix + "gate", ff_p, cols), self.mat(prefix + "up", ff_p, cols)], 1).reshape(
            2 * ff_p, cols)

    def experts(self, prefix, n, ff_p, width_p):
        """All experts' [n, 2 ff, width] and [n, width, ff]."""
        up = self.torch.zeros(n, 2 * ff_p, width_p, dtype=self.torch.bfloat16, device=self.device)
        down = self.torch.zeros(n, width_p, ff_p, dtype=self.torch.bfloat16, device=self.device)
        for e in range(n):
            up[e] = self.gate_up(f"{prefix}e{e}.", ff_p, width_p)
            down[e] = self.mat(f"{prefix}e{e}.down", width_p, ff_p)
        return up, down


class NativeLM(CausalLM):
    """Device model for `batch` sequences of up to `max_tokens` tokens. dtype "bfloat16": bf16 activations, cache and
    tensor-core products, fp32 residual stream, norms, scores, state and router; "float32": everything fp32 (weights stay
    in their bf16 storage, the products are the same numbers). chunk: most tokens per sequence that run through the layers
    at once. Subclasses set `native` (the prefix of their create / set_weight entries) and implement `_create` and
    `_load`."""

    native = ""

    def __init__(self, cfg, batch: int = 1, max_tokens: int = 4096, dtype: str = "bfloat16", chunk: int = 4096):
        import torch
        self.torch = torch
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype must be bfloat16 or float32, not {dtype}")
        self.cfg, self.batch, self.dtype, self.max_tokens = cfg, batch, dtype, max_tokens
        self.L = lib()
        self.width_p = up8(cfg.width)
        config, layers = self._create(chunk, _lib.BF16 if dtype == "bfloat16" else _lib.F32)
        h = getattr(self.L, f"ytcuda_{self.native}_create")(C.byref(config), C.cast(layers, C.c_void_p))
        if not h:
            raise _lib.YtCudaInvalidArgument(_lib.INVALID_ARG, _lib.last_error())
        self.h = C.c_void_p(h)
        self._keep = []

    def _create(self, chunk: int, dtype: int):
        """-> (ctypes configuration, ctypes array of layers)."""
        raise NotImplementedError

    def _load(self, ck: Checkpoint) -> None:
        """Calls _put for every weight."""
        raise NotImplementedError

    def _put(self, name: str, layer: int, t) -> None:
        t = t.contiguous()
        self._keep.append(t)
        check(getattr(self.L, f"ytcuda_{self.native}_set_weight")(self.h, name.encode(), layer, t.data_ptr()))

    def load_weights(self, weights) -> None:
        torch = self.torch
        ck = Checkpoint(weights, self.cfg.tensor_shapes(), torch.device("cuda", torch.cuda.current_device()))
        self._put("embed", 0, ck.mat("embed", cols=self.width_p))
        self._put("head", 0, ck.mat("head", cols=self.width_p))
        self._put("norm", 0, ck.vec("final.norm", self.width_p))
        self._load(ck)

    # ---- sequences
    def reset_kv_cache(self) -> None:
        check(self.L.ytcuda_lm_reset(self.h))

    def get_kv_cache_len(self) -> int:
        return self.L.ytcuda_lm_cache_len(self.h)

    def set_decode_path(self, path: int) -> None:
        """One new token of a single sequence: 0 the CUDA graph of fused decode kernels, 1 one launch per operator."""
        check(self.L.ytcuda_lm_set_decode_path(self.h, int(path)))

    def forward_rows(self, ids, want):
        """ids int32 [batch, len] (device) -> logits fp32 [len(want), vocab] of rows `want` of the flattened input."""
        torch = self.torch
        assert ids.is_cuda and ids.dtype == torch.int32 and ids.shape[0] == self.batch and ids.is_contiguous()
        logits = torch.empty(len(want), self.cfg.vocab, dtype=torch.float32, device=ids.device)
        rows = (C.c_int32 * len(want))(*want)
        check(self.L.ytcuda_lm_forward(self.h, ids.data_ptr(), ids.shape[1], C.cast(rows, C.c_void_p), len(want),
                                       logits.data_ptr(), torch.cuda.current_stream().cuda_stream))
        return logits

    def forward(self, ids):
        n = ids.shape[1]
        return self.forward_rows(ids, [b * n + n - 1 for b in range(self.batch)])

    def forward_at(self, ids, want):
        return self.forward_rows(ids, list(want))

    def close(self) -> None:
        if getattr(self, "h", None):
            self.L.ytcuda_lm_destroy(self.h)
            self.h = None
            self._keep = []

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass
