"""What every language model of the library shares: greedy and sampled generation, logits at chosen places of an input
and the device-status check. A model supplies forward / reset_kv_cache and, where it can, forward_at."""
from __future__ import annotations

import numpy as np

from . import _lib
from ._lib import lib


class CausalLM:
    """Subclasses set `torch`, `batch` (sequences, all of one length) and implement `forward` and `reset_kv_cache`."""

    batch: int = 1
    can_sample = True

    def forward(self, ids):
        """ids int32 [batch, len] on the device, appended to the sequences -> fp32 logits [batch, vocab] of the last
        position."""
        raise NotImplementedError

    def reset_kv_cache(self) -> None:
        raise NotImplementedError

    def get_kv_cache_len(self) -> int:
        raise NotImplementedError

    def forward_at(self, ids, want):
        """ids int32 [1, len] -> fp32 logits [len(want), vocab] at the ascending places `want` of the input. A model
        that computes the last position only gets the input in pieces that end at the wanted places."""
        torch = self.torch
        out, done = [], 0
        for w in want:
            out.append(self.forward(ids[:, done:w + 1].contiguous()).reshape(1, -1))
            done = w + 1
        if done < ids.shape[1]:
            self.forward(ids[:, done:].contiguous())
        return torch.cat(out) if out else None

    def argmax(self, logits):
        """Greedy token (int32) and its logit per row; the first maximum wins, as a host argmax over the row would."""
        from . import api
        val, idx = api.max(logits, -1)
        return idx.reshape(-1).to(self.torch.int32), val.reshape(-1)

    def check_status(self) -> None:
        """Reads the device status word (synchronises the stream). A bounded wait that ran out - under tensor
        parallelism: a peer that never arrived at an exchange - raises; the KV caches are then half written and the
        group has to call recover() before the next forward."""
        st = lib().ytcuda_device_status(self.torch.cuda.current_stream().cuda_stream)
        if st != _lib.OK:
            raise _lib.YtCudaError(st, _lib.last_error() or "a bounded device-side wait ran out")

    def generate_greedy(self, prompt_ids, steps: int):
        """prompt_ids int32 [batch, len] (device). Returns int32 [batch, steps] greedy tokens. The device status is
        checked once at the end, so that a step kernel that gave up on a peer raises instead of yielding tokens."""
        torch = self.torch
        out = torch.empty(self.batch, steps, dtype=torch.int32, device=prompt_ids.device)
        logits = self.forward(prompt_ids)
        for s in range(steps):
            tok, _ = self.argmax(logits)
            out[:, s] = tok
            if s + 1 < steps:
                logits = self.forward(tok.reshape(self.batch, 1).contiguous())
        self.check_status()
        return out

    def generate_topk(self, prompt_ids, steps: int, k: int = 20, seed: int = 42):
        """Sampled generation as Qwen3ForCausalLM::generate does it (reference qwen3.cpp:459-516): after every
        forward the next token is drawn among the k most probable ones. The uniform numbers come from a host
        generator (numpy's MT19937 seeded with `seed`; the reference's std::uniform_real_distribution consumes its
        std::mt19937 differently, so the streams are not the same). Single GPU. Returns int32 [batch, steps]."""
        from . import api
        torch = self.torch
        assert self.can_sample, "sampling needs the whole vocabulary on one GPU"
        rng = np.random.Generator(np.random.MT19937(seed))
        out = torch.empty(self.batch, steps, dtype=torch.int32, device=prompt_ids.device)
        logits = self.forward(prompt_ids)
        for s in range(steps):
            u = torch.from_numpy(rng.random(self.batch, dtype=np.float32)).to(prompt_ids.device)
            _, _, tok = api.topk_sample(logits, k, u)
            out[:, s] = tok
            if s + 1 < steps:
                logits = self.forward(tok.reshape(self.batch, 1).contiguous())
        return out
