"""What the models of this package have in common: steps from host ids, device-resident decoding,
sampling from the last logits, and the generate loop.  A subclass binds its C entry points in the
``_step`` / ``_step_device`` / ``_decode`` / ``_logits_ptr`` hooks."""
from __future__ import annotations

from typing import Optional

import numpy as np

from .runtime import B200Buffer, B200Runtime


class Model:
    rt: B200Runtime
    batch: int
    max_seq_len: int
    vocab_size: int

    # -- hooks --
    def _step(self, tokens: np.ndarray, n: int) -> np.ndarray:
        raise NotImplementedError

    def _step_device(self, ids: B200Buffer, s: int, n: int, out: B200Buffer) -> None:
        raise NotImplementedError

    def _decode(self, first_ids: B200Buffer, n: int, steps: int, out: Optional[B200Buffer]) -> None:
        raise NotImplementedError

    def _logits_ptr(self) -> int:
        raise NotImplementedError

    # -- one step from host ids: the call a token loop makes --
    def forward(self, x, s: Optional[int] = None, n: int = 0) -> np.ndarray:
        """x: [batch, s] token ids (any numeric dtype) at positions n ..; returns int64 [batch]: argmax of
        the logits at the last position."""
        tok = np.asarray(x).reshape(self.batch, -1)
        if s is not None and int(s) != tok.shape[1]:
            raise ValueError("forward: s does not match x")
        return self._step(tok, int(n))

    # -- device-resident variants (ids never leave HBM) --
    def forward_device(self, ids: B200Buffer, s: int, n: int, out: B200Buffer) -> None:
        self._step_device(ids, int(s), int(n), out)

    def decode_device(self, first_ids: np.ndarray, start_pos: int, steps: int) -> np.ndarray:
        """Greedy decode ``steps`` tokens with ids and position staying on the GPU (one C call; the
        step is replayed from a CUDA graph); returns [batch, steps]."""
        ids0 = self.rt.transfer_from_array(np.ascontiguousarray(first_ids, dtype=np.int64).reshape(self.batch))
        hist = self.rt.open_buffer((steps, self.batch), np.int64)
        self.decode_device_buffers(ids0, start_pos, steps, hist)
        out = hist.numpy().T.copy()
        hist.close()
        ids0.close()
        return out

    def decode_device_buffers(self, first_ids: B200Buffer, start_pos: int, steps: int, out: Optional[B200Buffer] = None) -> None:
        """Asynchronous form of :meth:`decode_device` on device buffers (``out``: [steps, batch] int64)."""
        self._decode(first_ids, int(start_pos), int(steps), out)

    def _logits_buffer(self) -> B200Buffer:
        return B200Buffer(self.rt, self._logits_ptr(), (self.batch, self.vocab_size), np.float32, owned=False)

    def logits(self) -> np.ndarray:
        """[batch, vocab] fp32 logits of the last step."""
        return self._logits_buffer().numpy()

    def sample(self, uniform, temperature: float = 1.0, top_k: int = 0) -> np.ndarray:
        """[batch] int64 ids drawn from the last step's logits (they stay on the device)."""
        ids = self.rt.sample(self._logits_buffer(), uniform, temperature, top_k)
        out = ids.numpy()
        ids.close()
        return out


def generate(model: Model, prompt_ids, max_length: int = 100, temperature: float = 0.0, top_k: int = 0, seed: int = 0) -> np.ndarray:
    """`gpt2-generate` (apps/gpt2/gpt2.lisp:97-113) on token ids: the first call feeds the whole
    prompt at start position 0, each later call one token; every call's argmax is appended.
    Returns [batch, prompt_len + max_length] int64.  With ``temperature`` > 0 the next id is drawn
    on the device from the step's logits instead (temperature / top-k sampling, seeded; beyond the
    reference, whose loop is greedy)."""
    tokens = np.ascontiguousarray(prompt_ids, dtype=np.int64).reshape(model.batch, -1)
    start_pos = 0
    rng = np.random.Generator(np.random.PCG64(seed))
    for _ in range(max_length):
        in_tokens = tokens[:, start_pos:]
        out = model.forward(in_tokens, in_tokens.shape[1], start_pos)
        if temperature > 0.0:
            out = model.sample(rng.random(model.batch, dtype=np.float32), temperature, top_k)
        start_pos = tokens.shape[1]
        tokens = np.concatenate([tokens, out.reshape(-1, 1)], axis=1)
    return tokens
