"""What every model family shares: the forward calls and the generation loops over one C handle.

A family provides ``vocab_size``, ``causal``, ``_ensure_handle(batch, seq, total)`` (the handle, grown to
hold that many sequences, token rows and positions, cache contents kept) and ``_caches(length, batch)``
(the per-layer cache handles returned to callers); the rest of the API -- ``forward``, the last-position
and selected-row forwards, device-resident greedy generation for one prompt or a batch of unequal ones --
is here.
"""
from __future__ import annotations

from typing import Optional

import numpy as np

from . import abi, ops
from .abi import check, lib, ptr


class HandleModel:
    causal = True

    def _ensure_handle(self, batch=1, seq=1, total=1):
        raise NotImplementedError

    def _caches(self, length, batch):
        raise NotImplementedError

    def _forward_hidden(self, h, ids_d, batch, seq, past):
        raise NotImplementedError("this model family returns logits only")

    # -- forward ---------------------------------------------------------------------------
    def forward(self, input_ids: np.ndarray, return_logits: bool = True, past_kv_cache: Optional[list] = None,
                use_cache: bool = False, logits_positions: str = "all"):
        """Reference src/rotor/bitnet_model.py:190-244.  ``logits_positions='last'`` returns
        logits of the last position only, shaped [batch, 1, vocab]."""
        torch = abi.require_cuda()
        ids = np.asarray(input_ids)
        squeeze = ids.ndim == 1
        if squeeze:
            ids = ids[None, :]
        batch, seq = ids.shape
        past = 0 if past_kv_cache is None else past_kv_cache[0].length
        h = self._ensure_handle(batch, seq, past + seq)
        ids_d = ops.to_device(ids.astype(np.int64))
        if return_logits:
            allpos = logits_positions == "all"
            npos = seq if allpos else 1
            logits = torch.empty((batch, npos, self.vocab_size), dtype=torch.float32, device="cuda")
            check(lib.rotor_b200_model_forward(h.h, ptr(ids_d), batch, seq, past,
                                               abi.LOGITS_ALL if allpos else abi.LOGITS_LAST, ptr(logits), None,
                                               abi.stream()), "model_forward")
            out = logits.cpu().numpy()
        else:
            out = self._forward_hidden(h, ids_d, batch, seq, past)
        abi.device_status()
        if squeeze:
            out = out[0]
        return out, (self._caches(past + seq, batch) if use_cache else None)

    def forward_last_logits_device(self, input_ids, past_kv_cache=None):
        """Like ``forward(..., use_cache=True, logits_positions='last')`` but the logits stay on the
        device: returns (CUDA float32 [batch, vocab], caches)."""
        torch = abi.require_cuda()
        ids = np.asarray(input_ids)
        if ids.ndim == 1:
            ids = ids[None, :]
        batch, seq = ids.shape
        past = 0 if past_kv_cache is None else past_kv_cache[0].length
        h = self._ensure_handle(batch, seq, past + seq)
        ids_d = ops.to_device(ids.astype(np.int64))
        logits = torch.empty((batch, self.vocab_size), dtype=torch.float32, device="cuda")
        check(lib.rotor_b200_model_forward(h.h, ptr(ids_d), batch, seq, past, abi.LOGITS_LAST, ptr(logits), None,
                                           abi.stream()), "model_forward")
        return logits, self._caches(past + seq, batch)

    def forward_rows_device(self, input_ids, past: int, rows):
        """Runs the tokens of one sequence that follow its first ``past`` cached ones and returns CUDA
        float32 [len(rows), vocab]: the logits at the given places among these tokens (any number of
        them, none included)."""
        torch = abi.require_cuda()
        ids = np.asarray(input_ids, dtype=np.int64).reshape(1, -1)
        seq = ids.shape[1]
        want = np.asarray(rows, dtype=np.int32).reshape(-1)
        h = self._ensure_handle(1, seq, past + seq)
        ids_d = ops.to_device(ids)
        logits = torch.empty((len(want), self.vocab_size), dtype=torch.float32, device="cuda")
        check(lib.rotor_b200_model_forward_rows(h.h, ptr(ids_d), 1, seq, past, want.ctypes.data if len(want) else None,
                                                len(want), ptr(logits) if len(want) else None, abi.stream()),
              "model_forward_rows")
        return logits

    # -- device-resident greedy generation ---------------------------------------------------
    def greedy_chunks(self, prompt_ids, max_new_tokens: int, use_graph: bool = True, chunk: int = 0):
        """Generator over lists of new token ids.  The prompt is prefilled once; every later
        step is a one-token forward whose greedy pick feeds the next step on the device.
        ``chunk`` > 0 hands tokens back every ``chunk`` steps (the first list holds the token
        picked after the prompt); 0 hands everything back at the end.  Stop iterating to stop
        generating."""
        torch = abi.require_cuda()
        prompt = np.asarray(prompt_ids, dtype=np.int64).reshape(1, -1)
        n_prompt = prompt.shape[1]
        if max_new_tokens <= 0:
            return
        h = self._ensure_handle(1, n_prompt, n_prompt + max_new_tokens)
        ids_d = ops.to_device(prompt)
        first = torch.empty(1, dtype=torch.int64, device="cuda")
        stream = torch.cuda.current_stream()
        if use_graph and stream.cuda_stream == 0:
            stream = self._side_stream()   # the legacy default stream cannot be captured
        s = stream.cuda_stream
        with torch.cuda.stream(stream):
            check(lib.rotor_b200_model_forward(h.h, ptr(ids_d), 1, n_prompt, 0, abi.LOGITS_NONE, None, ptr(first), s),
                  "prefill")
            first_host = [int(first.cpu()[0])]
        remaining = max_new_tokens - 1
        if chunk > 0 or remaining == 0:
            yield first_host
            first_host = []
        if remaining > 0:
            check(lib.rotor_b200_model_decode_begin(h.h, ptr(first), 1, n_prompt, s), "decode_begin")
            step = chunk if chunk > 0 else remaining
            buf = np.empty(step, dtype=np.int64)
            # The steps feed one another on the device, so the next chunk is launched BEFORE the current
            # one's tokens are read: the read goes through a second stream that waits for the chunk's own
            # event, and the device never idles for the host round trip.  A consumer that stops iterating
            # (EOS) leaves at most one chunk of surplus steps, which the close below waits out.
            copier = self._copy_stream()

            def launch(first_step):
                n = min(step, remaining - first_step)
                with torch.cuda.stream(stream):
                    check(lib.rotor_b200_model_decode_steps(h.h, n, int(use_graph), s), "decode_steps")
                    done_ev = torch.cuda.Event()
                    done_ev.record(stream)
                return first_step, n, done_ev

            try:
                queue = [launch(0)]
                launched = queue[0][1]
                while queue:
                    start, n, done_ev = queue.pop(0)
                    if launched < remaining:
                        queue.append(launch(launched))
                        launched += queue[-1][1]
                    copier.wait_event(done_ev)
                    check(lib.rotor_b200_model_read_tokens(h.h, start, n, buf.ctypes.data, copier.cuda_stream),
                          "read_tokens")
                    yield first_host + [int(t) for t in buf[:n]]
                    first_host = []
            finally:
                stream.synchronize()   # nothing of this generation is in flight when the handle is used again
        abi.device_status()

    def generate_greedy(self, prompt_ids, max_new_tokens: int, use_graph: bool = True, chunk: int = 0):
        """All new token ids of a device-resident greedy generation."""
        out = []
        for new in self.greedy_chunks(prompt_ids, max_new_tokens, use_graph, chunk):
            out += new
        return out

    def generate_greedy_batch(self, prompt_ids, max_new_tokens: int, use_graph: bool = True):
        """Device-resident greedy generation for a batch of prompts: one prefill, then every step
        advances all sequences at once.  ``prompt_ids`` is [batch, prompt_len] or a list of
        prompts of different lengths; those are right-padded for the prefill (a causal model
        never attends to the padding behind a token) and every sequence then continues from
        its own length.  Returns int64 [batch, max_new_tokens], row b holding what a
        single-prompt generation from prompt b gives."""
        torch = abi.require_cuda()
        rows = [np.asarray(p, dtype=np.int64).reshape(-1) for p in prompt_ids]
        batch = len(rows)
        if batch == 0:
            return np.zeros((0, max(max_new_tokens, 0)), dtype=np.int64)
        lens = np.array([len(r) for r in rows], dtype=np.int32)
        if lens.min() < 1:
            raise ValueError("every prompt needs at least one token")
        n_prompt = int(lens.max())
        ragged = bool((lens != n_prompt).any())
        if ragged and not self.causal:
            raise ValueError("prompts of different lengths need a causal model")
        prompts = np.zeros((batch, n_prompt), dtype=np.int64)
        for b, r in enumerate(rows):
            prompts[b, :len(r)] = r
        if max_new_tokens <= 0:
            return np.zeros((batch, 0), dtype=np.int64)
        h = self._ensure_handle(batch, n_prompt, n_prompt + max_new_tokens)
        ids_d = ops.to_device(prompts)
        first = torch.empty(batch, dtype=torch.int64, device="cuda")
        stream = torch.cuda.current_stream()
        if use_graph and stream.cuda_stream == 0:
            stream = self._side_stream()
        s = stream.cuda_stream
        out = np.empty((batch, max_new_tokens), dtype=np.int64)
        with torch.cuda.stream(stream):
            if ragged:
                check(lib.rotor_b200_model_forward_ragged(h.h, ptr(ids_d), batch, n_prompt, lens.ctypes.data,
                                                          abi.LOGITS_NONE, None, ptr(first), s), "prefill")
            else:
                check(lib.rotor_b200_model_forward(h.h, ptr(ids_d), batch, n_prompt, 0, abi.LOGITS_NONE, None,
                                                   ptr(first), s), "prefill")
            out[:, 0] = first.cpu().numpy()
            remaining = max_new_tokens - 1
            if remaining > 0:
                if ragged:
                    check(lib.rotor_b200_model_decode_begin_ragged(h.h, ptr(first), batch, lens.ctypes.data, s),
                          "decode_begin")
                else:
                    check(lib.rotor_b200_model_decode_begin(h.h, ptr(first), batch, n_prompt, s), "decode_begin")
                check(lib.rotor_b200_model_decode_steps(h.h, remaining, int(use_graph), s), "decode_steps")
                buf = np.empty((remaining, batch), dtype=np.int64)   # the token log is [step][sequence]
                check(lib.rotor_b200_model_read_tokens(h.h, 0, remaining, buf.ctypes.data, s), "read_tokens")
                out[:, 1:] = buf.T
        abi.device_status()
        return out

    def _copy_stream(self):
        torch = abi.require_cuda()
        if getattr(self, "_copier", None) is None:
            self._copier = torch.cuda.Stream()
        return self._copier

    def _side_stream(self):
        torch = abi.require_cuda()
        if getattr(self, "_stream", None) is None:
            self._stream = torch.cuda.Stream()
        self._stream.wait_stream(torch.cuda.current_stream())
        return self._stream
