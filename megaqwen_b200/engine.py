"""What every decoder object of the package shares, whatever its model: the
position, the sticky device status, single steps replayed from a CUDA graph,
device-resident greedy chains, the chunked greedy loop with its EOS scan, and
the checks of prefill lengths.  A decoder adds its weights, its cache or state
and two launches: one decode step and one prefill.

Names, state semantics and error texts are those of the reference's pybind
classes (csrc/megakernel/bindings_decode.cpp:80-280,
csrc/megakernel/bindings_prefill.cpp:731-1349).
"""
from __future__ import annotations

import torch

from . import _lib


def _ptr(t: torch.Tensor) -> int:
    return t.data_ptr()


class DecodeEngine:
    """Base of the decoders.  A subclass calls ``_init_engine`` and provides

    ``_launch(in_ptr, out_ptr, pos_ptr, logits_ptr, chained)``  one decode step (counted in ``launches``),
    ``step_launches``                                           kernels of one step,
    ``prefill_step / prefill_append / prefill_step_logits``     prompts and portions of prompts,
    ``reset``                                                   position and state,

    and, where it keeps more than a cache: ``_before_decode`` / ``_after_decode`` around decode
    launches (never captured in a graph) and ``_chain_persistent``.
    """

    def _init_engine(self, lib, device, vocab_size, max_seq_len, max_prefill_len) -> None:
        self._lib = lib
        self.device = device
        self.vocab_size_ = int(vocab_size)
        self.max_seq_len_ = int(max_seq_len)
        self.max_prefill_len_ = int(max_prefill_len)
        i32 = torch.int32
        # [0] = output token of single steps, [1] = sticky status word
        self._scalars = torch.zeros(4, dtype=i32, device=device)
        self._in_token = torch.zeros(1, dtype=i32, device=device)
        self._pos_dev = torch.zeros(1, dtype=i32, device=device)
        self._logits = None
        self._chain_cap = 0
        self._chain_tokens = None
        self._chain_pos = None
        self._graphs = {}
        self.position_ = 0
        self.use_pdl = True
        self.use_step_graph = True  # decode_step replays a captured one-step graph instead of launching every kernel
        self._step_graph = None
        self._step_graph_pdl = None
        self.launches = 0          # kernels launched through the C ABI by this object

    # ------------------------------------------------------------------ hooks
    def _before_decode(self) -> None:
        pass

    def _after_decode(self) -> None:
        pass

    def _chain_persistent(self, tokens: torch.Tensor, num_steps: int) -> bool:
        """Run the chain in one persistent launch if the decoder has one for it."""
        return False

    # ------------------------------------------------------------------ helpers
    def _stream(self) -> int:
        return torch.cuda.current_stream(self.device).cuda_stream

    def _check_status(self, status: int) -> None:
        if status:
            self._scalars[1] = 0
            what = []
            if status & _lib.MQ_STATUS_WAIT_TIMEOUT:
                what.append("a bounded device-side wait expired")
            if status & _lib.MQ_STATUS_BAD_POSITION:
                what.append("position outside the KV cache")
            if status & _lib.MQ_STATUS_BAD_TOKEN:
                what.append("token id outside the vocabulary")
            raise RuntimeError("megaqwen_b200 device status: " + ", ".join(what))

    def check_status(self) -> None:
        """Read the sticky device status word (one 4-byte copy) and raise if set."""
        self._check_status(int(self._scalars[1].item()))

    def _ensure_chain(self, n: int) -> None:
        if n > self._chain_cap:
            cap = max(n, 64)
            self._chain_tokens = torch.zeros(cap + 1, dtype=torch.int32, device=self.device)
            self._chain_pos = torch.zeros(cap, dtype=torch.int32, device=self.device)
            self._chain_cap = cap
            self._graphs = {}

    def _logits_buffer(self) -> torch.Tensor:
        if self._logits is None:
            self._logits = torch.empty(self.vocab_size_, dtype=torch.float32, device=self.device)
        return self._logits

    # ------------------------------------------------------------------ reference API
    def position(self) -> int:
        return self.position_

    def max_prefill_len(self) -> int:
        return self.max_prefill_len_

    def _single(self, input_token_id: int, logits_ptr) -> int:
        if self.position_ >= self.max_seq_len_:
            raise RuntimeError("decode_step would exceed max_seq_len")
        with torch.cuda.device(self.device):
            # scalar fills carry the value as a kernel argument: no host buffer to race on
            self._in_token.fill_(int(input_token_id))
            self._pos_dev.fill_(self.position_)
            self._before_decode()
            if logits_ptr is None and self.use_step_graph:
                self._replay_step_graph()
            else:
                self._launch(_ptr(self._in_token), _ptr(self._scalars), _ptr(self._pos_dev), logits_ptr, False)
            self.position_ += 1
            self._after_decode()
            tok, status = self._scalars[:2].tolist()
        self._check_status(status)
        return tok

    def _replay_step_graph(self) -> None:
        """One decode step (token and position in device scalars) captured once and replayed:
        the host cost of a step is one graph launch instead of one per kernel."""
        if self._step_graph is None or self._step_graph_pdl != self.use_pdl:
            g = torch.cuda.CUDAGraph()
            launches0 = self.launches
            s = torch.cuda.Stream(device=self.device)
            s.wait_stream(torch.cuda.current_stream(self.device))
            with torch.cuda.stream(s):
                with torch.cuda.graph(g, stream=s):
                    self._launch(_ptr(self._in_token), _ptr(self._scalars), _ptr(self._pos_dev), None, False)
            torch.cuda.current_stream(self.device).wait_stream(s)
            self.launches = launches0
            self._step_graph, self._step_graph_pdl = g, self.use_pdl
        self._step_graph.replay()
        self.launches += self.step_launches

    def decode_step(self, input_token_id: int) -> int:
        return self._single(input_token_id, None)

    def decode_step_logits(self, input_token_id: int):
        """One step that also returns the bf16-rounded logits as fp32 [vocab]
        (reference: launch_ldg_decode_with_logits, chat.py:241-314)."""
        tok = self._single(input_token_id, _ptr(self._logits_buffer()))
        return tok, self._logits.clone()

    def _chain(self, first_token, num_steps: int, use_graph: bool, what: str = "decode_steps") -> torch.Tensor:
        """Device-resident chain token[i] -> token[i+1]; returns the view of the
        num_steps generated tokens (cuda int32).  No host synchronisation."""
        if num_steps <= 0:
            return torch.empty(0, dtype=torch.int32, device=self.device)
        # the reference's bound (bindings_prefill.cpp:1049-1051, 1092): the last cache row stays unused
        if self.position_ + num_steps >= self.max_seq_len_:
            raise RuntimeError(f"{what} would exceed max_seq_len")
        with torch.cuda.device(self.device):
            self._ensure_chain(num_steps)
            self._before_decode()
            tk, ps = self._chain_tokens, self._chain_pos
            if torch.is_tensor(first_token):
                tk[0:1].copy_(first_token.reshape(1).to(torch.int32), non_blocking=True)
            else:
                tk[0:1].fill_(int(first_token))
            if use_graph and self._chain_persistent(tk, num_steps):
                self.position_ += num_steps
                return tk[1:num_steps + 1]
            _lib.check(self._lib.mq_launch_fill_iota(_ptr(ps), self.position_, num_steps, self._stream()), "mq_launch_fill_iota")
            self.launches += 1
            if use_graph:
                self._replay_graph(num_steps)
            else:
                for i in range(num_steps):
                    self._launch(_ptr(tk) + 4 * i, _ptr(tk) + 4 * (i + 1), _ptr(ps) + 4 * i, None, i > 0)
            self.position_ += num_steps
            self._after_decode()
            return tk[1:num_steps + 1]

    def _replay_graph(self, num_steps: int) -> None:
        key = (num_steps, self.use_pdl)      # the PDL attribute is baked into the captured launches
        g = self._graphs.get(key)
        tk, ps = self._chain_tokens, self._chain_pos
        if g is None:
            g = torch.cuda.CUDAGraph()
            launches0 = self.launches
            # capture on a side stream as torch requires; the chain reads tokens[0]
            # and positions[] which are refreshed before every replay
            s = torch.cuda.Stream(device=self.device)
            s.wait_stream(torch.cuda.current_stream(self.device))
            with torch.cuda.stream(s):
                with torch.cuda.graph(g, stream=s):
                    for i in range(num_steps):
                        self._launch(_ptr(tk) + 4 * i, _ptr(tk) + 4 * (i + 1), _ptr(ps) + 4 * i, None, i > 0)
            torch.cuda.current_stream(self.device).wait_stream(s)
            self.launches = launches0
            self._graphs[key] = g
        g.replay()
        self.launches += num_steps * self.step_launches

    def decode_steps_cuda(self, first_token, num_steps: int) -> torch.Tensor:
        return self._chain(first_token, num_steps, False).clone()

    def decode_steps_cuda_graph(self, first_token, num_steps: int) -> torch.Tensor:
        """Per-phase kernels replayed from a CUDA graph (reference:
        decode_steps_cuda_graph, bindings_prefill.cpp:1082-1150)."""
        return self._chain(first_token, num_steps, True, "decode_steps_cuda_graph").clone()

    def decode_steps(self, first_token_id: int, num_steps: int) -> torch.Tensor:
        out = self._chain(first_token_id, num_steps, True)
        host = torch.cat([out, self._scalars[1:2]]).cpu()
        self._check_status(int(host[-1]))
        return host[:-1]

    def decode_greedy_cuda(self, first_token, max_new_tokens: int, eos_ids, chunk: int = 32):
        """Greedy loop with tokens kept on the device; the EOS scan and one 4-byte
        read happen once per chunk.  Same contract as the reference
        (bindings_prefill.cpp:1159-1349): the result holds the CONSUMED tokens,
        i.e. per chunk ``[next_token] + generated[:-1]``, so ``out[0]`` is
        ``first_token`` and the last token a chunk generated is carried into the
        next chunk instead of being returned; EOS is searched in
        ``generated[:-1]`` of each chunk and excluded from the result;
        ``position()`` advances by whole chunks (the cache rows past an EOS were
        computed and stay).  Returns (tokens cuda int32[len], len, stop_reason)
        with stop_reason 0 = max_new_tokens, 1 = EOS."""
        max_new = int(max_new_tokens)
        if max_new <= 0:
            return torch.empty(0, dtype=torch.int32, device=self.device), 0, 0
        if chunk <= 0:
            chunk = 32
        if eos_ids is None or len(eos_ids) == 0:
            raise RuntimeError("eos_ids must be a non-empty int32 tensor")
        eos = torch.as_tensor(eos_ids).to(device=self.device, dtype=torch.int32).contiguous()
        out = torch.empty(max_new, dtype=torch.int32, device=self.device)
        hit = torch.empty(1, dtype=torch.int32, device=self.device)
        gen_len, stop_reason, cur = 0, 0, first_token
        while gen_len < max_new:
            steps = min(chunk, max_new - gen_len)
            tail = self._chain(cur, steps, steps == chunk)          # view of tokens[1 .. steps]
            tokens = self._chain_tokens                             # tokens[0] = consumed token of this chunk
            out[gen_len:gen_len + steps].copy_(tokens[:steps])
            stop_pos = -1
            if steps > 1:
                hit.fill_(steps - 1)
                _lib.check(self._lib.mq_launch_find_first_eos(_ptr(tokens) + 4, steps - 1, _ptr(eos), eos.numel(), _ptr(hit),
                                                              self._stream()), "mq_launch_find_first_eos")
                self.launches += 1
                idx = int(hit.item())
                if idx < steps - 1:
                    stop_pos = idx + 1          # tokens kept from this chunk; the EOS itself is dropped
            if stop_pos >= 0:
                gen_len += stop_pos
                stop_reason = 1
                break
            gen_len += steps
            cur = tail[steps - 1:steps].clone()
        self.check_status()
        return out[:gen_len], gen_len, stop_reason

    def _check_prefill(self, ids: torch.Tensor, pos0: int) -> int:
        """The reference's checks and texts (bindings_prefill.cpp:731-739); the ASR caller
        matches on them (megaqwen/qwen3_asr_megakernel.py:767-773)."""
        n = int(ids.numel())
        if n > self.max_prefill_len_:
            raise RuntimeError("Prefill sequence length exceeds maximum")
        if n == 0:
            raise RuntimeError("Empty input sequence")
        if pos0 + n > self.max_seq_len_:
            raise RuntimeError("Prefill sequence length exceeds maximum (max_seq_len)")
        return n

    def step_logits(self, input_ids, want):
        """Feed the next tokens of the sequence (a prompt, a portion of one, or a single token) and
        return the fp32 logits [len(want), vocab] after the tokens at the places ``want`` (ascending).
        Decoders that can read several rows of one prefill override this."""
        ids = [int(t) for t in input_ids]
        rows, at = [], 0
        for end in list(want) + ([len(ids) - 1] if not want or want[-1] != len(ids) - 1 else []):
            part = ids[at:end + 1]
            lg = self.decode_step_logits(part[0])[1] if len(part) == 1 else self.prefill_step_logits(part, append=True)[1]
            if end in want:
                rows.append(lg)
            at = end + 1
        return torch.stack(rows) if rows else torch.empty((0, self.vocab_size_), dtype=torch.float32, device=self.device)
