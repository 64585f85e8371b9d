"""A batch of sequences that live in one cache and are fed piece by piece: the step function under autoregressive
generation and the trace runner, for every base model of the registry.

Row b of the batch holds kv_len[b] tokens from cache slot begin[b] on.  extend() runs the next tokens of any rows, in
portions of any size; decode() runs one token of every row and is what a CUDA graph replays; release() gives a row back.
"""
import os
from typing import List, Optional, Sequence

import numpy as np
import torch

from . import _lib, modeling_drafter


class Session:
    def __init__(self, llm, batch: int, max_length: int, begin: Optional[Sequence[int]] = None):
        self.llm, self.batch, self.max_length = llm, batch, max_length
        dev = llm.device
        i32 = dict(dtype=torch.int32, device=dev)
        self.cache = llm.new_cache(batch, max_length)
        self.first_slot: List[int] = [0] * batch if begin is None else [int(v) for v in begin]
        self.lengths: List[int] = [0] * batch  # host copy of kv_len, up to date except inside a decode loop
        self.begin = torch.tensor(self.first_slot, **i32)
        self.kv_len = torch.zeros(batch, **i32)
        self.status = torch.zeros(1, **i32)
        # one-token steps: every buffer has a fixed address
        self.base_len = torch.zeros(batch, **i32)
        self.slot = torch.zeros(batch, **i32)
        self.rows = torch.arange(batch, **i32)
        self.row_start = torch.arange(batch + 1, **i32)
        self.next_tok = torch.zeros(batch, dtype=torch.int64, device=dev)
        self.last_hidden = torch.zeros(batch, llm.config.hidden_size, dtype=llm.dtype, device=dev)
        self._sparse = None
        self._u: Optional[torch.Tensor] = None

    # ------------------------------------------------------------------------------------------ any portions
    @torch.inference_mode()
    def extend(self, tok_ids: torch.Tensor, counts: Sequence[int]) -> torch.Tensor:
        """Runs counts[b] further tokens of every row b; tok_ids holds them back to back, row after row (int64).  Returns
        the final hidden states of these tokens (a workspace buffer: valid until the next step)."""
        llm, B = self.llm, self.batch
        cnt = np.asarray(counts, dtype=np.int32)
        assert cnt.shape == (B,) and (cnt >= 0).all() and int(cnt.sum()) == tok_ids.numel() > 0
        M = tok_ids.numel()
        base = np.asarray(self.lengths, dtype=np.int32)
        first = np.asarray(self.first_slot, dtype=np.int32)
        if (first + base + cnt > self.max_length).any():
            raise _lib.RedrafterError(f"a row would grow past the cache's {self.max_length} slots")
        start = np.zeros(B + 1, dtype=np.int32)
        np.cumsum(cnt, out=start[1:])
        row = np.repeat(np.arange(B, dtype=np.int32), cnt)
        slot = (first + base - start[:-1])[row] + np.arange(M, dtype=np.int32)
        meta = torch.from_numpy(np.concatenate([row, slot.astype(np.int32), start, base])).to(llm.device)
        tok_row, tok_slot, row_start, base_len = torch.split(meta, [M, M, B + 1, B])
        tok_pos = tok_slot  # a row starts at slot 0 unless its positions are the columns of a padded batch
        llm.gemm_status = self.status
        ws = llm.workspace(M, 1)
        hidden = llm.backbone(ws, self.cache.storage, M, None, tok_ids, tok_row, tok_pos, tok_slot, row_start, self.begin, base_len, B,
                              int(cnt.max()), int((base + cnt).max()), _lib.ATTN_CAUSAL, n_pos=self.max_length + 1)
        self.lengths = [int(v) for v in base + cnt]
        self.kv_len.copy_(base_len)
        self.kv_len.add_(row_start[1:] - row_start[:-1])
        self.cache.set_length(max(self.lengths))
        return hidden

    def release(self, row: int) -> None:
        """Gives row's slots and states back: its next tokens start a new sequence."""
        self.lengths[row] = 0
        self.kv_len[row] = 0

    @torch.inference_mode()
    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        """fp32 logits [rows, vocab] of the given final hidden states (a workspace buffer)."""
        ws = self.llm.workspace(1, hidden_rows.shape[0])
        self.llm.gemm_status = self.status
        return self.llm.lm_logits(hidden_rows.contiguous(), ws["logits"])

    def check(self) -> None:
        """Raises if a bounded wait inside a tensor-core kernel gave up (synchronises)."""
        code = int(self.status.item())
        if code != 0:
            raise _lib.RedrafterError(f"a tensor-core kernel gave up waiting on its pipeline (status {code})")

    # ------------------------------------------------------------------------------------------ one token per row
    def pick(self, sampling_args, tokens: Optional[torch.Tensor] = None, columns: Optional[torch.Tensor] = None) -> None:
        """Chooses every row's next token from last_hidden (arg-max, or a draw with the uniforms of draw_uniforms()) into
        next_tok, appends it to tokens at column columns[b] + kv_len[b], and moves the rows' counters on."""
        llm, B = self.llm, self.batch
        st = _lib.stream()
        V = llm.config.vocab_size
        if sampling_args.greedy and llm.fused_head_ok():
            llm.lm_argmax(self.last_hidden, None, out64=self.next_tok)
        else:
            logits = llm.workspace(B, B)["logits"]
            smax = None
            if sampling_args.greedy:
                llm.lm_logits(self.last_hidden, logits)
                _lib.call("rd_argmax_rows", _lib.ptr(logits), logits.stride(0), B, None, V, None, _lib.ptr(self.next_tok), st)
            else:
                if self._sparse is None:
                    self._sparse = modeling_drafter.new_sparse(B, llm.device)
                smax = llm.lm_logits_with_slice_max(self.last_hidden, logits)
                sp = modeling_drafter.vocab_topk(logits, self._sparse, subtract_max=False, temperature=sampling_args.temperature,
                                                 slice_max=smax)
                _lib.call("rd_sample_from_sparse", _lib.ptr(sp.val), _lib.ptr(sp.idx), _lib.ptr(sp.cnt), B, _lib.ptr(self._u),
                          _lib.ptr(self.next_tok), st)
        _lib.call("rd_decode_advance", _lib.ptr(self.next_tok), _lib.ptr(tokens), tokens.shape[1] if tokens is not None else 0,
                  _lib.ptr(columns), _lib.ptr(self.begin), _lib.ptr(self.kv_len), _lib.ptr(self.base_len), _lib.ptr(self.slot),
                  self.max_length, B, st)

    def draw_uniforms(self) -> None:
        if self._u is None:
            self._u = torch.zeros(self.batch, dtype=torch.float32, device=self.llm.device)
        self._u.copy_(torch.rand(self.batch, device=self.llm.device))

    def forward(self, max_kv: int) -> None:
        """Runs the picked token of every row; last_hidden receives the hidden states."""
        llm, B = self.llm, self.batch
        ws = llm.workspace(B, B)
        hidden = llm.backbone(ws, self.cache.storage, B, None, self.next_tok, self.rows, self.slot, self.slot, self.row_start, self.begin,
                              self.base_len, B, 1, max_kv, _lib.ATTN_CAUSAL, n_pos=self.max_length + 1)
        self.last_hidden.copy_(hidden)


class DecodeGraphs:
    """The two phases of a one-token step (pick, forward) captured as CUDA graphs, for models none of whose kernels is
    sized by a host value that changes from step to step.  Captured after eager steps, when every TMA descriptor set and
    workspace exists."""

    def __init__(self, session: Session, sampling_args, tokens: torch.Tensor, columns: torch.Tensor):
        stream = torch.cuda.Stream()
        stream.wait_stream(torch.cuda.current_stream())
        self.pick, self.forward = torch.cuda.CUDAGraph(), torch.cuda.CUDAGraph()
        before = _lib.launches
        with torch.cuda.stream(stream):
            for graph, fn in ((self.pick, lambda: session.pick(sampling_args, tokens, columns)),
                              (self.forward, lambda: session.forward(session.max_length))):
                # capture_begin directly: the torch.cuda.graph context manager empties the allocator's caches first
                graph.capture_begin(capture_error_mode="thread_local")
                try:
                    fn()
                finally:
                    graph.capture_end()
                if graph is self.pick:
                    self.n_pick = _lib.launches - before
        torch.cuda.current_stream().wait_stream(stream)
        self.n_forward = _lib.launches - before - self.n_pick
        # the captured kernels address these: they stay alive even if a larger request makes the model replace its set
        held = getattr(session.llm, "held_buffers", lambda: [])()
        self.buffers = (session.llm.workspace(session.batch, session.batch), session.llm._head_ws, held)
        _lib.launches = before  # capturing enqueues nothing


def graphs_enabled(llm, cuda_graphs: Optional[bool]) -> bool:
    on = (os.environ.get("RD_CUDA_GRAPHS", "1") != "0") if cuda_graphs is None else bool(cuda_graphs)
    return on and llm.graph_capturable
