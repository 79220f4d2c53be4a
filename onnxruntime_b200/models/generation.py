"""Greedy generation drivers for decoder graphs with GroupQueryAttention or PagedAttention.

Mirrors how the reference's tooling drives an exported LLM
(onnxruntime/python/tools/transformers/models/llama/benchmark_e2e.py:120-148,
435-512): inputs and outputs are bound once with ``IOBinding``; ``past`` and
``present`` of every layer are bound to the SAME pre-allocated cache buffer so
the KV cache never moves; the prompt runs once, then one token per step.  The
decode step has fixed shapes and addresses, so with ``enable_cuda_graph`` the
session captures it on the first step and replays it afterwards.
"""
from __future__ import annotations

from typing import Dict, Hashable, List, Optional, Sequence, Tuple, Union

import torch

from ..capi import InferenceSession, RunOptions
from .decoder_cache import CacheFull, CachePool
from .llama import LlamaConfig, empty_kv_cache


class DecoderRunner:
    """Owns the KV cache and the bindings of one (session, batch size, cache capacity)."""

    def __init__(self, session: InferenceSession, cfg: LlamaConfig, batch: int, max_len: int, tp_size: int = 1,
                 device: Optional[torch.device] = None, prefill_graph: bool = False):
        """``prefill_graph``: also capture the prompt run in a CUDA graph (one graph per prompt shape; worthwhile when the
        same prompt shape recurs, e.g. fixed-size prefill chunks).  Needs a session created with ``enable_cuda_graph``."""
        self.sess = session
        self.cfg = cfg
        self.batch = batch
        self.max_len = max_len
        self.device = device if device is not None else (
            torch.device("cuda", torch.cuda.current_device()) if "CUDAExecutionProvider" in session.get_providers() else torch.device("cpu"))
        self.cache = empty_kv_cache(cfg, batch, max_len, self.device, tp_size)
        self.out_names = [o.name for o in session.get_outputs()]
        self.has_argmax = "next_tokens" in self.out_names
        # static device buffers for the decode step (addresses must not change between graph replays)
        self.step_ids = torch.zeros(batch, 1, dtype=torch.int64, device=self.device)
        self.step_seqlens = torch.zeros(batch, dtype=torch.int32, device=self.device)
        self.step_next = torch.zeros(batch, 1, dtype=torch.int64, device=self.device)
        self.step_logits = torch.zeros(batch, 1, cfg.vocab_size, dtype=self.cache[0][0].dtype, device=self.device)
        self._decode_binding = None
        self._decode_total = None
        self._ro_decode = RunOptions()
        self._ro_decode.add_run_config_entry("gpu_graph_id", "1")
        self._ro_prefill = RunOptions()
        self._ro_prefill.add_run_config_entry("gpu_graph_id", "-1")
        self._prefill_graph = prefill_graph
        self._prefill_graph_ids: Dict[Tuple[int, int], int] = {}

    def _bind_common(self, binding, ids: torch.Tensor, seqlens: torch.Tensor, total: torch.Tensor, logits, next_tokens) -> None:
        binding.bind_torch_input("input_ids", ids)
        binding.bind_torch_input("seqlens_k", seqlens)
        binding.bind_torch_input("total_sequence_length", total)
        for i, (k, v) in enumerate(self.cache):
            binding.bind_torch_input(f"past_key_values.{i}.key", k)
            binding.bind_torch_input(f"past_key_values.{i}.value", v)
            binding.bind_torch_output(f"present.{i}.key", k)
            binding.bind_torch_output(f"present.{i}.value", v)
        binding.bind_torch_output("logits", logits)
        if self.has_argmax:
            binding.bind_torch_output("next_tokens", next_tokens)

    def prefill(self, input_ids: torch.Tensor) -> torch.Tensor:
        """Run the prompt [B, S]; returns the first generated token per sequence [B, 1] (device tensor)."""
        B, S = input_ids.shape
        assert B == self.batch and S <= self.max_len
        ids = input_ids.to(self.device)
        seqlens = torch.full((B,), S - 1, dtype=torch.int32, device=self.device)
        total = torch.tensor(S, dtype=torch.int32)
        logits = torch.empty(B, 1, self.cfg.vocab_size, dtype=self.cache[0][0].dtype, device=self.device)
        nxt = torch.empty(B, 1, dtype=torch.int64, device=self.device)
        binding = self.sess.io_binding()
        self._bind_common(binding, ids, seqlens, total, logits, nxt)
        ro = self._ro_prefill
        if self._prefill_graph:
            gid = self._prefill_graph_ids.setdefault((B, S), 2 + len(self._prefill_graph_ids))
            ro = RunOptions()
            ro.add_run_config_entry("gpu_graph_id", str(gid))
        try:
            self.sess.run_with_iobinding(binding, ro)
        except Exception:
            if ro is self._ro_prefill:
                raise
            # the prompt graph holds something that cannot be captured: run it eagerly from now on
            self._prefill_graph = False
            self.sess.run_with_iobinding(binding, self._ro_prefill)
        self.cur_len = S
        self.prefill_logits = logits
        if not self.has_argmax:
            nxt = logits.float().argmax(-1)
        return nxt

    def reorder_cache(self, rows: torch.Tensor) -> None:
        """Row i of every cache takes the content of row rows[i] (beam search: beams follow their parents)."""
        rows = rows.to(self.device)
        for k, v in self.cache:
            k.copy_(k.index_select(0, rows))
            v.copy_(v.index_select(0, rows))

    def _ensure_decode_binding(self) -> None:
        if self._decode_binding is not None:
            return
        binding = self.sess.io_binding()
        # the capacity bound is a host scalar: the cache capacity, so the captured graph stays valid every step
        self._decode_total = torch.tensor(self.max_len, dtype=torch.int32)
        self._bind_common(binding, self.step_ids, self.step_seqlens, self._decode_total, self.step_logits, self.step_next)
        self._decode_binding = binding

    def decode_step(self, tokens: Optional[torch.Tensor] = None) -> torch.Tensor:
        """One decode step.  ``tokens`` [B, 1] (device or pinned host); None re-uses the previous step's output,
        which already sits in the bound input buffer."""
        self._ensure_decode_binding()
        if tokens is not None:
            self.step_ids.copy_(tokens, non_blocking=True)
        else:
            self.step_ids.copy_(self.step_next)
        self.step_seqlens.fill_(self.cur_len)  # total length - 1 after appending this token
        self.sess.run_with_iobinding(self._decode_binding, self._ro_decode)
        self.cur_len += 1
        if not self.has_argmax:
            self.step_next.copy_(self.step_logits.float().argmax(-1))
        return self.step_next

    def decode_step_host(self, ids_pinned: torch.Tensor, seqlens_pinned: torch.Tensor, out_pinned: torch.Tensor) -> None:
        """One decode step driven from the host: inputs come from pinned host memory, the sampled tokens are
        copied back to pinned host memory and the call returns after they have arrived."""
        self._ensure_decode_binding()
        seqlens_pinned.fill_(self.cur_len)
        self.step_ids.copy_(ids_pinned, non_blocking=True)
        self.step_seqlens.copy_(seqlens_pinned, non_blocking=True)
        self.sess.run_with_iobinding(self._decode_binding, self._ro_decode)
        self.cur_len += 1
        if not self.has_argmax:
            self.step_next.copy_(self.step_logits.float().argmax(-1))
        out_pinned.copy_(self.step_next, non_blocking=True)
        torch.cuda.current_stream().synchronize() if self.device.type == "cuda" else None

    def generate(self, input_ids: torch.Tensor, max_new_tokens: int) -> torch.Tensor:
        out = [self.prefill(input_ids).clone()]
        for _ in range(max_new_tokens - 1):
            nxt = self.decode_step(out[-1])
            out.append(nxt.clone())
        return torch.cat(out, dim=1)


class PagedDecoderRunner:
    """Decoding over pooled caches: the serving form of a decoder.  Tokens of all sequences of a step are packed along
    one axis; all sequences share one pool of cache blocks (``block_table[b, j]`` names the block that holds tokens
    [j * block_size, (j + 1) * block_size) of sequence b, as in com.microsoft.PagedAttention,
    onnxruntime/contrib_ops/cuda/bert/paged_attention.cc) and one pool of state slots for models with recurrent layers
    (``state_slots[b]``).  What a model keeps is declared by ``cfg.cache_tensors()``.

    ``step`` runs one batch of any composition - whole prompts, portions of prompts, single tokens - for sequences named
    by the caller and returns the wanted logits; ``release`` gives a sequence's blocks and slot back.  ``prefill`` /
    ``decode_step`` drive a fixed batch of ``batch`` rows on top of the same pool.  A step that brings one token per
    sequence has fixed shapes and addresses and is captured as one CUDA graph per batch size."""

    def __init__(self, session: InferenceSession, cfg, batch: int, max_len: int, block_size: int = 256,
                 tp_size: int = 1, device: Optional[torch.device] = None, graph_id: int = 1, num_blocks: Optional[int] = None,
                 num_slots: Optional[int] = None):
        """``num_blocks``: size of the block pool (default: ``batch`` sequences of ``max_len`` tokens); ``max_len`` bounds
        one sequence; ``num_slots`` (default ``batch``) bounds the sequences that are open at a time."""
        self.sess, self.cfg, self.batch, self.max_len, self.block_size = session, cfg, batch, max_len, block_size
        self.device = device if device is not None else (
            torch.device("cuda", torch.cuda.current_device()) if "CUDAExecutionProvider" in session.get_providers() else torch.device("cpu"))
        self.blocks_per_seq = (max_len + block_size - 1) // block_size
        self.pool = CachePool(cfg.cache_tensors(tp_size), num_blocks or batch * self.blocks_per_seq, block_size, num_slots or batch, self.device)
        out_info = {o.name: o for o in session.get_outputs()}
        in_names = {i.name for i in session.get_inputs()}
        self.has_argmax = "next_tokens" in out_info
        self.has_slots = "state_slots" in in_names
        self.has_key_starts = "key_starts" in in_names
        self.logits_dtype = {"tensor(float)": torch.float32, "tensor(float16)": torch.float16,
                             "tensor(bfloat16)": torch.bfloat16}[out_info["logits"].type]
        self._steps: Dict[int, "_DecodeBuffers"] = {}
        self._graph_id = graph_id             # graph ids graph_id, graph_id + 1, ...: one captured graph per batch size
        self._ro_prefill = RunOptions()
        self._ro_prefill.add_run_config_entry("gpu_graph_id", "-1")
        self._rows: List[Tuple[str, int]] = [("row", b) for b in range(batch)]   # sequences of prefill / decode_step
        self.prefill_logits = self.step_logits = None

    @property
    def cur_len(self) -> int:
        """Tokens held by the longest row of the fixed batch."""
        return max((self.pool.sequences[r].length for r in self._rows if r in self.pool.sequences), default=0)

    @cur_len.setter
    def cur_len(self, length: int) -> None:
        self.assume_context(length)

    @property
    def cache(self) -> List[Tuple[torch.Tensor, torch.Tensor]]:
        """(key, value) block pools of the attention layers that own them (models that cache keys and values in every layer)."""
        paged = [self.pool.tensors[c.input] for c in self.pool.spec if c.kind == "paged"]
        return list(zip(paged[::2], paged[1::2]))

    @property
    def block_table(self) -> torch.Tensor:
        """Block table of the fixed batch."""
        return self._table(self._rows).to(self.device)

    def _table(self, seqs) -> torch.Tensor:
        t = torch.zeros(len(seqs), self.blocks_per_seq, dtype=torch.int32)
        for b, s in enumerate(seqs):
            blocks = self.pool.sequences[s].blocks
            t[b, :len(blocks)] = torch.tensor(blocks, dtype=torch.int32)
        return t

    def _slots(self, seqs) -> torch.Tensor:
        return torch.tensor([self.pool.sequences[s].slot for s in seqs], dtype=torch.int32)

    def _bind(self, binding, ids, cum, past, table, slots, key_starts, rows, logits, nxt) -> None:
        binding.bind_torch_input("input_ids", ids)
        binding.bind_torch_input("cumulative_sequence_length", cum)
        binding.bind_torch_input("past_seqlens", past)
        binding.bind_torch_input("block_table", table)
        binding.bind_torch_input("logits_indices", rows)
        if self.has_slots:
            binding.bind_torch_input("state_slots", slots)
        if self.has_key_starts:
            binding.bind_torch_input("key_starts", key_starts)
        for c in self.pool.spec:
            binding.bind_torch_input(c.input, self.pool.tensors[c.input])
            binding.bind_torch_output(c.output, self.pool.tensors[c.input])
        binding.bind_torch_output("logits", logits)
        if self.has_argmax:
            binding.bind_torch_output("next_tokens", nxt)

    # ------------------------------------------------------------------------------------------------- general steps
    def step(self, entries: Sequence[Tuple[Hashable, Sequence[int], Sequence[int]]]) -> torch.Tensor:
        """One batch: ``entries`` = (sequence, its next tokens, places among them whose logits are wanted).  A sequence
        seen for the first time is opened.  Returns the logits [wanted, vocab] in the order of the entries."""
        entries = [e for e in entries if len(e[1]) > 0]
        opened = []
        try:
            for seq, tokens, want in entries:
                if any(not 0 <= w < len(tokens) for w in want):
                    raise ValueError(f"sequence {seq!r}: a wanted place lies outside its {len(tokens)} tokens")
                if seq not in self.pool.sequences:
                    self.pool.open(seq)
                    opened.append(seq)
                if self.pool.sequences[seq].length + len(tokens) > self.max_len:
                    raise CacheFull(f"sequence {seq!r} would exceed {self.max_len} tokens")
                self.pool.reserve(seq, len(tokens))
        except Exception:
            for seq in opened:
                self.pool.close(seq)
            raise
        if not entries:
            return torch.empty(0, self.cfg.vocab_size, dtype=self.logits_dtype, device=self.device)
        seqs = [e[0] for e in entries]
        if all(len(e[1]) == 1 for e in entries):
            buf = self._decode_buffers(len(entries))
            buf.ids.copy_(torch.tensor([int(e[1][0]) for e in entries], dtype=torch.int64))
            self._run_decode(buf, seqs)
            wanted = [b for b, e in enumerate(entries) for _ in e[2]]
            return buf.logits[torch.tensor(wanted, dtype=torch.int64, device=self.device)]
        ids = torch.cat([torch.as_tensor(e[1], dtype=torch.int64).reshape(-1).cpu() for e in entries])
        starts, rows = [0], []
        for _, tokens, want in entries:
            rows += [starts[-1] + int(w) for w in want]
            starts.append(starts[-1] + len(tokens))
        logits, _ = self._run_packed(ids, starts, seqs, rows or [0])
        return logits if rows else logits[:0]

    def release(self, seq: Hashable) -> None:
        """The sequence is finished: its blocks and slot go back to the pool."""
        self.pool.close(seq)

    def _run_packed(self, ids: torch.Tensor, starts, seqs, rows) -> Tuple[torch.Tensor, torch.Tensor]:
        dev = self.device
        lengths = [self.pool.sequences[s].length for s in seqs]
        past = torch.tensor(lengths, dtype=torch.int32)
        # host tensor: the keys of sequence b, cached and new, are rows [key_starts[b], key_starts[b + 1]) of an expansion
        key_starts = torch.tensor([starts[b] + sum(lengths[:b]) for b in range(len(seqs) + 1)], dtype=torch.int32)
        logits = torch.empty(len(rows), self.cfg.vocab_size, dtype=self.logits_dtype, device=dev)
        nxt = torch.empty(len(rows), dtype=torch.int64, device=dev)
        binding = self.sess.io_binding()
        self._bind(binding, ids.to(dev), torch.tensor(starts, dtype=torch.int32).to(dev), past.to(dev), self._table(seqs).to(dev),
                   self._slots(seqs).to(dev), key_starts, torch.tensor(rows, dtype=torch.int64).to(dev), logits, nxt)
        self.sess.run_with_iobinding(binding, self._ro_prefill)
        for b, s in enumerate(seqs):
            self.pool.advance(s, starts[b + 1] - starts[b])
        if not self.has_argmax:
            nxt = logits.float().argmax(-1)
        return logits, nxt

    def _decode_buffers(self, rows: int) -> "_DecodeBuffers":
        if rows not in self._steps:
            buf = _DecodeBuffers(rows, self.blocks_per_seq, self.cfg.vocab_size, self.logits_dtype, self.device)
            buf.binding = self.sess.io_binding()
            self._bind(buf.binding, buf.ids, buf.cum, buf.past, buf.table, buf.slots, buf.key_starts, buf.rows, buf.logits, buf.next)
            buf.options.add_run_config_entry("gpu_graph_id", str(self._graph_id + len(self._steps)))
            self._steps[rows] = buf
        return self._steps[rows]

    def _run_decode(self, buf: "_DecodeBuffers", seqs) -> None:
        """One token per sequence, ids already in ``buf.ids``; room has been reserved."""
        layout = [(s, self.pool.sequences[s].slot, tuple(self.pool.sequences[s].blocks)) for s in seqs]
        if layout != buf.layout:
            buf.table.copy_(self._table(seqs))
            buf.slots.copy_(self._slots(seqs))
            buf.layout = layout
        lengths = [self.pool.sequences[s].length for s in seqs]
        if lengths.count(lengths[0]) == len(lengths):
            buf.past.fill_(lengths[0])
        else:
            buf.past.copy_(torch.tensor(lengths, dtype=torch.int32))
        self.sess.run_with_iobinding(buf.binding, buf.options)
        for s in seqs:
            self.pool.advance(s, 1)
        if not self.has_argmax:
            buf.next.copy_(buf.logits.float().argmax(-1))

    # ------------------------------------------------------------------------------------------- the fixed batch of rows
    def _reopen_rows(self) -> None:
        for r in self._rows:
            if r in self.pool.sequences:
                self.pool.close(r)
        for r in self._rows:
            self.pool.open(r)
        # full capacity at once, one block per row in turn: the block table of a row is fixed from here on, and no row owns
        # a contiguous range
        for j in range(self.blocks_per_seq):
            for r in self._rows:
                self.pool.reserve(r, min((j + 1) * self.block_size, self.max_len))

    def prefill(self, input_ids) -> torch.Tensor:
        """Prompts of the fixed batch: a tensor [B, S] or a list of B prompts of any lengths, packed without padding.
        Returns the first generated token of every row [B]."""
        prompts = [torch.as_tensor(p, dtype=torch.int64).reshape(-1) for p in input_ids]
        assert len(prompts) == self.batch and all(1 <= len(p) <= self.max_len for p in prompts)
        self._reopen_rows()
        starts = [0]
        for p in prompts:
            starts.append(starts[-1] + len(p))
        self.prefill_logits, nxt = self._run_packed(torch.cat(prompts), starts, self._rows, [s - 1 for s in starts[1:]])
        self._decode_buffers(self.batch).next.copy_(nxt)
        return nxt

    def assume_context(self, length: int) -> None:
        """Treat the caches as holding ``length`` tokens per sequence (benchmarks that time decode over a cache
        filled with arbitrary values instead of running a prompt first)."""
        assert 0 <= length < self.max_len
        if any(r not in self.pool.sequences for r in self._rows):
            self._reopen_rows()
        for r in self._rows:
            self.pool.sequences[r].length = length

    def decode_step(self, tokens: Optional[torch.Tensor] = None) -> torch.Tensor:
        """One token per sequence; ``tokens`` [B] or None to feed back the previous step's output."""
        buf = self._decode_buffers(self.batch)
        buf.ids.copy_(tokens.reshape(-1) if tokens is not None else buf.next, non_blocking=True)
        self._run_decode(buf, self._rows)
        self.step_logits = buf.logits
        return buf.next

    def reorder_cache(self, rows: torch.Tensor) -> None:
        """Row i takes the content of row rows[i] (beam search: beams follow their parents)."""
        self.pool.copy_sequence_state([self._rows[int(r)] for r in rows.tolist()], self._rows)

    def generate(self, input_ids, max_new_tokens: int) -> torch.Tensor:
        out = [self.prefill(input_ids).clone()]
        for _ in range(max_new_tokens - 1):
            out.append(self.decode_step(out[-1]).clone())
        return torch.stack(out, dim=1)


class _DecodeBuffers:
    """Device buffers of the one-token step of one batch size; their addresses are frozen into its CUDA graph."""

    def __init__(self, rows: int, max_blocks: int, vocab: int, logits_dtype: torch.dtype, device: torch.device):
        self.ids = torch.zeros(rows, dtype=torch.int64, device=device)
        self.cum = torch.arange(rows + 1, dtype=torch.int32, device=device)
        self.past = torch.zeros(rows, dtype=torch.int32, device=device)
        self.table = torch.zeros(rows, max_blocks, dtype=torch.int32, device=device)
        self.slots = torch.zeros(rows, dtype=torch.int32, device=device)
        self.key_starts = torch.zeros(rows + 1, dtype=torch.int32)     # one-token steps read the cache as it lies
        self.rows = torch.arange(rows, dtype=torch.int64, device=device)
        self.logits = torch.zeros(rows, vocab, dtype=logits_dtype, device=device)
        self.next = torch.zeros(rows, dtype=torch.int64, device=device)
        self.layout = None
        self.binding = None
        self.options = RunOptions()


# ----------------------------------------------------------------------------------------------------------------
# Logits processors, sampling and beam search on top of DecoderRunner.  The knobs are the attributes / inputs of the
# reference's generation operators (com.microsoft GreedySearch, Sampling, BeamSearch:
# onnxruntime/contrib_ops/cpu/transformers/{greedy_search.cc, sampling.cc, beam_search.cc, logits_processor.h});
# here the loop runs in Python over the session's bound decode step and all tensor work stays on the device.
class GenerationConfig:
    def __init__(self, max_new_tokens: int = 32, min_new_tokens: int = 0, eos_token_id: Optional[int] = None,
                 pad_token_id: int = 0, temperature: float = 1.0, top_k: int = 0, top_p: float = 1.0,
                 repetition_penalty: float = 1.0, no_repeat_ngram_size: int = 0, num_beams: int = 1,
                 length_penalty: float = 1.0, early_stopping: bool = False, num_return_sequences: int = 1,
                 vocab_mask: Optional[torch.Tensor] = None, seed: Optional[int] = None):
        self.__dict__.update(locals())
        del self.__dict__["self"]


def process_logits(logits: torch.Tensor, sequences: torch.Tensor, step: int, cfg: GenerationConfig) -> torch.Tensor:
    """logits [rows, vocab] (fp32), sequences [rows, len] = every token so far (prompt included).  Order of the
    reference's LogitsProcessorList: min length, repetition penalty, no-repeat n-gram, vocabulary mask, temperature."""
    logits = logits.float().clone()
    if cfg.eos_token_id is not None and step < cfg.min_new_tokens:
        logits[:, cfg.eos_token_id] = float("-inf")
    if cfg.repetition_penalty != 1.0:
        seen = torch.gather(logits, 1, sequences)
        seen = torch.where(seen < 0, seen * cfg.repetition_penalty, seen / cfg.repetition_penalty)
        logits.scatter_(1, sequences, seen)
    n = cfg.no_repeat_ngram_size
    if n > 0 and sequences.shape[1] + 1 >= n:
        L = sequences.shape[1]
        if n == 1:
            logits.scatter_(1, sequences, float("-inf"))
        else:
            grams = sequences.unfold(1, n, 1)                      # [rows, L - n + 1, n]
            tail = sequences[:, L - (n - 1):].unsqueeze(1)          # [rows, 1, n - 1]
            hit = (grams[:, :, : n - 1] == tail).all(-1)            # n-grams whose prefix equals the current tail
            banned = torch.where(hit, grams[:, :, n - 1], torch.full_like(grams[:, :, n - 1], -1))
            rows = torch.arange(logits.shape[0], device=logits.device).unsqueeze(1).expand_as(banned)
            keep = banned >= 0
            logits[rows[keep], banned[keep]] = float("-inf")
    if cfg.vocab_mask is not None:
        logits = logits.masked_fill(cfg.vocab_mask.to(logits.device).view(1, -1) == 0, float("-inf"))
    if cfg.temperature != 1.0 and cfg.temperature > 0:
        logits = logits / cfg.temperature
    return logits


def top_k_top_p_filter(logits: torch.Tensor, top_k: int, top_p: float) -> torch.Tensor:
    if top_k > 0:
        kth = torch.topk(logits, min(top_k, logits.shape[-1]), dim=-1).values[:, -1:]
        logits = logits.masked_fill(logits < kth, float("-inf"))
    if top_p < 1.0:
        sorted_logits, idx = torch.sort(logits, descending=True, dim=-1)
        cum = torch.softmax(sorted_logits, -1).cumsum(-1)
        drop = cum - torch.softmax(sorted_logits, -1) > top_p       # keep the token that crosses the threshold
        sorted_logits = sorted_logits.masked_fill(drop, float("-inf"))
        logits = torch.full_like(logits, float("-inf")).scatter(1, idx, sorted_logits)
    return logits


def generate(runner: Union[DecoderRunner, PagedDecoderRunner], input_ids: torch.Tensor, cfg: GenerationConfig) -> torch.Tensor:
    """Greedy (``num_beams == 1``, ``top_k == 0``, ``top_p == 1``, temperature 1), sampling or beam search.
    Returns [batch * num_return_sequences, prompt + generated] token ids, padded with ``pad_token_id`` after EOS.
    For beam search the runner must have been created with ``batch = prompts * num_beams``."""
    if cfg.num_beams > 1:
        return _beam_search(runner, input_ids, cfg)
    dev = runner.device
    sampling = cfg.top_k > 0 or cfg.top_p < 1.0 or cfg.seed is not None
    gen = torch.Generator(device=dev)
    if cfg.seed is not None:
        gen.manual_seed(cfg.seed)
    seqs = input_ids.to(dev)
    done = torch.zeros(seqs.shape[0], dtype=torch.bool, device=dev)
    runner.prefill(input_ids)
    logits = _last_logits(runner, prefill=True)
    for step in range(cfg.max_new_tokens):
        scores = process_logits(logits, seqs, step, cfg)
        if sampling:
            probs = torch.softmax(top_k_top_p_filter(scores, cfg.top_k, cfg.top_p), -1)
            nxt = torch.multinomial(probs, 1, generator=gen).squeeze(1)
        else:
            nxt = scores.argmax(-1)
        nxt = torch.where(done, torch.full_like(nxt, cfg.pad_token_id), nxt)
        seqs = torch.cat([seqs, nxt.unsqueeze(1)], 1)
        if cfg.eos_token_id is not None:
            done = done | (nxt == cfg.eos_token_id)
            if bool(done.all()):
                break
        if step + 1 < cfg.max_new_tokens:
            runner.decode_step(nxt.view(-1, 1))
            logits = _last_logits(runner, prefill=False)
    return seqs


def generate_requests(runner: PagedDecoderRunner, prompts: Sequence[Sequence[int]], cfg: GenerationConfig) -> List[List[int]]:
    """Greedy or sampled continuations of prompts of any lengths, with the processors and knobs of ``generate``.  At most
    ``runner.batch`` requests run at a time; a finished one frees its blocks and slot, and the next waiting prompt joins
    the running batch in a step of its own.  Returns the generated tokens of every request (end token included)."""
    if cfg.num_beams > 1:
        raise ValueError("beam search needs a fixed batch: use generate()")
    sampling = cfg.top_k > 0 or cfg.top_p < 1.0 or cfg.seed is not None
    gen = torch.Generator(device=runner.device)
    if cfg.seed is not None:
        gen.manual_seed(cfg.seed)
    texts = [[int(t) for t in p] for p in prompts]
    done: List[Optional[List[int]]] = [None] * len(texts)
    new: Dict[int, List[int]] = {}
    waiting, running = list(range(len(texts))), []

    def pick(i: int, logits: torch.Tensor) -> None:
        seq = torch.tensor([texts[i] + new[i]], dtype=torch.int64, device=runner.device)
        scores = process_logits(logits.reshape(1, -1), seq, len(new[i]), cfg)
        if sampling:
            tok = int(torch.multinomial(torch.softmax(top_k_top_p_filter(scores, cfg.top_k, cfg.top_p), -1), 1, generator=gen))
        else:
            tok = int(scores.argmax(-1))
        new[i].append(tok)
        if len(new[i]) >= cfg.max_new_tokens or tok == cfg.eos_token_id:
            done[i] = new.pop(i)
            running.remove(i)
            runner.release(("request", i))

    while waiting or running:
        joining = waiting[:runner.batch - len(running)]
        while joining:   # prompts that fit into the free blocks together with the tokens they will generate
            room = len(runner.pool.free_blocks)
            need = [(len(texts[i]) + cfg.max_new_tokens + runner.block_size - 1) // runner.block_size for i in joining]
            held = sum(max(0, (len(texts[i]) + cfg.max_new_tokens + runner.block_size - 1) // runner.block_size
                           - len(runner.pool.sequences[("request", i)].blocks)) for i in running)
            if sum(need) + held <= room:
                break
            joining.pop()
        if joining:
            logits = runner.step([(("request", i), texts[i], [len(texts[i]) - 1]) for i in joining])
            waiting = waiting[len(joining):]
            running += joining
            for i in joining:
                new[i] = []
        elif running:
            joining = list(running)
            logits = runner.step([(("request", i), [new[i][-1]], [0]) for i in joining])
        else:
            raise CacheFull(f"request {waiting[0]} does not fit into the cache")
        for row, i in enumerate(joining):
            pick(i, logits[row])
    return done


def _last_logits(runner: DecoderRunner, prefill: bool) -> torch.Tensor:
    src = runner.prefill_logits if prefill else runner.step_logits
    return src.reshape(src.shape[0], -1).float()


def _beam_search(runner: DecoderRunner, input_ids: torch.Tensor, cfg: GenerationConfig) -> torch.Tensor:
    """Beam search with the scorer of the reference (beam_search_scorer.cc): hypotheses are ranked by
    sum(log p) / length ** length_penalty, 2 * num_beams candidates are examined per step so that finished beams
    can be replaced, and the KV cache rows follow their beams."""
    dev = runner.device
    B, K = input_ids.shape[0], cfg.num_beams
    assert runner.batch == B * K, "beam search needs a runner with batch = prompts * num_beams"
    seqs = input_ids.to(dev).repeat_interleave(K, 0)
    prompt_len = seqs.shape[1]
    runner.prefill(seqs)
    logits = _last_logits(runner, prefill=True)
    beam_scores = torch.zeros(B, K, device=dev)
    beam_scores[:, 1:] = -1e9                    # all beams of a prompt start identical: keep one alive
    finished: List[List[Tuple[float, torch.Tensor]]] = [[] for _ in range(B)]
    done = [False] * B
    V = logits.shape[-1]
    for step in range(cfg.max_new_tokens):
        logp = torch.log_softmax(process_logits(logits, seqs, step, cfg), -1)
        cand = (beam_scores.view(B * K, 1) + logp).view(B, K * V)
        top_scores, top_idx = torch.topk(cand, 2 * K, dim=1)
        src_beam, token = top_idx // V, top_idx % V
        new_scores = torch.full((B, K), -1e9, device=dev)
        new_src = torch.zeros(B, K, dtype=torch.long, device=dev)
        new_tok = torch.full((B, K), cfg.pad_token_id, dtype=torch.long, device=dev)
        ts, sb, tk = top_scores.tolist(), src_beam.tolist(), token.tolist()
        cur_len = seqs.shape[1] + 1 - prompt_len
        for b in range(B):
            if done[b]:
                continue
            filled = 0
            for rank in range(2 * K):
                if cfg.eos_token_id is not None and tk[b][rank] == cfg.eos_token_id:
                    if rank < K:   # only candidates that would have survived may finish
                        hyp = torch.cat([seqs[b * K + sb[b][rank]], torch.tensor([cfg.eos_token_id], device=dev)])
                        finished[b].append((ts[b][rank] / (cur_len ** cfg.length_penalty), hyp))
                    continue
                new_scores[b, filled], new_src[b, filled], new_tok[b, filled] = ts[b][rank], sb[b][rank], tk[b][rank]
                filled += 1
                if filled == K:
                    break
            if len(finished[b]) >= K:
                best_open = float(new_scores[b].max()) / (cur_len ** cfg.length_penalty)
                worst_kept = sorted(f[0] for f in finished[b])[-K]
                if cfg.early_stopping or worst_kept >= best_open:
                    done[b] = True
        rows = (torch.arange(B, device=dev).unsqueeze(1) * K + new_src).view(-1)
        seqs = torch.cat([seqs.index_select(0, rows), new_tok.view(-1, 1)], 1)
        beam_scores = new_scores
        if all(done):
            break
        if step + 1 < cfg.max_new_tokens:
            runner.reorder_cache(rows)
            runner.decode_step(new_tok.view(-1, 1))
            logits = _last_logits(runner, prefill=False)
    out = []
    gen_len = seqs.shape[1] - prompt_len
    for b in range(B):
        hyps = list(finished[b])
        for k in range(K):   # open beams count as hypotheses of the current length
            hyps.append((float(beam_scores[b, k]) / (max(gen_len, 1) ** cfg.length_penalty), seqs[b * K + k]))
        hyps.sort(key=lambda h: -h[0])
        out.extend(h[1] for h in hyps[: cfg.num_return_sequences])
    width = max(h.shape[0] for h in out)
    return torch.stack([torch.nn.functional.pad(h, (0, width - h.shape[0]), value=cfg.pad_token_id) for h in out])
