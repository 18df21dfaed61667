"""The part of the inference engines that does not depend on the model family: batch buckets, the captured decode tick
and its reuse, ``generate``, request admission (``serve``), the samplers.

A family's engine (:class:`tah_b200.engine.engine.TaHEngine`, :class:`tah_b200.engine.hybrid.HybridEngine`) supplies

* ``_new_cache(rows, max_tokens)``  (re)build ``self.kv`` (and whatever else a row carries),
* ``prefill(ids, mask, max_new_tokens, row_ids)``  run prompts, return the logits of their last tokens and their lengths,
* ``_alloc_tick_buffers(rows, max_new)`` / ``_tick(state, sampling)``  one decode tick of every row, graph-capturable.
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field
from typing import List, Optional, Sequence

import torch

from tah_b200.engine.kv_cache import PagedKVCache
from tah_b200.ops import cuda as K
from tah_b200.utils.observe import MetricsSink, engine_counters, nvtx_range


@dataclass
class GenerationResult:
    tokens: List[List[int]]
    iter_counts: List[float]            # mean passes per emitted token, per row
    ticks: int = 0
    tokens_emitted: int = 0
    prefill_ms: float = 0.0
    decode_ms: float = 0.0
    extra: dict = field(default_factory=dict)


class DecodeEngine:
    """Scheduling and sampling shared by the engines; see the module docstring for what a subclass supplies."""

    def _init_scheduler(self, max_rows: int, max_seq_len: int, page_size: int, use_cuda_graph: bool) -> None:
        self.max_rows, self.max_seq_len, self.page_size = max_rows, max_seq_len, page_size
        self.use_cuda_graph = use_cuda_graph and os.environ.get("TAH_B200_NO_GRAPH", "0") != "1"
        self.kv: Optional[PagedKVCache] = None
        self._states = {}          # (rows, max_new, sampling, eos, override) -> tick state with its captured graph
        self._calls = 0
        self.graph_captures = 0
        self.graph_reuses = 0
        self.hard_override: Optional[torch.Tensor] = None     # [rows, max_seq_len] int8: extra passes per position
        self.kernel_launches_per_tick = 0
        # counters of the last generate() call (KV page occupancy per depth, ticks per token, passes per token,
        # graph reuse ...); appended to the JSONL file named by TAH_B200_METRICS when that variable is set
        self.last_counters: dict = {}
        path = os.environ.get("TAH_B200_METRICS")
        self.metrics = MetricsSink(path) if path else None

    # ------------------------------------------------------------------------------------------
    # scheduler state of a tick
    # ------------------------------------------------------------------------------------------
    def _alloc_scheduler_state(self, B: int, max_new: int):
        """The per-row scheduler tensors of a tick and their packing for the tick kernels (``csrc/sampling.cu``)."""
        dev = self.device
        i32 = lambda *s: torch.zeros(*s, dtype=torch.int32, device=dev)
        s = type("S", (), {})()
        s.tok, s.depth, s.pos, s.finished, s.n_out = i32(B), i32(B), i32(B), i32(B), i32(B)
        s.out_tokens, s.iter_sum, s.cur_iters, s.slot, s.gate = i32(B, max_new), i32(B), i32(B), i32(B), i32(B)
        s.tokens_done = torch.zeros(1, dtype=torch.int64, device=dev)
        s.need_soft, s.best, s.sampled = i32(B), i32(B), i32(B)
        s.best_val = torch.zeros(B, dtype=torch.float32, device=dev)
        s.samp_v = torch.zeros(B, 128, dtype=torch.float32, device=dev)
        s.samp_i = i32(B, 128)
        s.seed_dev = torch.zeros(1, dtype=torch.int64, device=dev)     # per-call sampling seed, read on the device
        s.graph = None
        kv = self.kv
        pad = lambda lst: list(lst) + [lst[0]] * (4 - len(lst))
        tensors = [s.tok, s.depth, s.pos, s.finished, s.n_out, s.out_tokens, s.iter_sum, s.cur_iters, s.slot, s.gate]
        tensors += pad(kv.len) + pad(kv.page_table) + pad(kv.free_stack) + pad(kv.free_count)
        tensors += [K.status_word(dev), s.tokens_done]
        s.ints = pad(kv.max_pages) + [kv.n_depths, self.page_size, B, max_new, -1, self.max_iter]
        s.tensors = tensors
        return s

    # ------------------------------------------------------------------------------------------
    # sampling
    # ------------------------------------------------------------------------------------------
    def _argmax(self, logits: torch.Tensor) -> torch.Tensor:
        val, idx = logits.float().max(dim=-1)
        if self.tp is None:
            return idx.to(torch.int32)
        return self.tp.merge_argmax(val, idx.to(torch.int32), self.w.vocab_shard[0])

    def _topk(self, x, k, flag, out_val, out_idx):
        """Sorted top-k of (this rank's vocabulary shard of) ``x``; merged across shards under TP."""
        K.topk_rows(x, k, flag=flag, out_val=out_val, out_idx=out_idx)
        if self.tp is not None:
            v, i = self.tp.merge_topk(out_val, out_idx, self.w.vocab_shard[0], k)
            out_val.copy_(v)
            out_idx.copy_(i)

    def _choose(self, logits, step, sampling, seed: int, seed_dev):
        """Next token of every row of ``logits`` outside a tick; ``step``: position each row's draw is keyed by."""
        if sampling is None:
            return self._argmax(logits)
        if logits.dtype != torch.bfloat16:
            logits = logits.to(torch.bfloat16)              # the samplers take bf16 logits
        k, args = sampling["top_k"], (sampling["temperature"], sampling["top_p"], sampling["min_p"])
        if 0 < k <= 128:
            val = torch.zeros(logits.shape[0], k, dtype=torch.float32, device=logits.device)
            idx = torch.zeros(logits.shape[0], k, dtype=torch.int32, device=logits.device)
            self._topk(logits, k, None, val, idx)
            return K.sample_topk(val, idx, *args, seed, step=step, seed_dev=seed_dev)
        if logits.stride(0) % 8 != 0:
            logits = torch.nn.functional.pad(logits, (0, -logits.shape[1] % 8))[:, :logits.shape[1]]
        return K.sample_full(logits, args[0], k, args[1], args[2], seed, step=step, seed_dev=seed_dev)

    def _pick_next(self, s, cum, sampling):
        """Next token of every row of a tick from its logits ``cum``: the arg-max in ``s.best`` or a sample."""
        if sampling is None:
            return s.best
        kk = sampling["top_k"]
        if 0 < kk <= 128:
            self._topk(cum, kk, None, s.samp_v, s.samp_i)
            K.sample_topk(s.samp_v, s.samp_i, sampling["temperature"], sampling["top_p"], sampling["min_p"],
                          0, step=s.pos, out=s.sampled, seed_dev=s.seed_dev)
        else:
            # no top-k filter (the reference's default top_k=0) or a set wider than the sorted route holds
            K.sample_full(cum, sampling["temperature"], kk, sampling["top_p"], sampling["min_p"], 0, step=s.pos,
                          out=s.sampled, seed_dev=s.seed_dev)
        return s.sampled

    # ------------------------------------------------------------------------------------------
    # generate
    # ------------------------------------------------------------------------------------------
    BUCKETS = (1, 2, 4, 8, 16, 32, 64, 128, 256, 512, 1024)

    def bucket_rows(self, n: int) -> int:
        """Row count of the batch bucket that serves ``n`` requests (the engine keeps one set of tick buffers and
        one captured graph per bucket); exact under tensor parallelism or when bucketing is switched off."""
        if self.tp is not None or os.environ.get("TAH_B200_NO_BUCKETS", "0") == "1" or self.hard_override is not None:
            return n
        for b in self.BUCKETS:
            if b >= n:
                return b
        return n

    def _tick_state(self, B: int, max_new: int, sampling: Optional[dict], eos_token_id: Optional[int]):
        """Tick buffers + captured graph for this (rows, max_new, sampling, eos, hard mask) shape.  A repeat call
        with the same shape clears the scheduler state and replays the graph captured by the first one."""
        samp_key = None if sampling is None else (sampling["temperature"], sampling["top_p"], sampling["min_p"],
                                                  sampling["top_k"])
        ov = self.hard_override
        key = (B, max_new, samp_key, eos_token_id, None if ov is None else (ov.data_ptr(), tuple(ov.shape)))
        s = self._states.get(key)
        if s is None:
            if len(self._states) >= 4:                      # keep a handful of shapes (batch buckets)
                self._states.pop(next(iter(self._states)))
            s = self._alloc_tick_buffers(B, max_new)
            if sampling is not None and 0 < sampling["top_k"] <= 128:
                s.samp_v = torch.zeros(B, sampling["top_k"], dtype=torch.float32, device=self.device)
                s.samp_i = torch.zeros(B, sampling["top_k"], dtype=torch.int32, device=self.device)
            s.ints[8] = -1 if eos_token_id is None else int(eos_token_id)
            s.binding = K.TickStateBinding(s.tensors, s.ints)
            self._states[key] = s
        else:
            for t in (s.tok, s.depth, s.pos, s.finished, s.n_out, s.out_tokens, s.iter_sum, s.cur_iters, s.slot,
                      s.gate, s.tokens_done, s.need_soft, s.best, s.sampled):
                t.zero_()
        return s

    @torch.no_grad()
    def generate(self, input_ids: torch.Tensor, attention_mask: Optional[torch.Tensor] = None, *,
                 max_new_tokens: int = 128, do_sample: bool = False, temperature: float = 1.0, top_p: float = 1.0,
                 top_k: int = 0, min_p: float = 0.0, eos_token_id: Optional[int] = None, seed: Optional[int] = None,
                 max_ticks: Optional[int] = None, sync_every: int = 64, on_tick=None) -> GenerationResult:
        """Prefill + decode.  ``seed=None`` draws the sampling seed from torch's global generator, so
        ``set_all_seeds`` / ``torch.manual_seed`` govern it and successive calls differ (the reference's loop
        samples with ``torch.multinomial`` on the global generator, ``tah/model/utils.py:84-125``)."""
        dev = self.device
        input_ids = input_ids.to(dev)
        if attention_mask is not None:
            attention_mask = attention_mask.to(dev)
        B_user = input_ids.shape[0]
        B = self.bucket_rows(B_user)
        if B != B_user:
            # batch bucket: pad with copies of the first prompt (their output is dropped), so that batch sizes of one
            # bucket share tick buffers and the captured graph
            pad = B - B_user
            input_ids = torch.cat([input_ids, input_ids[:1].expand(pad, -1)], 0)
            if attention_mask is not None:
                attention_mask = torch.cat([attention_mask, attention_mask[:1].expand(pad, -1)], 0)
        ev = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
        ev[0].record()
        with nvtx_range("engine/prefill"):
            last_logits, lens, _ = self.prefill(input_ids, attention_mask, max_new_tokens)
        sampling = None
        if do_sample:
            if temperature <= 0:
                raise ValueError("sampling needs temperature > 0")
            if not (0 < top_k <= 128) and self.tp is not None:
                raise NotImplementedError("tensor-parallel engine sampling needs 0 < top_k <= 128 "
                                          "(the full-vocabulary sampler runs on one GPU)")
            sampling = dict(temperature=float(temperature), top_p=float(top_p), min_p=float(min_p), top_k=int(top_k))
            if seed is None:
                seed = int(torch.randint(0, 2 ** 62, (1,)).item())
        self._calls += 1
        s = self._tick_state(B, max_new_tokens, sampling, eos_token_id)
        if sampling is not None:
            s.seed_dev.fill_(int(seed) & (2 ** 62 - 1))
        # first token from the prefill logits
        first = self._choose(last_logits, lens.to(torch.int32) - 1, sampling, 0, s.seed_dev)
        s.pos.copy_(lens.to(torch.int32) - 1)
        s.need_soft.zero_()
        s.binding.tick_end(s.need_soft, first)          # emits token 1, pos = len, depth = 0
        s.cur_iters.zero_()
        ev[1].record()
        ticks = 0
        limit = max_ticks if max_ticks is not None else max_new_tokens * self.max_iter + 1
        if self.use_cuda_graph and limit > 0 and s.graph is None:
            self._tick(s, sampling)            # eager tick: lazy one-time kernel setup happens outside capture
            ticks = 1
            if on_tick is not None:
                on_tick(ticks, s)
        run = self._tick_runner(s, sampling)
        with nvtx_range("engine/decode"):
            while ticks < limit:
                run()
                ticks += 1
                if on_tick is not None:
                    on_tick(ticks, s)
                if ticks % sync_every == 0 or ticks == limit:
                    done = bool(((s.finished != 0) | (s.n_out >= max_new_tokens))[:B_user].all())
                    if done:
                        break
        ev[2].record()
        torch.cuda.synchronize()
        K.check_status(dev)
        n_out = s.n_out.tolist()
        out = s.out_tokens.tolist()
        iters = (s.iter_sum.float() / s.n_out.clamp(min=1).float()).tolist()
        out, n_out, iters = out[:B_user], n_out[:B_user], iters[:B_user]
        res = GenerationResult(tokens=[row[:n] for row, n in zip(out, n_out)], iter_counts=iters, ticks=ticks,
                               tokens_emitted=int(s.tokens_done.item()) if B == B_user else int(sum(n_out)),
                               prefill_ms=ev[0].elapsed_time(ev[1]),
                               decode_ms=ev[1].elapsed_time(ev[2]),
                               extra={"graph_captures": self.graph_captures, "graph_reuses": self.graph_reuses})
        self.last_counters = dict(engine_counters(self, res), graph_captures=self.graph_captures,
                                  graph_reuses=self.graph_reuses, rows=B)
        if self.metrics is not None:
            self.metrics.log(self.last_counters, step=self._calls)
        return res

    # ------------------------------------------------------------------------------------------
    # serving: request admission into free rows, pages returned on completion
    # ------------------------------------------------------------------------------------------
    @torch.no_grad()
    def serve(self, prompts: Sequence[torch.Tensor], *, max_new_tokens: int = 128, rows: Optional[int] = None,
              eos_token_id: Optional[int] = None, do_sample: bool = False, temperature: float = 1.0, top_p: float = 1.0,
              top_k: int = 0, min_p: float = 0.0, seed: Optional[int] = None, check_every: int = 16):
        """Continuous batching over a queue of requests (1-D token id tensors of any lengths).

        ``rows`` batch rows decode in lock step (one captured tick graph for that row count).  Every
        ``check_every`` ticks the host looks at the rows: a row whose request finished (EOS or ``max_new_tokens``)
        hands back its tokens, its KV pages of every depth return to the device free stacks, and the next queued
        request is admitted into the row - its prompt is prefilled into freshly assigned pages while the other rows
        keep their state - so the batch stays full while requests of different lengths come and go.  Returns the
        generated token lists in request order and a statistics dict (ticks, admissions, peak pages in use)."""
        dev = self.device
        if self.tp is not None:
            raise NotImplementedError("serve() runs on one GPU; use generate() under tensor parallelism")
        n_req = len(prompts)
        B = min(rows or self.max_rows, n_req, self.max_rows)
        longest = max(int(p.numel()) for p in prompts)
        sampling = None
        if do_sample:
            sampling = dict(temperature=float(temperature), top_p=float(top_p), min_p=float(min_p), top_k=int(top_k))
            if seed is None:
                seed = int(torch.randint(0, 2 ** 62, (1,)).item())

        def pad_batch(ps):
            T = max(int(p.numel()) for p in ps)
            ids = torch.zeros(len(ps), T, dtype=torch.long, device=dev)
            mask = torch.zeros(len(ps), T, dtype=torch.long, device=dev)
            for i, p in enumerate(ps):
                ids[i, T - p.numel():] = p.to(dev)
                mask[i, T - p.numel():] = 1
            return ids, mask

        def first_tokens(logits, lens):
            return self._choose(logits, lens.to(torch.int32) - 1, sampling, int(seed or 0), None)

        # the cache is sized for the longest request in every row
        ids, mask = pad_batch(prompts[:B])
        if self.kv is not None and (self.kv.rows != B or self.kv.max_pages[0] * self.page_size < longest + max_new_tokens + 1):
            self.kv = None
        if self.kv is None:
            self._new_cache(B, longest + max_new_tokens + 1)
        logits, lens, _ = self.prefill(ids, mask, max_new_tokens)
        self._calls += 1
        s = self._tick_state(B, max_new_tokens, sampling, eos_token_id)
        if sampling is not None:
            s.seed_dev.fill_(int(seed) & (2 ** 62 - 1))
        s.pos.copy_(lens.to(torch.int32) - 1)
        s.need_soft.zero_()
        s.binding.tick_end(s.need_soft, first_tokens(logits, lens))
        s.cur_iters.zero_()
        owner = list(range(B))                       # request index held by each row (-1 = idle)
        next_req = B
        results: List[Optional[List[int]]] = [None] * n_req
        stats = {"ticks": 0, "admitted": B, "rows": B, "peak_pages": [0] * self.kv.n_depths, "pages_released": 0}
        if self.use_cuda_graph and s.graph is None:
            self._tick(s, sampling)                  # lazy one-time kernel setup outside capture
            stats["ticks"] += 1
        run = self._tick_runner(s, sampling)
        budget = (n_req // B + 2) * (max_new_tokens * self.max_iter + check_every + 1)
        while any(o >= 0 for o in owner) and stats["ticks"] < budget:
            for _ in range(check_every):
                run()
            stats["ticks"] += check_every
            done = ((s.finished != 0) | (s.n_out >= max_new_tokens)).tolist()
            for d in range(self.kv.n_depths):
                stats["peak_pages"][d] = max(stats["peak_pages"][d], self.kv.pages_in_use(d))
            fin = [r for r in range(B) if done[r] and owner[r] >= 0]
            if not fin:
                continue
            n_out = s.n_out.tolist()
            toks = s.out_tokens[fin].tolist()
            for r, row_toks in zip(fin, toks):
                results[owner[r]] = row_toks[:n_out[r]]
                owner[r] = -1
            rows_t = torch.tensor(fin, device=dev)
            stats["pages_released"] += self.kv.free_rows(rows_t)
            take = min(len(fin), n_req - next_req)
            if take:
                rows_new = rows_t[:take]
                ids, mask = pad_batch(prompts[next_req:next_req + take])
                logits, lens, _ = self.prefill(ids, mask, max_new_tokens, row_ids=rows_new)
                first = first_tokens(logits, lens).to(torch.int32)
                # what tick_end does for a row that emits its first token
                hit_eos = (first == eos_token_id) if eos_token_id is not None else torch.zeros_like(first, dtype=torch.bool)
                s.out_tokens[rows_new] = 0
                s.out_tokens[rows_new, 0] = torch.where(hit_eos, torch.zeros_like(first), first)
                s.n_out[rows_new] = (~hit_eos).to(torch.int32)
                s.finished[rows_new] = hit_eos.to(torch.int32)
                s.tokens_done += int((~hit_eos).sum())
                s.tok[rows_new], s.depth[rows_new] = first, 0
                s.pos[rows_new] = lens.to(torch.int32)
                s.cur_iters[rows_new], s.iter_sum[rows_new], s.need_soft[rows_new] = 0, 0, 0
                for j in range(take):
                    owner[fin[j]] = next_req + j
                next_req += take
                stats["admitted"] += take
        torch.cuda.synchronize()
        K.check_status(dev)
        if any(r is None for r in results):
            raise RuntimeError("serve(): tick budget exhausted before every request finished")
        stats["tokens"] = sum(len(r) for r in results)
        return results, stats

    def _tick_runner(self, s, sampling):
        if not self.use_cuda_graph:
            def run_eager():
                before = K.launch_count
                self._tick(s, sampling)
                self.kernel_launches_per_tick = K.launch_count - before
            return run_eager
        if s.graph is not None:
            self.graph_reuses += 1
            return s.graph.replay
        # Capture records the launches of one tick without running them.  Everything a tick touches
        # was allocated beforehand, so replays reuse the same addresses.
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        graph = torch.cuda.CUDAGraph()
        before = K.launch_count
        with torch.cuda.stream(side):
            with torch.cuda.graph(graph, stream=side):
                self._tick(s, sampling)
        self.kernel_launches_per_tick = K.launch_count - before      # own kernels recorded in the graph
        torch.cuda.current_stream().wait_stream(side)
        s.graph = graph
        self.graph_captures += 1
        return graph.replay

    # ------------------------------------------------------------------------------------------
    # synthetic context (benchmarks)
    # ------------------------------------------------------------------------------------------
    @torch.no_grad()
    def fast_forward(self, s, context: int) -> None:
        """Benchmark aid: make every row look as if it had already processed ``context`` tokens, so that ticks
        can be timed at a chosen decode depth without generating up to it.  The page tables of every depth
        get the pages a row of that length owns (taken from the free stacks exactly as a tick would), the
        lengths and positions are advanced, and the skipped tokens are counted as emitted.  The K/V content of
        the skipped positions is whatever the pools hold (zeros after allocation): the kernels' work per tick
        depends on the lengths only.  Call between ticks, with no tick in flight."""
        kv, ps, dev = self.kv, self.page_size, self.device
        B = s.pos.shape[0]
        torch.cuda.synchronize()
        pos_new = torch.full_like(s.pos, int(context))
        delta = (pos_new - s.pos).clamp(min=0)
        targets = [pos_new + (s.depth > 0).to(torch.int32)]
        for d in range(1, kv.n_depths):
            if self.hard_override is not None:
                cnt = (self.hard_override[:B, :context] >= d).sum(1).to(torch.int32)
            else:
                cnt = kv.len[d].clone()
            targets.append(cnt + (s.depth > d).to(torch.int32))
        rows = torch.arange(B, device=dev)
        for d, tgt in enumerate(targets):
            tgt = torch.maximum(tgt, kv.len[d]).to(torch.int64)
            have = (kv.len[d].to(torch.int64) + ps - 1) // ps
            need = (tgt + ps - 1) // ps - have
            total, free = int(need.sum()), int(kv.free_count[d])
            if total > free or int(((tgt + ps - 1) // ps).max()) > kv.max_pages[d]:
                raise RuntimeError(f"KV pool of depth {d} too small for a context of {context} tokens")
            if total > 0:
                first = torch.cumsum(need, 0) - need
                row_of_page = torch.repeat_interleave(rows, need)
                rank = torch.arange(total, device=dev)
                page_ids = kv.free_stack[d][(free - 1 - rank)]
                col = have[row_of_page] + rank - first[row_of_page]
                kv.page_table[d][row_of_page, col] = page_ids
                kv.free_count[d].fill_(free - total)
            kv.len[d].copy_(tgt.to(torch.int32))
        s.n_out += delta
        s.tokens_done += int(delta.sum())
        s.pos.copy_(torch.maximum(pos_new, s.pos))
        torch.cuda.synchronize()
