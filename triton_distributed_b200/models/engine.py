"""Serving engine: prefill, then a CUDA-graph-captured decode step replayed per token.

API parity with ``python/triton_dist/models/engine.py:37-187``: ``Engine(model_config, temperature, top_p,
verbose, group)``, attributes ``backend`` / ``no_graph`` / ``enable_profile``, and ``serve(input_ids, gen_len)``.
The decode graph contains the whole forward (embedding to logits); sampling runs after each replay, as
in the reference (:164-177). ``start`` / ``extend`` are the step function underneath: the next tokens of every sequence in,
logits of any of them out, from the cache that earlier steps left.
"""
from __future__ import annotations

import time

import torch
import torch.distributed as dist

from ..kernels.allreduce import AllReduceMethod
from .auto import AutoLLM
from .config import ModelConfig
from .kv_cache import PagedCache
from .utils import logger, sample_token


class Engine:

    def __init__(self, model_config: ModelConfig, temperature: float = 0.6, top_p: float = 0.95, verbose: bool = False,
                 group=None, model=None):
        self.model_config = model_config
        self.temperature, self.top_p, self.verbose, self.group = temperature, top_p, verbose, group
        self.backend = "triton_dist_AR"      # decode backend: torch | triton_dist | triton_dist_AR
        self.prefill_backend = None          # None = same as `backend`
        self.no_graph = False
        self.enable_profile = False
        self.ar_method: AllReduceMethod | None = None
        self.model = model if model is not None else AutoLLM.from_pretrained(model_config, group)
        self.kv_cache: PagedCache | None = None
        self.graph = None
        self.bsz = None
        self.length = 0                      # tokens every sequence holds in the cache (host copy of its offsets)
        self._decode_cache = None            # the cache the decode step was prepared for

    # ------------------------------------------------------------------ set-up
    def _init_kv_cache(self, bsz: int) -> None:
        if self.kv_cache is None or self.kv_cache.batch_size != bsz:
            self.graph = self._decode_cache = None
            self.kv_cache = self.model.make_cache(bsz, self.model_config.max_length)
        self.kv_cache.clear()
        self.length = 0

    def _set_backend(self, backend: str, max_M: int) -> None:
        m = self.model
        if backend == "triton_dist":
            m.init_triton_dist_ctx(max_M)
        elif backend == "triton_dist_AR":
            m.init_triton_dist_AR_ctx(max_M, self.ar_method)
        m.set_fwd(backend)

    def _decode_step(self) -> None:
        self._static_pos.copy_(self.kv_cache.kv_offset.to(torch.int64)[:, None])
        self._static_logits = self.model.inference(self._static_ids, self._static_pos, self.kv_cache)

    def _init_cuda_graph(self) -> None:
        """Warm up on a side stream, then capture one decode step (static input / position / logits buffers)."""
        self.graph = None
        if self.no_graph:
            return
        state = self.kv_cache.save_state()  # the warm-up steps are not part of the sequences
        s = torch.cuda.Stream()
        s.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(s):
            for _ in range(3):
                self._decode_step()
        torch.cuda.current_stream().wait_stream(s)
        self.kv_cache.restore_state(state)
        torch.cuda.synchronize()
        if dist.is_initialized() and self.model_config.world_size > 1:
            dist.barrier(group=self.group)
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            self._decode_step()
        self.graph = g
        torch.cuda.synchronize()

    # ------------------------------------------------------------------ steps
    def start(self, bsz: int) -> None:
        """Begin `bsz` new sequences; what earlier ones held in the cache is given back."""
        self.bsz = bsz
        self._init_kv_cache(bsz)

    @torch.no_grad()
    def extend(self, input_ids: torch.Tensor, want: list[int] | None = None) -> torch.Tensor | None:
        """Run the next tokens [B, S] of every sequence. Returns fp32 logits [B, len(want), V] at the places `want` among
        these tokens (None: the last one; empty: the head is skipped and None returned). One token per sequence takes the
        captured decode step, several take the prefill path. The logits of a decode step are valid until the next one."""
        bsz, S = input_ids.shape
        if self.kv_cache is None or bsz != self.bsz:
            raise ValueError("start() the sequences first")
        if self.length + S > self.model_config.max_length:
            raise ValueError("the sequences would exceed max_length")
        logits = None
        if S == 1:
            if self._decode_cache is not self.kv_cache:
                self.prepare_decode(input_ids)
            elif self.graph is None:
                self._set_backend(self.backend, max(bsz, self.model_config.world_size))
            logits = self._run_decode(input_ids)
            if want is not None:
                logits = logits.expand(-1, len(want), -1) if want else None
        else:
            self._set_backend(self.prefill_backend or self.backend, bsz * S)
            pos = torch.arange(self.length, self.length + S, device=input_ids.device, dtype=torch.int64)[None, :].expand(bsz, S).contiguous()
            kw = {"kv_len": self.length + S}
            if want is None:
                logits = self.model.inference(input_ids, pos, self.kv_cache, **kw)
            else:
                hidden = self.model.inference(input_ids, pos, self.kv_cache, wo_lm_head=True, **kw)
                logits = self.model.lm_logits(hidden[:, want]) if want else None
        self.kv_cache.inc_offset(S)
        self.length += S
        return logits

    @torch.no_grad()
    def prefill(self, input_ids: torch.Tensor) -> torch.Tensor:
        self.start(input_ids.shape[0])
        return sample_token(self.extend(input_ids), self.temperature, self.top_p)

    @torch.no_grad()
    def prepare_decode(self, first_token: torch.Tensor) -> None:
        bsz = first_token.shape[0]
        self._set_backend(self.backend, max(bsz, self.model_config.world_size))
        self._static_ids = first_token.clone()
        self._static_pos = torch.zeros((bsz, 1), dtype=torch.int64, device=first_token.device)
        self._static_logits = None
        self._decode_cache = self.kv_cache
        self._init_cuda_graph()

    def _run_decode(self, token: torch.Tensor | None) -> torch.Tensor:
        """One decode step on the static buffers (`token` None: the ids already there); logits [B, 1, V]."""
        if token is not None:
            self._static_ids.copy_(token, non_blocking=True)
        if self.graph is not None:
            self.graph.replay()
        else:
            self._decode_step()
        return self._static_logits

    @torch.no_grad()
    def decode_one(self, token: torch.Tensor | None = None) -> torch.Tensor:
        """One decode step: feed `token` (default: the previously sampled one), return the next token ids [B, 1]."""
        nxt = sample_token(self._run_decode(token), self.temperature, self.top_p)
        self.kv_cache.inc_offset()
        self.length += 1
        self._static_ids.copy_(nxt)
        return nxt

    @torch.no_grad()
    def serve(self, input_ids: torch.Tensor, gen_len: int) -> torch.Tensor:
        """Prefill `input_ids` [B, S] and generate `gen_len` tokens. Returns [B, S + gen_len]."""
        if input_ids.shape[1] + gen_len > self.model_config.max_length:
            raise ValueError("prompt + generation exceeds max_length")
        t0 = time.time()
        nxt = self.prefill(input_ids)
        out = [input_ids, nxt]
        self.prepare_decode(nxt)
        torch.cuda.synchronize()
        t1 = time.time()
        prof = None
        if self.enable_profile:
            from ..utils import get_torch_prof_ctx
            prof = get_torch_prof_ctx(True)
            prof.__enter__()
        for _ in range(gen_len - 1):
            out.append(self.decode_one())
        torch.cuda.synchronize()
        from ..runtime.heap import get_heap, heap_initialized
        if heap_initialized():
            get_heap().check_status("Engine.serve")  # an expired wait means tokens computed from incomplete sums
        if prof is not None:
            prof.__exit__(None, None, None)
            prof.export_chrome_trace(f"decode_rank{self.model_config.rank}.json")
        t2 = time.time()
        if self.verbose and self.model_config.rank == 0:
            logger.info(f"prefill+setup {t1 - t0:.3f}s, decode {gen_len - 1} steps {t2 - t1:.3f}s "
                        f"({(t2 - t1) / max(gen_len - 1, 1) * 1e3:.3f} ms/step)")
        return torch.cat(out, dim=1)
