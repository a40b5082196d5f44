"""Paged engine for models that carry state besides keys and values.

:class:`StatefulSampler` is :class:`~arctic_platform_b200.engine.sampler.SamplerEngine` -- same admission, page
allocator, slots, sampling kernels, CUDA-graph decode loop, ``generate`` -- with the layers and their memory supplied by
the model through a small protocol (``models/registry.py`` lists the architectures):

* ``model.cache_layout()``       what each layer run keeps per sequence: paged K/V with its own head sizes (value size 0: key
                                 rows only; or the run whose pages it reads), an fp32 recurrent state and what else its recurrence carries
                                 (``aux``), the history of a short convolution (any of them may be absent);
* ``model.prepare_serving(n)``   tables for ``n`` positions;
* ``model.serve_rows(batch, cache)``   one pass over a ragged :class:`~arctic_platform_b200.ops.serving.StepBatch`,
                                 reading and advancing caches and states; the same code for prompts, portions, decoded
                                 tokens and any mixture;
* ``model.output_rows`` / ``model.logits``   final norm and head.

Keys and values live in the pages the base engine hands out; everything else lives in STATE SLOTS, one per sequence and
numbered like the decode rows.  A sequence that starts ignores what its slot held before, so slots need no clearing.
``n`` samples of one prompt share its full pages and get copies of its state.

Besides ``generate`` there is a step interface for callers that decide themselves which sequence advances when
(``open_sequence``, ``step``, ``close_sequence``): one call runs one ragged batch.  ``generate`` prefills through the same
step, in portions of at most ``prefill_tokens`` rows.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from ..models import registry
from ..ops.serving import PAGE, StepBatch, StepEntry
from ..utils.transfer_stats import to_device
from .sampler import SamplerEngine, _Seq


class StateCache:
    """Device memory of all layer runs: page pools, state slots, and the per-slot bookkeeping of a step."""

    def __init__(self, layout: List[Dict[str, tuple]], pages: int, slots: int, device, dtype: torch.dtype):
        self.k: List[Optional[torch.Tensor]] = []
        self.v: List[Optional[torch.Tensor]] = []
        self.state: List[Optional[torch.Tensor]] = []
        self.aux: List[Optional[torch.Tensor]] = []
        self.conv: List[Optional[torch.Tensor]] = []
        f32 = dict(device=device, dtype=torch.float32)
        for run in layout:
            kv, st, ax, cv = (run.get(n) for n in ("kv", "state", "aux", "conv"))
            if "kv_from" in run:                              # reads the pages an earlier run writes
                self.k.append(self.k[run["kv_from"]])
                self.v.append(self.v[run["kv_from"]])
                for kept in (self.state, self.aux, self.conv):
                    kept.append(None)
                continue
            # zero-filled: the unwritten tail of a last page is multiplied by weight 0 and must be finite
            self.k.append(torch.zeros((pages, kv[0], PAGE, kv[1]), device=device, dtype=dtype) if kv else None)
            self.v.append(torch.zeros((pages, kv[0], PAGE, kv[2]), device=device, dtype=dtype) if kv and kv[2] else None)
            self.state.append(torch.zeros((slots,) + tuple(st), **f32) if st else None)
            self.aux.append(torch.zeros((slots,) + tuple(ax), **f32) if ax else None)
            self.conv.append(torch.zeros((slots, 2) + tuple(cv), **f32) if cv and cv[0] else None)
        self.prev = torch.zeros(slots, device=device, dtype=torch.int32)      # last token fed
        self.parity = torch.zeros(slots, device=device, dtype=torch.int32)    # valid half of double-buffered state

    def _paged(self):
        return list({id(t): t for t in self.k + self.v if t is not None}.values())

    def _slotted(self):
        return [t for t in self.state + self.aux + self.conv if t is not None] + [self.prev, self.parity]

    def num_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._paged() + self._slotted())

    def copy_pages(self, src: torch.Tensor, dst: torch.Tensor) -> None:
        for t in self._paged():
            t[dst] = t[src]

    def copy_slots(self, src: torch.Tensor, dst: torch.Tensor) -> None:
        for t in self._slotted():
            t[dst] = t[src]


@dataclass
class _Open:
    length: int = 0
    pages: np.ndarray = field(default_factory=lambda: np.zeros(0, dtype=np.int32))


class StatefulSampler(SamplerEngine):
    MIN_PAGES = 1

    def __init__(self, cfg, device="cuda", model=None, *, prefill_tokens: int = 8192, dtype: Optional[torch.dtype] = None,
                 quantization: Optional[str] = None, tp_group=None, cascade: bool = False, **kw):
        if quantization:
            raise ValueError(f"{cfg.name}: the stateful engine serves {cfg.architecture} unquantised, got {quantization!r}")
        if tp_group is not None:
            raise NotImplementedError(f"{cfg.name}: {cfg.architecture} is served on one GPU per replica")
        if torch.device(device).type != "cuda":
            raise RuntimeError(f"{cfg.name}: {cfg.architecture} is served by CUDA kernels; no CUDA device was given")
        if model is None:
            model = registry.new_model(cfg, device, dtype or torch.bfloat16)
        self.prefill_tokens = int(prefill_tokens)
        self._open: Dict[int, _Open] = {}
        self._dropped: List[tuple] = []
        super().__init__(cfg, device, model=model, cascade=False, **kw)
        self._places = [p.data_ptr() for p in self.model.parameters()]

    # ------------------------------------------------------------------ memory
    def _alloc_cache(self) -> None:
        self.model.prepare_serving(self.max_seq_len)
        self.cache = StateCache(self.model.cache_layout(), self.num_pages, self.max_batch, self.device, self.model.dtype)
        from ..utils import memory_budget
        memory_budget.set_kv_resident(self.device, self.kv_bytes())

    def weights_updated(self) -> None:
        """A checkpoint may bring tensors of another size than the model was made with; captured steps hold the old addresses."""
        super().weights_updated()
        places = [p.data_ptr() for p in self.model.parameters()]
        if places != self._places:
            self._graphs.clear()
        self._places = places

    def _alloc_layer_buffers(self) -> None:
        self.d_slots = torch.full((self.max_batch,), -1, device=self.device, dtype=torch.int32)

    def kv_bytes(self) -> int:
        return self.cache.num_bytes() if self.cache is not None else 0

    def _cascade_on(self) -> bool:
        return False

    def _copy_pages(self, src, dst) -> None:
        self.cache.copy_pages(src, dst)

    def _fork_slots(self, forks) -> None:
        pairs = [(s, d) for s, others in forks for d in others]
        if pairs:
            t = torch.tensor(pairs, device=self.device)
            self.cache.copy_slots(t[:, 0], t[:, 1])

    # ------------------------------------------------------------------ steps
    @torch.no_grad()
    def _forward(self, entries: Sequence[StepEntry], on_layer=None) -> Tuple[StepBatch, torch.Tensor]:
        batch = StepBatch.build(entries, self.device)
        return batch, self.model.serve_rows(batch, self.cache, on_layer)

    def _rows_of(self, rows: Sequence[int]) -> torch.Tensor:
        return to_device(torch.tensor(list(rows), dtype=torch.int32), self.device)

    def _decode_logits(self, B: int) -> torch.Tensor:
        batch = StepBatch(B, B, self.d_tokens[:B], None, self.d_q_start[:B], self.d_active[:B], self.d_q_start[:B],
                          self.d_pos[:B], self.d_page_table, self.d_slots[:B])
        x = self.model.serve_rows(batch, self.cache)
        return self._output_logits(self.model.output_rows(x, None), self.d_logits[:B])

    def _output_logits(self, h, out=None):
        return self.model.logits(h, out)

    def _plan_portions(self, lens: Sequence[int]) -> List[List[Tuple[int, int, int]]]:
        """Cuts prompts of the given lengths into steps of at most ``prefill_tokens`` rows: per step a list of
        ``(prompt, first token, tokens)``, a prompt's portions in order and at most one of them in a step."""
        steps: List[List[Tuple[int, int, int]]] = [[]]
        room = self.prefill_tokens
        for i, n in enumerate(lens):
            at = 0
            while at < n:
                if room == 0:
                    steps.append([])
                    room = self.prefill_tokens
                take = min(room, n - at)
                steps[-1].append((i, at, take))
                at += take
                room -= take
        return [s for s in steps if s]

    @torch.no_grad()
    def _prefill_runs(self, runs: List[dict], prompts_np, live: Dict[int, _Seq]) -> torch.Tensor:
        """Prefills every admitted prompt once, in the slot of its first rollout; returns the final-norm hidden row of
        every prompt's last token, in the order of ``runs[*]["prompts"]``."""
        firsts = [(mem[0], live[mem[0]]) for run in runs for _gid, mem in run["prompts"]]
        pages = [np.concatenate([sq.shared_pages, sq.private_pages]) for _, sq in firsts]
        out: List[Optional[torch.Tensor]] = [None] * len(firsts)
        for portions in self._plan_portions([sq.prompt_len for _, sq in firsts]):
            entries = [StepEntry(firsts[i][0], prompts_np[firsts[i][1].req][at:at + n], at, pages[i])
                       for i, at, n in portions]
            batch, x = self._forward(entries)
            ends = [(i, int(batch.host[j, 0]) + n - 1) for j, (i, at, n) in enumerate(portions)
                    if at + n == firsts[i][1].prompt_len]
            if ends:
                h = self.model.output_rows(x, self._rows_of([r for _, r in ends]))
                for j, (i, _) in enumerate(ends):
                    out[i] = h[j]
        return torch.stack(out)

    def generate(self, prompts, sampling_params=None):
        if self._open:
            raise RuntimeError(f"{len(self._open)} sequences are open for stepping; close them before generate()")
        return super().generate(prompts, sampling_params)

    # ------------------------------------------------------------------ step interface
    def open_sequence(self) -> int:
        """Reserves a state slot for a new sequence."""
        if self._asleep:
            raise RuntimeError("sampler is asleep; call wake() first")
        slot = next((s for s in range(self.max_batch) if s not in self._open), None)
        if slot is None:
            raise RuntimeError(f"all {self.max_batch} state slots are in use")
        self._open[slot] = _Open()
        return slot

    def close_sequence(self, slot: int) -> None:
        """Gives the sequence's pages and its slot back."""
        self.pages.release(self._open.pop(slot).pages)

    @torch.no_grad()
    def step(self, work: Sequence[Tuple[int, Sequence[int], Sequence[int]]], on_layer=None) -> torch.Tensor:
        """One ragged batch: ``(slot, next tokens of its sequence, places among them whose logits are wanted)`` per
        sequence.  Returns fp32 logits ``[wanted places, V]`` in the order of ``work``."""
        need = {}
        for slot, tokens, want in work:
            sq = self._open[slot]
            if sq.length + len(tokens) > self.max_seq_len:
                raise ValueError(f"sequence of {sq.length + len(tokens)} tokens exceeds max_seq_len {self.max_seq_len}")
            if any(not 0 <= w < len(tokens) for w in want):
                raise ValueError("a wanted place lies outside the step's tokens")
            need[slot] = max(0, (sq.length + len(tokens) + PAGE - 1) // PAGE - len(sq.pages))
        if sum(need.values()) > self.pages.free_count():
            raise RuntimeError(f"KV cache too small: {sum(need.values())} pages needed, {self.pages.free_count()} free")
        entries, rows, at = [], [], 0
        for slot, tokens, want in work:
            sq = self._open[slot]
            if need[slot]:
                sq.pages = np.concatenate([sq.pages, self.pages.alloc(need[slot])])
            entries.append(StepEntry(slot, np.asarray(tokens, dtype=np.int64), sq.length, sq.pages))
            rows += [at + w for w in want]
            at += len(tokens)
        _, x = self._forward(entries, on_layer)
        for slot, tokens, _ in work:
            self._open[slot].length += len(tokens)
        if not rows:
            return torch.empty((0, self.cfg.vocab_size), device=self.device, dtype=torch.float32)
        return self._output_logits(self.model.output_rows(x, self._rows_of(rows)))

    @torch.no_grad()
    def score(self, prompts: Sequence[Sequence[int]], completions: Sequence[Sequence[int]], top_k: int = 1,
              portion: int = 1024):
        """Log-probabilities of given completions (teacher forcing), one list per sequence; ``top_k`` > 1 also returns the
        ``top_k`` most likely tokens per position, as ``{"log_probs": rows, "top_log_probs": [[{token: lp}]]}``."""
        rows, tops = [], []
        for prompt, comp in zip(prompts, completions):
            if len(prompt) == 0:
                raise ValueError("empty prompt")
            seq = [*prompt, *comp]
            slot, lp, top = self.open_sequence(), [], []
            try:
                for at in range(0, len(seq) - 1, portion):
                    part = seq[at:min(at + portion, len(seq) - 1)]
                    want = list(range(max(0, len(prompt) - 1 - at), len(part)))
                    z = self.step([(slot, part, want)])
                    if not want:
                        continue
                    z = torch.log_softmax(z, -1)
                    nxt = torch.tensor([seq[at + w + 1] for w in want], device=z.device)
                    lp += z.gather(1, nxt[:, None])[:, 0].tolist()
                    if top_k > 1:
                        v, i = torch.topk(z, int(top_k), dim=-1)
                        top += [dict(zip(ii, vv)) for ii, vv in zip(i.tolist(), v.tolist())]
            finally:
                self.close_sequence(slot)
            rows.append(lp)
            tops.append(top)
        return {"log_probs": rows, "top_log_probs": tops} if top_k > 1 else rows

    # ------------------------------------------------------------------ sleep / wake
    def sleep(self, level: int = 1) -> None:
        """Level 1 frees caches and states, level 2 the weights too (they come back with the next weight sync)."""
        if self._open:
            raise RuntimeError("sequences are open for stepping; close them before sleep()")
        self.cache = None
        self._graphs = {}
        if level >= 2:
            self._dropped = [(p, p.shape) for p in self.model.parameters()]
            for p, _ in self._dropped:
                p.data = torch.empty(0, device=self.device, dtype=p.dtype)
        self._asleep = True
        from ..utils import memory_budget
        memory_budget.set_kv_resident(self.device, 0)
        if level >= 2 or not memory_budget.shares_allocator(self.device):
            torch.cuda.empty_cache()

    def wake(self, tags: Optional[Sequence[str]] = None) -> None:
        tags = set(tags or ("weights", "kv_cache"))
        if "weights" in tags:
            for p, shape in self._dropped:           # zeros until the weights arrive (padding rows stay zero)
                p.data = torch.zeros(shape, device=self.device, dtype=p.dtype)
            self._dropped = []
        if "kv_cache" in tags:
            if self.cache is None:
                self._alloc_cache()
            self._asleep = False
