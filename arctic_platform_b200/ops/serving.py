"""Operations of a serving step over a ragged batch (CUDA only).

A step advances several sequences at once, each by its own run of new tokens: a portion of a prompt of any length, or
one decoded token.  :class:`StepBatch` is the device-side description of such a step; the functions below launch the
kernels of ``serve_*.cu``, ``retention*.cu``, ``ssm*.cu``, ``recurrent.cu``, ``*_mma.cu`` and ``gemm_*.cu`` on it.  They take bf16 or fp32 activations;
the residual streams and all carried state are fp32.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, field
from typing import Dict, Optional, Sequence, Tuple

import numpy as np
import torch

from . import _lib, gemm
from ..utils.transfer_stats import to_device

PAGE = 16               # tokens per KV page
NORM_ROWS = 8           # rows per block of the norm + convolution kernel

_FN: Dict[str, object] = {}


def _fn(name: str):
    if name not in _FN:
        c = ctypes
        vp, i, ll, f = c.c_void_p, c.c_int, c.c_longlong, c.c_float
        sigs = {
            "apb_embed_hash": [vp] * 9 + [ll, ll, ll, i, i, f, i, vp, vp, ll, vp, i, vp, i, i, vp],
            "apb_loop_begin": [vp, vp, i, i, vp, ll, i, vp],
            "apb_norm_conv": [vp] * 13 + [i, i, i, f, i, vp],
            "apb_gain_norm_rows": [vp, vp, vp, i, f, vp, i, i, i, f, i, vp],
            "apb_qk_norm_cache": [vp, ll, i, i, i, vp, vp, vp, i, i, i, i, i, f, i, vp],
            "apb_rope_cache": [vp, ll, i, i, i] + [vp] * 8 + [i, vp, vp] + [i] * 7 + [vp],
            "apb_stream_step": [vp] * 7 + [i] * 5 + [f, i, vp],
            "apb_softmax_attn": [vp, ll] + [vp] * 6 + [i, vp, vp, vp, ll] + [i] * 5 + [f, f, i, i, vp, f, f, i, vp, vp, ll, i, i, vp],
            "apb_softmax_attn_mma": [vp, ll] + [vp] * 4 + [i, vp, i, vp, vp, vp, ll, vp] + [i] * 7
                                    + [f, f, i, i, vp, f, f, i, vp, vp, ll, i, vp],
            "apb_row_norm_rope_cache": [vp, ll, i, i, i] + [vp] * 10 + [i, vp, vp] + [i] * 5 + [f, i, vp],
            "apb_residual_step": [vp] * 7 + [i, f] + [vp] * 5 + [i, i, i, f, f, i, i, vp, vp, vp, ll, i, vp, f, i, i, vp],
            "apb_half_rope_cache": [vp, ll, i, i, i] + [vp] * 8 + [i, vp, vp] + [i] * 5 + [f, i, vp],
            "apb_recurrent": [i, vp, vp] + [i] * 6 + [vp],
            "apb_memory_mma": [vp, i, i, vp, vp, vp, i, vp, vp, vp, vp, i, vp],
            "apb_delta_mma": [vp, vp, i, vp, i, vp, vp, vp],
            "apb_time_mix_mma": [vp, vp, i, vp, vp, i, vp, vp, vp, vp, i, vp],
            "apb_short_conv": [vp, ll, i, vp, vp, i, vp, vp, vp, ll, i] + [vp] * 5 + [i, i, vp],
            "apb_token_shift": [vp] * 10 + [i, i, i, vp, vp, i, i, vp, i, vp],
            "apb_tanh_rows": [vp, ll, i, i, i, vp],
            "apb_latent_norm_cache": [vp, ll, i, i] + [vp] * 11 + [i, i, i, i, i, f, i, vp],
            "apb_latent_rotate": [vp, ll] + [vp] * 8 + [i] * 6 + [vp],
            "apb_latent_gather": [vp, vp, i, vp, i, vp, vp, i, i, i, vp],
            "apb_moe_serve_route": [vp, ll, vp, vp, i, i, i, i] + [vp] * 9 + [i, i, i, i, i, vp],
            "apb_moe_serve_gather": [vp, i, ll, vp, vp, vp, i, vp, vp, vp],
            "apb_moe_serve_gather_scaled": [vp, i, i, vp, vp, vp, vp, i, vp, vp, i, vp],
            "apb_gemm_simt_grouped": [vp, vp, vp, i, i, i, ll, ll, ll, i, vp, ll, f, vp, i, vp, i, vp],
            "apb_gemm_bf16_grouped_glu": [vp, vp, i, i, i, ll, ll, i, f, vp, ll, vp, i, vp, ll, vp],
            "apb_gemm_simt_heads": [vp, vp, vp, i, i, i, i, ll, ll, ll, ll, ll, i, vp, ll, i, vp],
            "apb_gemm_bf16_grouped_dev": [vp, vp, vp, i, i, i, ll, ll, ll, i, f, vp, ll, vp, i, vp, ll, vp],
            "apb_gemm_bf16_heads": [vp, vp, vp, i, i, i, i, ll, ll, ll, i, i, i, vp, ll, vp],
            "apb_softmax_attn_wide": [vp, ll] + [vp] * 4 + [i, vp, i, vp, vp, ll, vp] + [i] * 7 + [f, i, vp, vp, ll, i, vp],
            "apb_flash_tc": [vp, ll, i, vp, i, vp, i, vp, ll, vp, vp, ll, ll, vp, ll] + [i] * 5 + [f, f, i, vp, vp, ll, i, vp],
            "apb_softmax_attn_tc": [vp, ll, i, vp, i, vp, i, vp, vp, i, vp, ll, i, i, i, i, f, f, vp, f, f, vp],
            "apb_ssm": [vp, ll, i, i, vp, vp, i] + [vp] * 6 + [ll] + [vp] * 7 + [i, vp] + [i] * 8 + [vp],
            "apb_ssm_mma": [vp, ll] + [vp] * 9 + [i, vp, vp, vp] + [i] * 5 + [vp],
            "apb_ssm_out": [vp, vp, ll, vp, vp, ll, i, i, i, f, i, vp],
            "apb_serve_commit": [vp] * 5 + [i, vp, vp, vp],
            "apb_sigmoid_attn": [vp, ll, vp, vp, vp, vp, vp, vp, i, vp, vp, vp, vp, ll, i, i, i, i, i, f, f, i, vp],
            "apb_sigmoid_attn_mma": [vp, ll, vp, vp, vp, vp, i, vp, i, vp, vp, vp, vp, ll, vp] + [i] * 7 + [f, f, vp],
            "apb_sigmoid_attn_tc": [vp, ll, i, vp, i, vp, i, vp, vp, i, vp, vp, ll, i, i, i, i, f, f, vp],
            "apb_retention": [vp, ll, i, i, i, i, vp, vp, i, vp, f, vp, vp, vp, ll, f, f, vp, vp, vp, vp, vp] + [i] * 8 + [vp],
            "apb_retention_mma": [vp, ll, i, i, i, vp, vp, i, vp, f] + [vp] * 7 + [i, vp, vp, i, vp, vp, i, i, i, i, vp],
            "apb_retention_out": [vp, ll, i, vp, vp, ll, f, f, vp, vp, vp, vp, vp, i, i, i, i, vp],
            "apb_gemm_simt": [vp, vp, vp, i, i, i, ll, ll, ll, i, vp, vp, ll, f, i, vp],
            "apb_gemm_bf16_glu": [vp, vp, i, i, i, ll, ll, i, f, vp, ll, vp],
        }
        _FN[name] = _lib.declare(name, sigs[name])
    return _FN[name]


def _call(name: str, *args) -> None:
    _lib.check(_fn(name)(*args, _lib.stream_ptr()), name)


def dtype_code(dtype: torch.dtype) -> int:
    if dtype == torch.bfloat16:
        return 0
    if dtype == torch.float32:
        return 1
    raise ValueError(f"the serving kernels take bfloat16 or float32, got {dtype}")


# --------------------------------------------------------------------------------------------- the batch
@dataclass
class StepEntry:
    """One sequence's part of a step: ``tokens`` continue the sequence in state slot ``slot`` at position ``pos0``;
    ``pages`` are its KV pages, in order, enough for ``pos0 + len(tokens)`` tokens."""
    slot: int
    tokens: np.ndarray
    pos0: int
    pages: np.ndarray


@dataclass
class StepBatch:
    rows: int
    n_entries: int
    tokens: torch.Tensor                   # [rows] int32
    row_entry: Optional[torch.Tensor]      # [rows], None: row i belongs to entry i
    start: torch.Tensor                    # [entries] first row, rows, state slot, position of the first row
    len: torch.Tensor
    slot: torch.Tensor
    pos0: torch.Tensor
    page_table: torch.Tensor               # [entries, max_pages]
    kv_slot: torch.Tensor                  # [rows] cache slot of every row (written by ``embed``)
    tiles: Optional[torch.Tensor] = None   # [n, 2] (entry, first row) of the norm + convolution blocks
    one_token: bool = True                 # some entry has exactly one row
    longer: bool = False                   # some entry has more than one row
    tables: Dict[tuple, torch.Tensor] = field(default_factory=dict)       # derived tables, on the device / host
    host_tables: Dict[tuple, dict] = field(default_factory=dict)
    host: Optional[np.ndarray] = None      # [entries, 4] start, len, slot, pos0 (None for a captured decode step)
    parts: Dict[tuple, "StepBatch"] = field(default_factory=dict)

    @staticmethod
    def plan(entries: Sequence[StepEntry]) -> Dict[str, np.ndarray]:
        """Host tables of a step: pure bookkeeping, no device involved."""
        lens = np.array([len(e.tokens) for e in entries], dtype=np.int32)
        if len(entries) == 0 or (lens <= 0).any():
            raise ValueError("every entry of a step brings at least one token")
        slots = np.array([e.slot for e in entries], dtype=np.int32)
        if len(set(slots.tolist())) != len(entries):
            raise ValueError("a sequence can take part in a step only once")
        start = np.concatenate([[0], np.cumsum(lens)[:-1]]).astype(np.int32)
        pos0 = np.array([e.pos0 for e in entries], dtype=np.int32)
        n_pages = [(e.pos0 + len(e.tokens) + PAGE - 1) // PAGE for e in entries]
        for e, n in zip(entries, n_pages):
            if len(e.pages) < n:
                raise ValueError(f"slot {e.slot}: {len(e.pages)} pages do not hold {e.pos0 + len(e.tokens)} tokens")
        table = np.zeros((len(entries), max(n_pages)), dtype=np.int32)
        for i, (e, n) in enumerate(zip(entries, n_pages)):
            table[i, :n] = e.pages[:n]
        tiles = np.array([(i, r) for i, n in enumerate(lens) for r in range(0, n, NORM_ROWS)], dtype=np.int32)
        return {"tokens": np.concatenate([np.asarray(e.tokens) for e in entries]).astype(np.int32),
                "row_entry": np.repeat(np.arange(len(entries), dtype=np.int32), lens), "start": start, "len": lens,
                "slot": slots, "pos0": pos0, "table": table, "tiles": tiles}

    @staticmethod
    def build(entries: Sequence[StepEntry], device) -> "StepBatch":
        p = StepBatch.plan(entries)
        names = ("tokens", "row_entry", "start", "len", "slot", "pos0", "table", "tiles")
        flat = torch.from_numpy(np.concatenate([p[n].reshape(-1) for n in names]))
        dev = to_device(flat.pin_memory(), device)                   # all tables of the step in one copy
        t, o = {}, 0
        for n in names:
            t[n] = dev[o:o + p[n].size].view(p[n].shape)
            o += p[n].size
        lens = p["len"]
        rows = int(lens.sum())
        return StepBatch(rows, len(entries), t["tokens"], t["row_entry"], t["start"], t["len"], t["slot"], t["pos0"],
                         t["table"], torch.empty(rows, device=device, dtype=torch.int32), t["tiles"],
                         bool((lens == 1).any()), bool((lens > 1).any()), host=np.stack([p["start"], lens, p["slot"], p["pos0"]], 1))

    def table(self, key, make) -> torch.Tensor:
        """Device copy of a host table derived from the batch, made once and shared by its layers."""
        if key not in self.tables:
            self.tables[key] = to_device(torch.from_numpy(make()).pin_memory(), self.tokens.device)
        return self.tables[key]

    def part(self, e0: int, e1: int) -> "StepBatch":
        """The entries ``[e0, e1)`` as a batch of their own over rows that start at 0 (views of this one)."""
        if self.host is None or (e0, e1) == (0, self.n_entries):
            return self
        if (e0, e1) not in self.parts:
            host = self.host[e0:e1].copy()
            r0, r1 = int(host[0, 0]), int(host[-1, 0] + host[-1, 1])
            host[:, 0] -= r0
            lens = host[:, 1]
            self.parts[e0, e1] = StepBatch(
                r1 - r0, e1 - e0, self.tokens[r0:r1], self.row_entry[r0:r1] - e0, self.start[e0:e1] - r0, self.len[e0:e1],
                self.slot[e0:e1], self.pos0[e0:e1], self.page_table[e0:e1], self.kv_slot[r0:r1], None,
                bool((lens == 1).any()), bool((lens > 1).any()), host=host)
        return self.parts[e0, e1]

    def entry_ptrs(self):
        return _lib.ptr(self.start), _lib.ptr(self.len), _lib.ptr(self.slot), _lib.ptr(self.pos0)


# --------------------------------------------------------------------------------------------- embedding and loop input
def embed(b: StepBatch, table: torch.Tensor, bigram: Optional[torch.Tensor], hash_spec: Optional[Tuple[int, int, int]],
          prev: torch.Tensor, x: torch.Tensor, x0: Optional[torch.Tensor] = None, scale: float = 1.0) -> None:
    """``x [rows, W]`` fp32 = (token rows + hashed bigram rows) * ``scale`` (``hash_spec`` = buckets, multiplier of the
    previous and of the current token); ``x [rows, streams, W]`` receives them once per stream, ``x0`` in the activation
    type.  Also fills ``b.kv_slot``."""
    V, W = table.shape
    buckets, mp, mc = hash_spec or (0, 0, 0)
    _call("apb_embed_hash", _lib.ptr(b.tokens), _lib.ptr(b.row_entry), *b.entry_ptrs(), _lib.ptr(prev), _lib.ptr(table),
          _lib.ptr(bigram), buckets, mp, mc, V, W, float(scale), x.shape[1] if x.dim() == 3 else 1, _lib.ptr(x), _lib.ptr(x0), 0 if x0 is None else x0.stride(0),
          _lib.ptr(b.page_table), b.page_table.stride(0), _lib.ptr(b.kv_slot), b.rows, dtype_code(table.dtype))


def loop_begin(x: torch.Tensor, init: torch.Tensor, out: torch.Tensor) -> None:
    """``out [rows, W]`` (a column slice) = ``x`` in the activation type; ``x`` = ``init [W]`` in every row."""
    _call("apb_loop_begin", _lib.ptr(x), _lib.ptr(init), x.shape[0], x.shape[1], _lib.ptr(out), out.stride(0),
          dtype_code(out.dtype))


# --------------------------------------------------------------------------------------------- norms and convolutions
def norm_conv(b: StepBatch, x: torch.Tensor, gain: torch.Tensor, w1: Optional[torch.Tensor],
              w2: Optional[torch.Tensor], two: bool, state: Optional[torch.Tensor], parity: torch.Tensor, taps: int,
              eps: float) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``h = x / rms(x) * gain`` and up to two causal depth-wise input convolutions of it: ``h + conv(h, w_k)`` with
    ``w_k [taps, W]`` (None: ``h``).  ``state [slots, 2, taps - 1, W]`` fp32 is the double-buffered history of ``h``."""
    T, W = x.shape
    o1 = torch.empty((T, W), device=x.device, dtype=gain.dtype)
    o2 = torch.empty_like(o1) if two else None
    n = b.n_entries if b.tiles is None else b.tiles.shape[0]
    _call("apb_norm_conv", _lib.ptr(x), _lib.ptr(gain), _lib.ptr(w1), _lib.ptr(w2), _lib.ptr(o1), _lib.ptr(o2),
          _lib.ptr(state), _lib.ptr(parity), *b.entry_ptrs(), _lib.ptr(b.tiles), n, W, taps, float(eps),
          dtype_code(gain.dtype))
    return o1, o2


def gain_norm_rows(x: torch.Tensor, rows: Optional[torch.Tensor], gain: torch.Tensor, eps: float,
                   offset: float = 0.0, groups: int = 1) -> torch.Tensor:
    """``x / rms(x) * (offset + gain)`` of some rows, in the activation type; rms over ``groups`` equal parts of a row."""
    n = x.shape[0] if rows is None else rows.shape[0]
    out = torch.empty((n, x.shape[1]), device=x.device, dtype=gain.dtype)
    _call("apb_gain_norm_rows", _lib.ptr(x), _lib.ptr(rows), _lib.ptr(gain), int(gain.numel() > 1), float(offset),
          _lib.ptr(out), n, x.shape[1], groups, float(eps),
          dtype_code(gain.dtype))
    return out


def qk_norm_cache(b: StepBatch, p: torch.Tensor, cols: Tuple[int, int, int], kcache: torch.Tensor, vcache: torch.Tensor,
                  heads: int, eps: float) -> None:
    """q and k columns of ``p`` divided by their root mean square per head (q in place), k and v into the page cache
    (``[pages, G, PAGE, D]`` and ``[pages, G, PAGE, E]``)."""
    G, D, E = kcache.shape[1], kcache.shape[3], vcache.shape[3]
    _call("apb_qk_norm_cache", _lib.ptr(p), p.stride(0), *cols, _lib.ptr(b.kv_slot), _lib.ptr(kcache), _lib.ptr(vcache),
          b.rows, heads, G, D, E, float(eps), dtype_code(p.dtype))


def rope_cache(b: StepBatch, p: torch.Tensor, cols: Tuple[int, ...], rope: Tuple[torch.Tensor, torch.Tensor], rot_dims: int,
               q_heads: int, dim: int, kcache: torch.Tensor, vcache: torch.Tensor, write: bool = True) -> None:
    """Rotates the first ``rot_dims`` of every ``dim`` columns of the q and k columns of ``p`` (neighbouring pairs); q in
    place, k and v into the page cache (``[pages, G, PAGE, maps * dim]`` and ``[pages, G, PAGE, E]``).  ``write`` False: q only."""
    G, E = kcache.shape[1], vcache.shape[3]
    q_col, k_col, v_col = (*cols, 0, 0)[:3]
    _call("apb_rope_cache", _lib.ptr(p), p.stride(0), q_col, k_col, v_col, _lib.ptr(b.row_entry), *b.entry_ptrs(),
          _lib.ptr(b.kv_slot), _lib.ptr(rope[0]), _lib.ptr(rope[1]), rot_dims, _lib.ptr(kcache), _lib.ptr(vcache), b.rows,
          q_heads, G * (kcache.shape[3] // dim) if write else 0, G, dim, E, dtype_code(p.dtype))


def row_norm_rope_cache(b: StepBatch, p: torch.Tensor, cols: Tuple[int, int, int], wq: torch.Tensor, wk: torch.Tensor,
                        rope: Tuple[torch.Tensor, torch.Tensor], rot_dims: int, heads: int, kcache: torch.Tensor,
                        vcache: torch.Tensor, eps: float) -> None:
    """q and k columns of ``p`` normed over the whole projection (weights ``wq``, ``wk``), then the first ``rot_dims`` of every
    head rotated (dimension i with i + rot_dims / 2); q in place, k and v into the page cache."""
    G, D, E = kcache.shape[1], kcache.shape[3], vcache.shape[3]
    _call("apb_row_norm_rope_cache", _lib.ptr(p), p.stride(0), *cols, _lib.ptr(wq), _lib.ptr(wk), _lib.ptr(b.row_entry),
          *b.entry_ptrs(), _lib.ptr(b.kv_slot), _lib.ptr(rope[0]), _lib.ptr(rope[1]), rot_dims, _lib.ptr(kcache), _lib.ptr(vcache),
          b.rows, heads, G, D, E, float(eps), dtype_code(p.dtype))


def half_rope_cache(b: StepBatch, p: torch.Tensor, cols: Tuple[int, int, int], rope: Tuple[torch.Tensor, torch.Tensor], rot_dims: int,
                    heads: int, kcache: torch.Tensor, vcache: torch.Tensor, value_eps: Optional[float] = None) -> None:
    """Rotates the first ``rot_dims`` of every query and key head of ``p`` (dimension i with i + rot_dims / 2); q in place, k and v into
    the page cache.  ``value_eps``: every value head is divided by its root mean square first."""
    G, D, E = kcache.shape[1], kcache.shape[3], vcache.shape[3]
    _call("apb_half_rope_cache", _lib.ptr(p), p.stride(0), *cols, _lib.ptr(b.row_entry), *b.entry_ptrs(), _lib.ptr(b.kv_slot),
          _lib.ptr(rope[0]), _lib.ptr(rope[1]), rot_dims, _lib.ptr(kcache), _lib.ptr(vcache), b.rows, heads, G, D, E,
          -1.0 if value_eps is None else float(value_eps), dtype_code(p.dtype))


# --------------------------------------------------------------------------------------------- normed residual
@dataclass
class ExpertMix:
    """Output of a mixture of experts that has not been summed yet: rows ``out [slots, W]`` of the routed experts with the
    rows ``slots [rows, top]`` (-1: none) and ``weights [rows, top]`` (None: all 1) of every token, and ``ident [rows]`` (None: 0)
    times its input."""
    out: torch.Tensor
    slots: torch.Tensor
    weights: Optional[torch.Tensor]
    ident: Optional[torch.Tensor]
    h: torch.Tensor


def residual_step(x: torch.Tensor, y: Optional[torch.Tensor], post: Optional[torch.Tensor], pre: Optional[torch.Tensor], eps: float,
                  *, mix: Optional[ExpertMix] = None, offset: float = 1.0, again: Optional[tuple] = None, write: bool = True,
                  clear: bool = False, dtype: Optional[torch.dtype] = None, y2: Optional[torch.Tensor] = None,
                  post2: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, gate_bias: Optional[torch.Tensor] = None,
                  mult: float = 1.0, groups: int = 1) -> torch.Tensor:
    """One pass over the residual ``x [rows, W]`` (fp32): ``x <- x + mult * sigmoid(gate + gate_bias) * s / rms(s) * (offset + post)``
    with ``s`` = ``y`` (fp32) plus the sum of ``mix`` (both may be absent; without ``post`` s itself), plus the same of a second output
    ``y2`` with ``post2`` under the same gate, plus the embedding output if ``again`` = (tokens, table, scale) is given; then
    ``x / rms(x) * (offset + pre)`` in the activation type (rms over ``groups`` equal parts), without ``pre`` the fp32 x.  ``gate``
    ``[rows, W]`` columns in fp32 or the activation type (None: 1).  ``write`` False leaves ``x`` as it was; ``clear`` zeroes ``y`` and
    ``y2`` after reading them."""
    T, W = x.shape
    dt = next((t.dtype for t in (pre, post, gate_bias) if t is not None), dtype)
    out = torch.empty((T, W), device=x.device, dtype=dt if pre is not None else torch.float32)
    tok, table, scale = again or (None, None, 0.0)
    m = (mix.out, mix.slots, mix.weights, mix.ident, mix.h) if mix is not None else (None,) * 5
    _call("apb_residual_step", _lib.ptr(x), _lib.ptr(y), _lib.ptr(post), _lib.ptr(pre), _lib.ptr(out), _lib.ptr(tok), _lib.ptr(table),
          0 if table is None else table.shape[0], float(scale), *(_lib.ptr(t) for t in m), 0 if mix is None else mix.slots.shape[1],
          T, W, float(offset), float(eps), int(write), int(clear), _lib.ptr(y2), _lib.ptr(post2), _lib.ptr(gate),
          0 if gate is None else gate.stride(0), int(gate is not None and gate.dtype == torch.float32), _lib.ptr(gate_bias), float(mult),
          groups, dtype_code(dt or torch.float32))
    return out


# --------------------------------------------------------------------------------------------- parallel residual streams
def stream_step(x: torch.Tensor, y: Optional[torch.Tensor], mix: Optional[torch.Tensor], out_w: Optional[torch.Tensor],
                in_w: Optional[torch.Tensor], gain: Optional[torch.Tensor], eps: float, *, write: bool = True,
                clear: bool = False, dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """One pass over the streams ``x [rows, S, W]`` (fp32): ``x_t <- sum_s mix[s, t] x_s + out_w[t] y`` (``y`` None: left
    alone), then ``u = sum_t in_w[t] x_t`` (None: the plain sum) and ``u / rms(u) * gain`` in the activation type -- without
    ``gain`` the fp32 ``u``.  ``write`` False leaves ``x`` as it was; ``clear`` zeroes ``y`` after reading it."""
    T, S, W = x.shape
    dt = gain.dtype if gain is not None else (dtype or (in_w if in_w is not None else mix).dtype)
    h = torch.empty((T, W), device=x.device, dtype=dt if gain is not None else torch.float32)
    _call("apb_stream_step", _lib.ptr(x), _lib.ptr(y), _lib.ptr(mix), _lib.ptr(out_w), _lib.ptr(in_w), _lib.ptr(gain),
          _lib.ptr(h), T, W, S, int(write), int(clear), float(eps), dtype_code(dt))
    return h


def commit(b: StepBatch, prev: torch.Tensor, parity: torch.Tensor) -> None:
    """End of a step: last tokens of the entries, parity of the double-buffered states."""
    _call("apb_serve_commit", _lib.ptr(b.tokens), *b.entry_ptrs(), b.n_entries, _lib.ptr(prev), _lib.ptr(parity))


# --------------------------------------------------------------------------------------------- products
def linear(a: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, *, accumulate: bool = False,
           out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``a [M, K] @ w [N, K]^T``.  ``accumulate``: added onto fp32 ``out`` (few rows: cut along K over the SMs)."""
    M, K = a.shape
    N = w.shape[0]
    if out is None:
        out = torch.empty((M, N), device=a.device, dtype=out_dtype or a.dtype)
    f32_out = out.dtype == torch.float32
    if _simt(a, w, out):
        epi = gemm.EPI_F32_ACCUM if accumulate else (gemm.EPI_F32 if f32_out else gemm.EPI_BF16)
        _gemm_simt(a, w, out, epi)
        return out
    if accumulate:
        tiles = ((M + 127) // 128) * ((N + 127) // 128)
        splits = max(1, min(_sm_count(a.device) // tiles, (K + 63) // 64))
        gemm.gemm_raw(a, w, out, M=M, N=N, K=K, epi=gemm.EPI_F32_ATOMIC if splits > 1 else gemm.EPI_F32_ACCUM,
                      splits=splits, bn=128 if splits > 1 else 0)
    else:
        gemm.gemm_raw(a, w, out, M=M, N=N, K=K, epi=gemm.EPI_F32 if f32_out else gemm.EPI_BF16)
    return out


def accumulates(rows: int, width: int, device) -> bool:
    """Whether :func:`project` may add parts of its products into the output, which then has to start as zeros."""
    return 2 * ((rows + 127) // 128) * ((width + 127) // 128) <= _sm_count(device)


def project(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
    """``out [M, N]`` fp32 = ``a @ w^T``; few rows: cut along K over the SMs and added onto ``out``, which holds zeros."""
    linear(a, w, out, accumulate=accumulates(a.shape[0], w.shape[0], a.device) and not _simt(a, w, out))


def gate_up(x: torch.Tensor, w_gu: torch.Tensor, out: torch.Tensor, epi: int, limit: float = 0.0) -> None:
    """``out [M, ff]`` (may be a column slice) = the GLU ``epi`` of the products; gate and up rows interleaved in ``w_gu``."""
    M, K = x.shape
    N = w_gu.shape[0]
    if _simt(x, w_gu, out) or N % 16:
        _gemm_simt(x, w_gu, None, epi, out2=out, limit=limit)
    else:
        _call("apb_gemm_bf16_glu", _lib.ptr(x), _lib.ptr(w_gu), M, N, K, x.stride(0), w_gu.stride(0), epi, float(limit),
              _lib.ptr(out), out.stride(0))


def gate_up_gelu(x: torch.Tensor, w_gu: torch.Tensor, out: torch.Tensor) -> None:
    """gelu_tanh(gate) * up."""
    gate_up(x, w_gu, out, gemm.EPI_GEGLU)


def gate_up_silu(x: torch.Tensor, w_gu: torch.Tensor, out: torch.Tensor) -> None:
    """silu(gate) * up."""
    gate_up(x, w_gu, out, gemm.EPI_SWIGLU)


def gate_up_clamped(x: torch.Tensor, w_gu: torch.Tensor, out: torch.Tensor, limit: float) -> None:
    """g sigmoid(1.702 g) (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit)."""
    gate_up(x, w_gu, out, gemm.EPI_CLAMP_GLU, limit)


_SMS: Dict[int, int] = {}


def _sm_count(device) -> int:
    i = torch.device(device).index or 0
    if i not in _SMS:
        _SMS[i] = torch.cuda.get_device_properties(i).multi_processor_count
    return _SMS[i]


def _simt(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> bool:
    """fp32 operands, or rows the TMA-fed kernels cannot address (not a multiple of 16 bytes)."""
    return (a.dtype == torch.float32 or bool(a.stride(0) % 8 or w.stride(0) % 8 or w.shape[0] % 8 or out.stride(0) % 8)
            or bool((a.data_ptr() | w.data_ptr() | out.data_ptr()) & 15))


def _gemm_simt(a, w, out, epi, out2=None, limit=0.0) -> None:
    _call("apb_gemm_simt", _lib.ptr(a), _lib.ptr(w), _lib.ptr(out), a.shape[0], w.shape[0], a.shape[1], a.stride(0),
          w.stride(0), 0 if out is None else out.stride(0), epi, None, _lib.ptr(out2),
          0 if out2 is None else out2.stride(0), float(limit), dtype_code(a.dtype))


def heads_linear(a: torch.Tensor, a_step: int, w: torch.Tensor, heads: int, k: int, out: torch.Tensor, out_step: int,
                 gate: Optional[torch.Tensor] = None) -> None:
    """Product per head: ``out[:, h out_step + n] = a[:, h a_step + k] w[h N + n, k]``, optionally times the sigmoid of ``gate``
    (laid out like ``out``).  Behind a head's ``k`` columns ``a`` holds finite values."""
    N = w.shape[0] // heads
    gp, gs = (_lib.ptr(gate), gate.stride(0)) if gate is not None else (None, 0)
    epi = gemm.EPI_SIGMOID_GATE if gate is not None else gemm.EPI_BF16
    odd = _simt(a, w, out) or N % 8 or a_step % 8 or out_step % 8
    if gate is not None:
        odd = odd or gate.stride(0) % 8 or gate.data_ptr() & 15
    args = (_lib.ptr(a), _lib.ptr(w), _lib.ptr(out), a.shape[0], N, k, heads, a.stride(0), w.stride(0), out.stride(0), a_step,
            out_step, epi, gp, gs)
    if odd:
        _call("apb_gemm_simt_heads", *args, dtype_code(a.dtype))
    else:
        _call("apb_gemm_bf16_heads", *args)


# --------------------------------------------------------------------------------------------- mixture of experts
def experts(b: StepBatch, h: torch.Tensor, logits: torch.Tensor, correction: Optional[torch.Tensor], counters: torch.Tensor,
            w_gu: torch.Tensor, w_down: torch.Tensor, n: int, n_experts: int, top: int, ff: int, *, sigmoid: bool = False,
            scale_input: bool = False, epi: int = gemm.EPI_SWIGLU, limit: float = 0.0) -> ExpertMix:
    """Routes every row of ``h`` by its fp32 ``logits`` (``n`` scores -- their softmax, or with ``sigmoid`` each one's sigmoid --, the
    first ``n_experts`` of them experts with weights, the others identity experts) and runs the experts, GLU layers with the activation
    ``epi``, as two grouped products.  ``w_gu [experts * 2 ff, W]`` (gate and up interleaved), ``w_down [experts * W, >= ff]``;
    ``counters [experts + 1]`` int32 are zero between calls.  ``scale_input``: a token's weight multiplies the expert's input instead
    of its output (no identity experts)."""
    T, W = h.shape
    dev, E, P = h.device, n_experts, T * top
    I, ldf = 2 * ff, w_down.shape[1]
    simt = h.dtype == torch.float32 or bool(W % 8 or I % 16 or w_gu.stride(0) % 8 or ldf % 8)
    tile = 64 if simt else 128
    blocks = (P + tile - 1) // tile + min(E, P)
    max1, max2 = blocks * ((I + tile - 1) // tile), blocks * ((W + tile - 1) // tile)
    i32 = dict(device=dev, dtype=torch.int32)
    f32 = dict(device=dev, dtype=torch.float32)
    o1 = (3 * P + E + 2 + 3) // 4 * 4                                             # tile tables on 16-byte boundaries
    ints = torch.empty(o1 + 4 * (max1 + max2), **i32)                             # one allocation for all tables
    expert, rank, slots = (ints[i * P:(i + 1) * P].view(T, top) for i in range(3))
    first, n_tiles = ints[3 * P:3 * P + E], ints[3 * P + E:3 * P + E + 2]
    tiles1, tiles2 = ints[o1:o1 + 4 * max1], ints[o1 + 4 * max1:o1 + 4 * (max1 + max2)]
    weights, ident = torch.empty((T, top), **f32), torch.empty(T, **f32)
    _call("apb_moe_serve_route", _lib.ptr(logits), logits.stride(0), _lib.ptr(correction), _lib.ptr(b.kv_slot), T, n, E, top,
          _lib.ptr(expert), _lib.ptr(rank), _lib.ptr(weights), _lib.ptr(ident), _lib.ptr(counters), _lib.ptr(first), _lib.ptr(tiles1),
          _lib.ptr(tiles2), _lib.ptr(n_tiles), I, W, tile, int(sigmoid), dtype_code(h.dtype))
    xs = torch.empty((P, W), device=dev, dtype=h.dtype)
    if scale_input:
        _call("apb_moe_serve_gather_scaled", _lib.ptr(h), T, W, _lib.ptr(expert), _lib.ptr(rank), _lib.ptr(first), _lib.ptr(weights), top,
              _lib.ptr(slots), _lib.ptr(xs), dtype_code(h.dtype))
    else:
        _call("apb_moe_serve_gather", _lib.ptr(h), T, W * h.element_size(), _lib.ptr(expert), _lib.ptr(rank), _lib.ptr(first), top,
              _lib.ptr(slots), _lib.ptr(xs))
    act = (torch.zeros if ldf != ff else torch.empty)((P, ldf), device=dev, dtype=h.dtype)
    out = torch.empty((P, W), device=dev, dtype=h.dtype)
    n1, n2 = _lib.ptr(n_tiles), _lib.ptr(n_tiles[1:])
    if simt:
        dt = dtype_code(h.dtype)
        _call("apb_gemm_simt_grouped", _lib.ptr(xs), _lib.ptr(w_gu), None, P, I, W, W, w_gu.stride(0), 0, epi, _lib.ptr(act),
              ldf, float(limit), _lib.ptr(tiles1), max1, n1, dt)
        _call("apb_gemm_simt_grouped", _lib.ptr(act), _lib.ptr(w_down), _lib.ptr(out), P, W, ff, ldf, w_down.stride(0), W, gemm.EPI_BF16,
              None, 0, 0.0, _lib.ptr(tiles2), max2, n2, dt)
    else:
        _call("apb_gemm_bf16_grouped_glu", _lib.ptr(xs), _lib.ptr(w_gu), P, I, W, W, w_gu.stride(0), epi, float(limit), _lib.ptr(act), ldf,
              _lib.ptr(tiles1), max1, n1, w_gu.shape[0])
        _call("apb_gemm_bf16_grouped_dev", _lib.ptr(act), _lib.ptr(w_down), _lib.ptr(out), P, W, ff, ldf, w_down.stride(0), W,
              gemm.EPI_BF16, 1.0, None, 0, _lib.ptr(tiles2), max2, n2, w_down.shape[0])
    return ExpertMix(out, slots, None, None, h) if scale_input else ExpertMix(out, slots, weights, ident, h)


# --------------------------------------------------------------------------------------------- sequence mixers
SHORT_ROWS = 16         # entries up to this length take the few-query tiles, longer ones the tcgen05 kernel
MAX_SPLITS = 8


def tile_work(host: np.ndarray, heads: int, kv_heads: int, min_len: int, tile: int = 128) -> np.ndarray:
    """Work items of the tcgen05 attention kernel for the entries of at least ``min_len`` rows, longest key range
    first: ``[n, 12]`` int32 = entry, key blocks, KV head, 0, then for each of two groups (first row, valid rows, head,
    keys visible to the first row).  The groups are two query heads of the KV head on the same row tile; a head left over
    pairs two consecutive row tiles (``valid = 0``: no second group)."""
    R = heads // kv_heads
    parts = []
    for en, (start, n, _slot, pos0) in enumerate(host.tolist()):
        if n < min_len:
            continue
        t = np.arange(0, n, tile)
        rows, valid, keys = start + t, np.minimum(tile, n - t), pos0 + t + 1
        last = keys + valid - 1                                              # keys visible to a tile's last row

        def items(rows0, valid0, keys0, h0, rows1, valid1, keys1, h1, seen):
            m = len(rows0)
            it = np.zeros((kv_heads, m, 12), dtype=np.int64)
            g = np.arange(kv_heads)[:, None]
            it[..., 0], it[..., 1], it[..., 2] = en, (seen + tile - 1) // tile, g
            for o, (r, v, h, k) in ((4, (rows0, valid0, h0, keys0)), (8, (rows1, valid1, h1, keys1))):
                it[..., o], it[..., o + 1], it[..., o + 2], it[..., o + 3] = r, v, g * R + h, k
            parts.append(it.reshape(-1, 12))

        for h in range(0, R - 1, 2):
            items(rows, valid, keys, h, rows, valid, keys, h + 1, last)
        if R % 2:
            a, b = slice(0, None, 2), slice(1, None, 2)
            odd = len(t) % 2
            second = [np.concatenate([x[b], x[-1:] * 0]) if odd else x[b] for x in (rows, valid, keys, last)]
            items(rows[a], valid[a], keys[a], R - 1, second[0], second[1], second[2], R - 1, np.maximum(last[a], second[3]))
    if not parts:
        return np.zeros((0, 12), dtype=np.int32)
    work = np.concatenate(parts)
    return np.ascontiguousarray(work[np.argsort(-work[:, 1], kind="stable")], dtype=np.int32)


def sigmoid_attention(b: StepBatch, q: torch.Tensor, heads: int, kcache: torch.Tensor, vcache: torch.Tensor,
                      bias: torch.Tensor, scale: float, out: torch.Tensor, out_scale: float = 1.0) -> None:
    """``q [rows, heads * D]`` (column slice) over the entries' pages -> ``out [rows, heads * E]`` (column slice).
    bf16 with head sizes that are multiples of 8 runs on tensor cores; fp32 and odd sizes on CUDA cores."""
    G, D, E = kcache.shape[1], kcache.shape[3], vcache.shape[3]
    aligned = not (D % 8 or E % 8 or q.stride(0) % 8 or out.stride(0) % 8 or (q.data_ptr() | out.data_ptr()) & 15)
    if q.dtype != torch.bfloat16 or not aligned or max(D, E) > 256:
        _call("apb_sigmoid_attn", _lib.ptr(q), q.stride(0), _lib.ptr(b.row_entry), *b.entry_ptrs(),
              _lib.ptr(b.page_table), b.page_table.stride(0), _lib.ptr(kcache), _lib.ptr(vcache), _lib.ptr(bias),
              _lib.ptr(out), out.stride(0), b.rows, heads, G, D, E, float(scale), float(out_scale), dtype_code(q.dtype))
        return
    lens = np.ones(1, dtype=np.int64) if b.host is None else b.host[:, 1]
    limit = SHORT_ROWS if max(D, E) <= 128 else int(lens.max())
    short = lens[lens <= limit]
    if len(short):
        longest = int(short.max())
        passes = min(256, (longest * (heads // G) + 15) // 16)
        splits = max(1, min(MAX_SPLITS, 2 * _sm_count(q.device) // (b.n_entries * G * passes)))
        part = torch.empty((b.n_entries, longest, heads, splits, E), device=q.device, dtype=torch.float32) \
            if splits > 1 else None
        _call("apb_sigmoid_attn_mma", _lib.ptr(q), q.stride(0), *b.entry_ptrs(), b.n_entries, _lib.ptr(b.page_table),
              b.page_table.stride(0), _lib.ptr(kcache), _lib.ptr(vcache), _lib.ptr(bias), _lib.ptr(out), out.stride(0),
              _lib.ptr(part), heads, G, D, E, 1, longest, splits, float(scale), float(out_scale))
    if len(short) < len(lens):
        work = b.table(("sigmoid", heads, G), lambda: tile_work(b.host, heads, G, limit + 1))
        _call("apb_sigmoid_attn_tc", _lib.ptr(q), q.stride(0), b.rows, _lib.ptr(work), work.shape[0],
              _lib.ptr(b.page_table), b.page_table.stride(0), _lib.ptr(kcache), _lib.ptr(vcache), kcache.shape[0],
              _lib.ptr(bias), _lib.ptr(out), out.stride(0), heads, G, D, E, float(scale), float(out_scale))


@dataclass(frozen=True)
class SoftmaxSpec:
    """Softmax attention over the page cache: ``score = scale q.k``, capped to ``cap tanh(score / cap)`` (0: no cap), chunks of
    ``chunk`` positions and windows of the last ``window`` positions (0: none).  ``maps`` 2: differential attention,
    ``out = o / rms(o) * post_scale`` with ``o = a1 - lambda a2``."""
    scale: float
    cap: float = 0.0
    chunk: int = 0
    maps: int = 1
    post_scale: float = 1.0
    eps: float = 1e-5
    window: int = 0


MAX_FIXED_CAP = 64.0    # the tcgen05 kernel's bound on the score cap


def chunk_tiles(host: np.ndarray, heads: int, kv_heads: int, min_len: int, chunk: int, tile: int = 128) -> np.ndarray:
    """Work items of the tcgen05 softmax kernel for the entries of at least ``min_len`` rows, longest key range first:
    ``[n, 8]`` int32 = entry, KV head, head, first row, valid rows, position of the first row, first key of the walk (a
    multiple of ``PAGE``), first visible key.  No tile leaves its first row's chunk."""
    parts = []
    for en, (start, n, _slot, pos0) in enumerate(host.tolist()):
        if n < min_len:
            continue
        at, end = [pos0], pos0 + n
        if chunk:
            at += range((pos0 // chunk + 1) * chunk, end, chunk)
        at = np.array(at, dtype=np.int64)                                       # first positions of the runs
        runs = np.diff(np.append(at, end))
        per = -(-runs // tile)
        base = np.repeat(at, per)
        pos = base + (np.arange(per.sum()) - np.repeat(np.cumsum(per) - per, per)) * tile
        valid = np.minimum(tile, np.repeat(at + runs, per) - pos)
        first = pos // chunk * chunk if chunk else np.zeros_like(pos)
        it = np.empty((heads, len(pos), 8), dtype=np.int64)
        h = np.arange(heads)[:, None]
        it[..., 0], it[..., 1], it[..., 2] = en, h // (heads // kv_heads), h
        it[..., 3], it[..., 4], it[..., 5] = start + pos - pos0, valid, pos
        it[..., 6], it[..., 7] = first // PAGE * PAGE, first
        parts.append(it.reshape(-1, 8))
    if not parts:
        return np.zeros((0, 8), dtype=np.int32)
    work = np.concatenate(parts)
    return np.ascontiguousarray(work[np.argsort(work[:, 6] - work[:, 5] - work[:, 4], kind="stable")], dtype=np.int32)


def flash_fits(dim: int, rot: int, vdim: int) -> bool:
    """Whether the tcgen05 kernel with a running reference takes heads of these sizes."""
    return dim % 16 == 0 and rot % 16 == 0 and vdim % 8 == 0 and vdim <= 128 and -(-dim // 64) + -(-rot // 64) <= 4


def flash_tiles(host: np.ndarray, heads: int, kv_heads: int, min_len: int, window: int, base: Optional[np.ndarray] = None,
                tile: int = 128) -> np.ndarray:
    """Work items of the tcgen05 kernel with a running reference for the entries of at least ``min_len`` rows, longest key range
    first: ``[n, 12]`` int32 = entry, KV head, first key of the walk (a multiple of ``PAGE``), ``base`` of the entry, then for
    each of two tiles (first row, valid rows, head, position of the first row).  The tiles are two query heads of a KV head on the
    same rows; a head left over pairs consecutive row tiles (``valid = 0``: no second tile)."""
    R = heads // kv_heads
    parts = []
    for en, (start, n, _slot, pos0) in enumerate(host.tolist()):
        if n < min_len:
            continue
        t = np.arange(0, n, tile)
        rows, valid, pos = start + t, np.minimum(tile, n - t), pos0 + t

        def items(sel0, h0, sel1, h1):
            a = [x[sel0] for x in (rows, valid, pos)]
            c = [x[sel1] for x in (rows, valid, pos)]
            m, m1 = len(a[0]), len(c[0])
            it = np.zeros((kv_heads, m, 12), dtype=np.int64)
            g = np.arange(kv_heads)[:, None]
            it[..., 0], it[..., 1], it[..., 3] = en, g, 0 if base is None else base[en]
            it[..., 2] = (np.maximum(0, a[2] - window + 1) if window else np.zeros_like(a[2])) // PAGE * PAGE
            it[..., 4], it[..., 5], it[..., 6], it[..., 7] = a[0], a[1], g * R + h0, a[2]
            it[:, :m1, 8], it[:, :m1, 9], it[:, :m1, 10], it[:, :m1, 11] = c[0], c[1], g * R + h1, c[2]
            parts.append(it.reshape(-1, 12))

        for h in range(0, R - 1, 2):
            items(slice(None), h, slice(None), h + 1)
        if R % 2:
            items(slice(0, None, 2), R - 1, slice(1, None, 2), R - 1)
    if not parts:
        return np.zeros((0, 12), dtype=np.int32)
    work = np.concatenate(parts)
    keys = np.maximum(work[:, 7] + work[:, 5], work[:, 11] + work[:, 9]) - work[:, 2]
    return np.ascontiguousarray(work[np.argsort(-keys, kind="stable")], dtype=np.int32)


def shared_row(dim: int, vdim: int, dtype: torch.dtype) -> int:
    """Columns of a cache row of ``dim`` key columns whose first ``vdim`` are the values.  Where the tensor-core kernel takes the
    sizes: padded to a multiple of 16 (zeros) and by 8 more, which spreads the rows over the shared-memory banks."""
    fits = dtype == torch.bfloat16 and dim % 8 == 0 and vdim % 8 == 0 and dim <= 640 and vdim <= 512
    return (dim + 15) // 16 * 16 + 8 if fits else dim


MAX_WIDE_SPLITS = 16


def wide_splits(blocks: int, sms: int) -> int:
    """Key splits of the wide-row kernel (one CTA per SM): full waves, against the cost of writing and merging the parts."""
    return min(range(1, MAX_WIDE_SPLITS + 1), key=lambda s: -(-blocks * s // sms) / s + 0.04 * (s - 1) * blocks / sms)


def softmax_attention(b: StepBatch, q: torch.Tensor, heads: int, kcache: torch.Tensor, vcache: Optional[torch.Tensor],
                      spec: SoftmaxSpec, lam: Optional[torch.Tensor], out: torch.Tensor, *, dim: int = 0, vdim: int = 0,
                      sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, gate_cols: int = 1) -> None:
    """``q [rows, heads * maps * D]`` (column slice, rotated) over the entries' pages -> ``out [rows, heads * E]`` (column
    slice).  Without a ``vcache`` the values are the first ``vdim`` of the ``dim`` columns of the key rows (:func:`shared_row`).  ``sink [heads]`` fp32: a score per
    head that counts in the denominator only; ``gate``: columns of the activations whose sigmoid multiplies the output, one per
    head (``gate_cols`` 1) or one per output column (``gate_cols`` E).
    bf16 with head sizes that are multiples of 8 runs on tensor cores; fp32 and odd sizes on CUDA cores."""
    G, DK = kcache.shape[1], kcache.shape[3]
    E = vdim if vcache is None else vcache.shape[3]
    D = DK // spec.maps if vcache is not None else dim
    shape = (float(spec.scale), float(spec.cap), spec.chunk, spec.maps, _lib.ptr(lam), float(spec.post_scale), float(spec.eps))
    tail = shape + (spec.window, _lib.ptr(sink), _lib.ptr(gate), 0 if gate is None else gate.stride(0), gate_cols)
    aligned = not (D % 8 or E % 8 or q.stride(0) % 8 or out.stride(0) % 8 or (q.data_ptr() | out.data_ptr()) & 15)
    wide = vcache is None and DK > D
    if not wide and (vcache is None or q.dtype != torch.bfloat16 or not aligned or max(DK, E) > 256):
        _call("apb_softmax_attn", _lib.ptr(q), q.stride(0), _lib.ptr(b.row_entry), *b.entry_ptrs(), _lib.ptr(b.page_table),
              b.page_table.stride(0), _lib.ptr(kcache), _lib.ptr(vcache), _lib.ptr(out), out.stride(0), b.rows, heads, G, D, E,
              *tail, dtype_code(q.dtype))
        return
    plain = spec.maps == 1 and not spec.chunk
    tc = spec.maps == 2 and D % 16 == 0 and D <= 64 and E <= 128 and 0 < spec.cap <= MAX_FIXED_CAP
    flash = plain and vcache is not None and flash_fits(D, 0, E) and not out.data_ptr() & 15
    lens = np.ones(1, dtype=np.int64) if b.host is None else b.host[:, 1]
    limit = SHORT_ROWS if tc or flash else int(lens.max())
    short = lens[lens <= limit]
    if len(short):
        longest = int(short.max())
        f32 = dict(device=q.device, dtype=torch.float32)
        if wide:
            splits = wide_splits(b.n_entries * G * -(-longest * (heads // G) // 32), _sm_count(q.device))
            part = torch.empty((b.n_entries, longest, heads, splits, E + 2), **f32) if splits > 1 else None
            _call("apb_softmax_attn_wide", _lib.ptr(q), q.stride(0), *b.entry_ptrs(), b.n_entries, _lib.ptr(b.page_table),
                  b.page_table.stride(0), _lib.ptr(kcache), _lib.ptr(out), out.stride(0), _lib.ptr(part), heads, G, D, E, 1, longest,
                  splits, float(spec.scale), *tail[7:])
        else:
            passes = min(256, (longest * (heads // G) * spec.maps + 15) // 16)
            splits = max(1, min(MAX_SPLITS, 2 * _sm_count(q.device) // (b.n_entries * G * passes)))
            part = torch.empty((b.n_entries, longest, heads, spec.maps, splits, E + 2), **f32) if splits > 1 else None
            _call("apb_softmax_attn_mma", _lib.ptr(q), q.stride(0), *b.entry_ptrs(), b.n_entries, _lib.ptr(b.page_table),
                  b.page_table.stride(0), _lib.ptr(kcache), _lib.ptr(vcache), _lib.ptr(out), out.stride(0), _lib.ptr(part), heads, G,
                  D, E, 1, longest, splits, *tail)
    if len(short) == len(lens):
        return
    if flash:
        work = b.table(("flash", heads, G, spec.window), lambda: flash_tiles(b.host, heads, G, limit + 1, spec.window))
        _call("apb_flash_tc", _lib.ptr(q), q.stride(0), b.rows, _lib.ptr(work), work.shape[0], _lib.ptr(b.page_table),
              b.page_table.stride(0), _lib.ptr(kcache), D, None, _lib.ptr(vcache), E, kcache.shape[0] * G * PAGE, _lib.ptr(out),
              out.stride(0), heads, G, D, 0, E, float(spec.scale), float(spec.cap), *tail[7:])
    else:
        work = b.table(("softmax", heads, G, spec.chunk), lambda: chunk_tiles(b.host, heads, G, limit + 1, spec.chunk))
        _call("apb_softmax_attn_tc", _lib.ptr(q), q.stride(0), b.rows, _lib.ptr(work), work.shape[0], _lib.ptr(b.page_table),
              b.page_table.stride(0), _lib.ptr(kcache), _lib.ptr(vcache), kcache.shape[0], _lib.ptr(out), out.stride(0), heads,
              G, D, E, *shape[:2], *shape[4:])


# --------------------------------------------------------------------------------------------- latent attention
@dataclass(frozen=True)
class LatentSpec:
    """Latent attention: heads of ``dim`` plain and ``rot`` rotated query / key columns and ``vdim`` value columns; the cache
    keeps ``rank`` latent and ``rot`` rotated key columns per token, shared by all heads."""
    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int
    scale: float


def latent_norm_cache(b: StepBatch, p: torch.Tensor, q_col: int, c_col: int, q_gain: torch.Tensor, c_gain: torch.Tensor,
                      rope: Tuple[torch.Tensor, torch.Tensor], cache: torch.Tensor, eps: float, rot: int) -> None:
    """Norm of the query latent (columns ``q_col`` of ``p``, in place) and of the key / value latent (``c_col``), rotation of the
    shared key part of ``rot`` columns behind it; both go to the page cache ``[pages, 1, PAGE, >= rank + rot]``."""
    Q, C = q_gain.numel(), c_gain.numel()
    _call("apb_latent_norm_cache", _lib.ptr(p), p.stride(0), q_col, c_col, _lib.ptr(q_gain), _lib.ptr(c_gain), _lib.ptr(b.row_entry),
          *b.entry_ptrs(), _lib.ptr(b.kv_slot), _lib.ptr(rope[0]), _lib.ptr(rope[1]), _lib.ptr(cache), cache.shape[3],
          b.rows, Q, C, rot, float(eps), dtype_code(p.dtype))


def latent_rotate(b: StepBatch, q: torch.Tensor, s: LatentSpec, rope: Tuple[torch.Tensor, torch.Tensor],
                  dst: Optional[torch.Tensor] = None) -> None:
    """Rotates the rotated part of every head of ``q [rows, heads * (dim + rot)]``, in place or into the last ``rot`` columns of
    the heads of ``dst [rows, heads * (rank + rot)]``."""
    _call("apb_latent_rotate", _lib.ptr(q), q.stride(0), _lib.ptr(b.row_entry), *b.entry_ptrs(), _lib.ptr(rope[0]), _lib.ptr(rope[1]),
          _lib.ptr(dst), b.rows, s.heads, s.dim, s.rot, s.rank, dtype_code(q.dtype))


def entry_runs(host: Optional[np.ndarray], n_entries: int, limit: int) -> list:
    """Maximal runs ``(e0, e1)`` of neighbouring entries of at most ``limit`` rows (no host table: all entries are single rows)."""
    if host is None:
        return [(0, n_entries)]
    out, e0 = [], None
    for e, n in enumerate(host[:, 1].tolist() + [limit + 1]):
        if n <= limit and e0 is None:
            e0 = e
        elif n > limit and e0 is not None:
            out.append((e0, e))
            e0 = None
    return out


LATENT_ROWS = 32        # entries up to this length work on the latents themselves
EXPAND_TOKENS = 65536   # tokens of context whose keys and values are expanded at a time (a longer entry alone)


def expansion_plan(host: np.ndarray, heads: int, min_len: int, budget: int = EXPAND_TOKENS) -> list:
    """Groups of the entries of at least ``min_len`` rows whose contexts are expanded together: ``pages [n, 4]`` int32 (entry,
    page of the entry, first row of the copy, tokens) for the gather kernel and ``work`` (:func:`flash_tiles`)."""
    groups, at = [], 0
    for en, (_start, n, _slot, pos0) in enumerate(host.tolist()):
        if n < min_len:
            continue
        size = -(-(pos0 + n) // PAGE) * PAGE
        if not groups or at + size > budget:
            groups.append([])
            at = 0
        groups[-1].append((en, at, size))
        at += size
    plans = []
    for group in groups:
        base = np.zeros(len(host), dtype=np.int64)
        mine = host.copy()
        mine[:, 1] = 0
        for en, row, _ in group:
            base[en], mine[en, 1] = row, host[en, 1]
        pages = [np.stack([np.full(size // PAGE, en), np.arange(size // PAGE), row + np.arange(0, size, PAGE),
                           np.full(size // PAGE, PAGE)], 1) for en, row, size in group]
        plans.append({"pages": np.concatenate(pages).astype(np.int32), "work": flash_tiles(mine, heads, heads, min_len, 0, base)})
    return plans


def latent_attention(b: StepBatch, q: torch.Tensor, s: LatentSpec, cache: torch.Tensor, w_absorb: torch.Tensor,
                     w_expand: torch.Tensor, sink: Optional[torch.Tensor], gate: Optional[torch.Tensor],
                     rope: Tuple[torch.Tensor, torch.Tensor], out: torch.Tensor) -> None:
    """``q [rows, heads * (dim + rot)]`` (not rotated yet) over the entries' latents -> ``out [rows, heads * vdim]`` (column
    slice), times the sigmoid of the ``gate`` columns.  ``w_expand`` holds the key rows (heads * dim) and, from the next multiple of
    8 on, the value rows (heads * vdim) over the latent, ``w_absorb [heads * rank, dim]`` the key rows transposed per head.

    Short entries work on the latents: the key projection is applied to the query and the value projection to the weighted sum.
    Long ones expand the keys and values of all heads from the latents of their whole context first."""
    H, D, R, C, E = s.heads, s.dim, s.rot, s.rank, s.vdim
    spec = SoftmaxSpec(s.scale)
    v_col = (H * D + 7) // 8 * 8
    w_value = w_expand[v_col:][:H * E]
    gated = [] if gate is None else [gate]
    aligned = not (C % 8 or any(t.stride(0) % 8 or t.data_ptr() & 15 for t in [q, out] + gated))
    expand = b.host is not None and q.dtype == torch.bfloat16 and aligned and flash_fits(D, R, E) and R > 0
    limit = LATENT_ROWS if expand else b.rows
    for e0, e1 in entry_runs(b.host, b.n_entries, limit):
        p = b.part(e0, e1)
        r0 = 0 if b.host is None else int(b.host[e0, 0])
        rows = slice(r0, r0 + p.rows)
        ql = torch.empty((p.rows, H * (C + R)), device=q.device, dtype=q.dtype)
        heads_linear(q[rows], D + R, w_absorb, H, D, ql, C + R)
        latent_rotate(p, q[rows], s, rope, ql)
        o = torch.empty((p.rows, H * C), device=q.device, dtype=q.dtype)
        softmax_attention(p, ql, H, cache, None, spec, None, o, dim=C + R, vdim=C, sink=sink)
        heads_linear(o, C, w_value, H, C, out[rows], E, None if gate is None else gate[rows])
    if not expand or not (b.host[:, 1] > limit).any():
        return
    latent_rotate(b, q, s, rope)
    key = ("expanded", H)
    if key not in b.host_tables:
        b.host_tables[key] = expansion_plan(b.host, H, limit + 1)
    for n, plan in enumerate(b.host_tables[key]):
        pages, work = (b.table(key + (n, t), lambda t=t: plan[t]) for t in ("pages", "work"))
        keys = plan["pages"].shape[0] * PAGE
        latents, rotated = (torch.empty((keys, w), device=q.device, dtype=q.dtype) for w in (C, R))
        _call("apb_latent_gather", _lib.ptr(cache), _lib.ptr(pages), pages.shape[0], _lib.ptr(b.page_table), b.page_table.stride(0),
              _lib.ptr(latents), _lib.ptr(rotated), cache.shape[3], C, R)
        kv = linear(latents, w_expand[:, :C])
        v = kv[:, v_col:]
        _call("apb_flash_tc", _lib.ptr(q), q.stride(0), b.rows, _lib.ptr(work), work.shape[0], None, 0, _lib.ptr(kv), kv.stride(0),
              _lib.ptr(rotated), _lib.ptr(v), kv.stride(0), keys, _lib.ptr(out), out.stride(0), H, H, D, R, E, float(s.scale), 0.0, 0,
              _lib.ptr(sink), _lib.ptr(gate), 0 if gate is None else gate.stride(0), E)


MIN_SEGMENT = 256       # tokens; a multiple of the kernel's chunk


def segment_plan(host: np.ndarray, slices: int, slots: int) -> Dict[str, object]:
    """Cuts entries longer than one row into segments so that about ``slots`` blocks (``slices`` per segment) run at
    once.  ``seg [n, 6]``: entry, first token, tokens, scratch state before the segment (-1: none), scratch state for its
    contribution (-1: none), last of its entry.  ``chains [m, 4]``: entry, first scratch state, segments, first segment --
    for the entries of more than one segment."""
    work = [(en, int(n)) for en, n in enumerate(host[:, 1]) if n > 1]
    want, size = slots // slices, max(n for _, n in work)
    if want >= 3 * len(work):            # fewer: the extra pass over the states costs more than it frees
        lo, hi = 1, -(-size // 32)       # the smallest segment (in chunks of 32) that needs no second wave of blocks
        while lo < hi:
            mid = (lo + hi) // 2
            if sum(-(-n // (mid * 32)) for _, n in work) <= want:
                hi = mid
            else:
                lo = mid + 1
        size = max(MIN_SEGMENT, lo * 32)
    seg, chains, states = [], [], 0
    for en, n in work:
        k = -(-n // size)
        step = -(-(-(-n // k)) // 32) * 32 if k > 1 else n
        k = -(-n // step)
        if k > 1:
            chains.append((en, states, k, len(seg)))
        for i in range(k):
            last = i + 1 == k
            seg.append((en, i * step, min(step, n - i * step), states + i if k > 1 else -1,
                        -1 if last else states + i + 1, int(last)))
        states += k if k > 1 else 0
    return {"seg": np.array(seg, dtype=np.int32).reshape(-1, 6), "states": states,
            "chains": np.array(chains, dtype=np.int32).reshape(-1, 4)}


def segments(b: StepBatch, slices: int):
    """``(plan, seg, chains)`` of :func:`segment_plan` for two blocks per SM, the tables on the device (``chains`` None: no entry has
    several segments)."""
    key = ("segments", slices)
    if key not in b.host_tables:
        b.host_tables[key] = segment_plan(b.host, slices, 2 * _sm_count(b.tokens.device))
    plan = b.host_tables[key]
    return plan, b.table(key + ("seg",), lambda: plan["seg"]), b.table(key + ("chains",), lambda: plan["chains"]) if len(plan["chains"]) else None


def retention(b: StepBatch, p: torch.Tensor, cols: Tuple[int, int, int, int], rope: Tuple[torch.Tensor, torch.Tensor],
              rot_dims: int, log2_decay: torch.Tensor, state: torch.Tensor, out: torch.Tensor, eps: float,
              k_scale: float, out_scale: float = 1.0) -> None:
    """Retention of the q, k, v columns of ``p`` with the carried ``state [slots, H, D, E]`` (fp32), per-head norm, the
    silu gate of the g columns; ``out [rows, H * E]`` (column slice)."""
    _, H, D, E = state.shape
    scratch = torch.empty((b.rows, H, E), device=p.device, dtype=torch.float32) if b.longer else None
    aligned = not (D % 8 or E % 8 or p.stride(0) % 8 or p.data_ptr() & 15 or any(c % 8 for c in cols))
    mma = b.longer and p.dtype == torch.bfloat16 and aligned and D <= 128
    if b.one_token or not mma:
        _call("apb_retention", _lib.ptr(p), p.stride(0), *cols, _lib.ptr(rope[0]), _lib.ptr(rope[1]), rot_dims,
              _lib.ptr(log2_decay), float(k_scale), _lib.ptr(state), _lib.ptr(scratch), _lib.ptr(out), out.stride(0),
              float(out_scale), float(eps), _lib.ptr(b.row_entry), *b.entry_ptrs(), b.n_entries, b.rows, H, D, E,
              int(b.one_token), int(b.longer and not mma), dtype_code(p.dtype))
    if mma:
        slices = H * ((E + 63) // 64)
        plan, seg, chains = segments(b, slices)
        qk = torch.empty((b.rows, H, 4, (D + 15) // 16 * 16), device=p.device, dtype=torch.bfloat16)
        carry = torch.empty((plan["states"], H, D, E), device=p.device, dtype=torch.float32) if plan["states"] else None
        _call("apb_retention_mma", _lib.ptr(p), p.stride(0), *cols[:3], _lib.ptr(rope[0]), _lib.ptr(rope[1]), rot_dims,
              _lib.ptr(log2_decay), float(k_scale), _lib.ptr(state), _lib.ptr(scratch), *b.entry_ptrs(), _lib.ptr(seg),
              len(plan["seg"]), _lib.ptr(carry), _lib.ptr(chains), len(plan["chains"]), _lib.ptr(b.row_entry), _lib.ptr(qk),
              b.rows, H, D, E)
        _call("apb_retention_out", _lib.ptr(p), p.stride(0), cols[3], _lib.ptr(scratch), _lib.ptr(out), out.stride(0),
              float(out_scale), float(eps), _lib.ptr(b.row_entry), *b.entry_ptrs(), b.rows, H, E, dtype_code(p.dtype))


SSM_ROWS = 16           # rows per block of the state-space mixer's convolution


def row_tiles(host: np.ndarray, rows: int) -> np.ndarray:
    """``[n, 2]`` int32 (entry, first row) of the blocks of up to ``rows`` rows of the entries longer than one row."""
    return np.array([(en, r) for en, n in enumerate(host[:, 1].tolist()) if n > 1 for r in range(0, n, rows)], dtype=np.int32)


@dataclass(frozen=True)
class SsmWeights:
    """Parameters of a state-space mixer besides its projections: ``conv [taps, channels]``, ``conv_bias [channels]``, and per
    head ``dt_bias``, ``a_log``, ``skip``."""
    conv: torch.Tensor
    conv_bias: torch.Tensor
    dt_bias: torch.Tensor
    a_log: torch.Tensor
    skip: torch.Tensor


def state_space(b: StepBatch, p: torch.Tensor, xbc_col: int, dt_col: int, w: SsmWeights, groups: int, hist: Optional[torch.Tensor],
                parity: torch.Tensor, state: torch.Tensor) -> torch.Tensor:
    """Convolution, step sizes and recurrence over the columns ``[x | B | C]`` and ``dt`` of ``p`` with the carried
    ``state [slots, H, N, E]`` and convolution history ``hist [slots, 2, taps - 1, channels]`` (fp32); ``y [rows, H * E]`` fp32,
    before the gate."""
    _, H, N, E = state.shape
    taps, channels = w.conv.shape
    y = torch.empty((b.rows, H * E), device=p.device, dtype=torch.float32)
    ldx = (channels + 7) // 8 * 8
    xbc = torch.empty((b.rows, ldx), device=p.device, dtype=p.dtype) if b.longer else None
    steps = torch.empty((b.rows, H, 2), device=p.device, dtype=torch.float32) if b.longer else None
    tiles = b.table(("rows", SSM_ROWS), lambda: row_tiles(b.host, SSM_ROWS)) if b.longer else None
    mma = b.longer and p.dtype == torch.bfloat16 and N % 8 == 0 and E % 8 == 0 and N <= 128
    _call("apb_ssm", _lib.ptr(p), p.stride(0), xbc_col, dt_col, _lib.ptr(w.conv), _lib.ptr(w.conv_bias), taps, _lib.ptr(hist),
          _lib.ptr(parity), _lib.ptr(w.dt_bias), _lib.ptr(w.a_log), _lib.ptr(w.skip), _lib.ptr(xbc), ldx, _lib.ptr(steps),
          _lib.ptr(state), _lib.ptr(y), *b.entry_ptrs(), b.n_entries, _lib.ptr(tiles),
          tiles.shape[0] if b.longer else 0, H, E, groups, N, int(b.one_token), int(b.longer and not mma), dtype_code(p.dtype))
    if mma:
        slices = H * ((E + 63) // 64)
        plan, seg, chains = segments(b, slices)
        f32 = dict(device=p.device, dtype=torch.float32)
        carry = torch.empty((plan["states"], H, N, E), **f32) if plan["states"] else None
        decay = torch.empty((len(plan["seg"]), H), **f32) if plan["states"] else None
        _call("apb_ssm_mma", _lib.ptr(xbc), ldx, _lib.ptr(steps), _lib.ptr(w.skip), _lib.ptr(state), _lib.ptr(y),
              *b.entry_ptrs(), _lib.ptr(seg), len(plan["seg"]), _lib.ptr(carry), _lib.ptr(decay), _lib.ptr(chains),
              len(plan["chains"]), H, E, groups, N)
    return y


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, gain: torch.Tensor, parts: int, eps: float, out: torch.Tensor) -> None:
    """``out [rows, n]`` (column slice) = ``v / rms(v) * gain`` in ``parts`` equal parts of every row, ``v = y silu(z)``;
    ``y`` fp32, ``z`` a column slice in the activation type."""
    _call("apb_ssm_out", _lib.ptr(y), _lib.ptr(z), z.stride(0), _lib.ptr(gain), _lib.ptr(out), out.stride(0), y.shape[0],
          y.shape[1], parts, float(eps), dtype_code(out.dtype))


# --------------------------------------------------------------------------------------------- matrix states per head
CHUNK = 32              # tokens per chunk of the tensor-core kernels
MAX_MMA_STATE = 128     # rows of a state that they hold in registers


def first_tiles(host: np.ndarray, rows: int) -> np.ndarray:
    """``[m, 2]`` int32 (entry, index of its first block in :func:`row_tiles`) of the entries longer than one row."""
    out, at = [], 0
    for en, n in enumerate(host[:, 1].tolist()):
        if n > 1:
            out.append((en, at))
            at += -(-n // rows)
    return np.array(out, dtype=np.int32)


def segment_chunks(host: np.ndarray, seg: np.ndarray) -> np.ndarray:
    """Index of the first chunk (in :func:`row_tiles`) of every segment of a :func:`segment_plan`."""
    first = dict(first_tiles(host, CHUNK).tolist())
    return np.array([first[en] + t // CHUNK for en, t in seg[:, :2].tolist()], dtype=np.int32)


RULES = {"memory": 0, "delta": 1, "time_mix": 2}


@dataclass(frozen=True)
class RecurrentSpec:
    """A mixer with an fp32 state ``[dim, vdim]`` per head (``csrc/recurrent.cuh`` has the recurrences): ``rule`` "memory" (matrix
    memory with exponential gates capped at ``cap``), "delta" (gated delta rule behind a short convolution) or "time_mix" (decay per
    key channel, bonus for the current token).  The head's output is normed, multiplied by a gain (``shared_gain``: one of ``vdim``
    for all heads) and by the silu (else the sigmoid) of the gate columns."""
    rule: str
    heads: int
    key_heads: int
    dim: int
    vdim: int
    eps: float
    cap: float = 0.0
    silu: bool = True
    shared_gain: bool = False

    @property
    def channels(self) -> int:
        return 2 * self.key_heads * self.dim + self.heads * self.vdim


@dataclass
class RecurrentInputs:
    """Projections and weights of a recurrent mixer.  ``p [rows, ...]`` activations; ``q``, ``k``, ``v``, ``g`` (gate), ``a``, ``b`` (gates of
    the recurrence, one column per head) are offsets in elements from a row's first.  "memory": ``a``, ``b`` input and forget gate,
    ``w0``, ``w1`` their biases; "delta": ``a`` the decay, ``b`` the step size, ``w0`` the log decay rates, ``w1`` the decay bias, ``conv
    [taps, channels]`` over q, k, v side by side; "time_mix": ``z`` the fp32 decay projection, ``w0`` its bias, ``w1`` the bonus."""
    p: torch.Tensor
    q: int
    k: int
    v: int
    g: int
    w0: torch.Tensor
    w1: torch.Tensor
    gain: torch.Tensor
    a: int = 0
    b: int = 0
    z: Optional[torch.Tensor] = None
    conv: Optional[torch.Tensor] = None


class _RecurrentParams(ctypes.Structure):           # csrc/recurrent.cuh
    _p, _l, _i, _f = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float
    _fields_ = [("start", _p), ("len", _p), ("slot", _p), ("pos0", _p), ("p", _p), ("ld", _l), ("q_off", _l), ("k_off", _l), ("v_off", _l),
                ("a_off", _l), ("b_off", _l), ("w0", _p), ("w1", _p), ("z", _p), ("ldz", _l), ("cap", _f), ("conv_w", _p), ("taps", _i),
                ("hist", _p), ("parity", _p), ("xc", _p), ("ldx", _l), ("state", _p), ("aux", _p), ("H", _i), ("KH", _i), ("D", _i),
                ("E", _i), ("y", _p), ("gain", _p), ("gain_step", _i), ("g_off", _l), ("silu", _i), ("out", _p), ("ldo", _l), ("eps", _f)]


def recurrent(b: StepBatch, s: RecurrentSpec, x: RecurrentInputs, state: torch.Tensor, out: torch.Tensor, *,
              aux: Optional[torch.Tensor] = None, hist: Optional[torch.Tensor] = None, parity: Optional[torch.Tensor] = None) -> None:
    """Advances ``state [slots, H, D, E]`` (fp32) by the batch's tokens; ``out [rows, H * E]`` (column slice).  ``aux [slots, H, D + 1]``
    ("memory": normaliser and running maximum), ``hist [slots, 2, taps - 1, channels]`` ("delta": convolution history), fp32."""
    H, D, E = s.heads, s.dim, s.vdim
    rule, dt, p = RULES[s.rule], dtype_code(x.p.dtype), x.p
    y = torch.empty((b.rows, H * E), device=p.device, dtype=torch.float32) if b.longer else None
    taps = 0 if x.conv is None else x.conv.shape[0]
    xc, ldx = None, (s.channels + 7) // 8 * 8
    if s.rule == "delta" and b.longer:
        xc = torch.empty((b.rows, ldx), device=p.device, dtype=p.dtype)
        tiles = b.table(("rows", SSM_ROWS), lambda: row_tiles(b.host, SSM_ROWS))
        _call("apb_short_conv", _lib.ptr(p), p.stride(0), x.q, _lib.ptr(x.conv), None, taps, _lib.ptr(hist), _lib.ptr(parity), _lib.ptr(xc),
              ldx, s.channels, *b.entry_ptrs(), _lib.ptr(tiles), tiles.shape[0], dt)
    params = _RecurrentParams(
        *b.entry_ptrs(), _lib.ptr(p), p.stride(0), x.q, x.k, x.v, x.a, x.b, _lib.ptr(x.w0), _lib.ptr(x.w1), _lib.ptr(x.z),
        0 if x.z is None else x.z.stride(0), s.cap, _lib.ptr(x.conv), taps, _lib.ptr(hist), _lib.ptr(parity), _lib.ptr(xc), ldx, _lib.ptr(state),
        _lib.ptr(aux), H, s.key_heads, D, E, _lib.ptr(y), _lib.ptr(x.gain), 0 if s.shared_gain else E, x.g, int(s.silu), _lib.ptr(out),
        out.stride(0), s.eps)
    ref = ctypes.byref(params)
    aligned = not (D % 8 or E % 8 or p.stride(0) % 8 or p.data_ptr() & 15 or (x.q | x.k | x.v) % 8 or (x.z is not None and x.z.stride(0) % 4))
    mma = b.longer and p.dtype == torch.bfloat16 and aligned and D <= MAX_MMA_STATE
    if b.one_token or (b.longer and not mma):
        _call("apb_recurrent", rule, ref, _lib.ptr(b.row_entry), b.n_entries, b.rows, int(b.one_token), int(b.longer and not mma), 0, dt)
    if not b.longer:
        return
    if mma:
        f32 = dict(device=p.device, dtype=torch.float32)
        if s.rule == "delta":
            tiles = b.table(("rows", CHUNK), lambda: row_tiles(b.host, CHUNK))
            heads = b.table(("chunks", CHUNK), lambda: first_tiles(b.host, CHUNK))
            square = torch.empty((tiles.shape[0], H, 4, CHUNK, CHUNK), device=p.device, dtype=torch.bfloat16)
            scalars = torch.empty((tiles.shape[0], H, 4 * CHUNK + 4), **f32)
            _call("apb_delta_mma", ref, _lib.ptr(tiles), tiles.shape[0], _lib.ptr(heads), heads.shape[0], _lib.ptr(square), _lib.ptr(scalars))
        else:
            plan, seg, chains = segments(b, H * ((E + 63) // 64))
            n_seg, parts = len(plan["seg"]), plan["states"]
            carry = torch.empty((parts, H, D, E), **f32) if parts else None
            if s.rule == "memory":
                gates, aux0 = torch.empty((b.rows, H, 2), **f32), torch.empty((b.n_entries, H, D + 1), **f32)
                carry_aux = torch.empty((parts, H, D + 1), **f32) if parts else None
                totals = torch.empty((n_seg, H, 2), **f32) if parts else None
                _call("apb_memory_mma", ref, b.rows, b.n_entries, _lib.ptr(gates), _lib.ptr(aux0), _lib.ptr(seg), n_seg, _lib.ptr(carry),
                      _lib.ptr(carry_aux), _lib.ptr(totals), _lib.ptr(chains), len(plan["chains"]))
            else:
                decay = torch.empty((n_seg, H, D), **f32) if parts else None
                tiles = b.table(("rows", CHUNK), lambda: row_tiles(b.host, CHUNK))
                at = b.table(("segment chunks", H * ((E + 63) // 64)), lambda: segment_chunks(b.host, plan["seg"]))
                square = torch.empty((tiles.shape[0], H, 2, CHUNK, CHUNK), device=p.device, dtype=torch.bfloat16)
                _call("apb_time_mix_mma", ref, _lib.ptr(tiles), tiles.shape[0], _lib.ptr(seg), _lib.ptr(at), n_seg, _lib.ptr(square),
                      _lib.ptr(carry), _lib.ptr(decay), _lib.ptr(chains), len(plan["chains"]))
    _call("apb_recurrent", rule, ref, _lib.ptr(b.row_entry), b.n_entries, b.rows, 0, 0, 1, dt)


MANY_ROWS = 1024


def token_shift(b: StepBatch, h: torch.Tensor, mu: torch.Tensor, hist: torch.Tensor, parity: torch.Tensor, w: torch.Tensor, step: int,
                cols: Sequence[int]) -> torch.Tensor:
    """``h [rows, W]`` blended with the row of the token before, ``h + (h' - h) mu[s]`` for every ``mu [n, W]``, and the products of the
    blends with their weights: rows ``s * step`` and following of ``w``, ``cols[s]`` of them.  ``hist [slots, 2, 1, W]`` fp32 carries the
    last row.  Returns ``[n, rows, N]`` with ``N >= max(cols)``; columns from ``cols[s]`` on are undefined."""
    T, W = h.shape
    n, N = len(cols), (max(cols) + 7) // 8 * 8
    dev, dt = h.device, dtype_code(h.dtype)
    mixed = torch.empty((n, T, W), device=dev, dtype=h.dtype)
    out = torch.empty((n, T, N), device=dev, dtype=h.dtype)
    simt = _simt(h, w, out[0]) or bool(step % 8)
    ptrs = (_lib.ptr(h), _lib.ptr(mu), _lib.ptr(hist), _lib.ptr(parity), _lib.ptr(mixed), _lib.ptr(b.row_entry), *b.entry_ptrs(), T, W, n)
    if not simt and T >= MANY_ROWS:          # each product fills the GPU
        _call("apb_token_shift", *ptrs, None, None, 1, step, None, dt)
        for i, c in enumerate(cols):
            linear(mixed[i], w[i * step:i * step + (c + 7) // 8 * 8], out[i][:, :(c + 7) // 8 * 8])
        return out
    tile = 64 if simt else 128
    most = sum(-(-T // tile) * -(-c // tile) for c in cols)
    tiles = torch.empty(4 * most + 4, device=dev, dtype=torch.int32)
    count = tiles[4 * most:]
    _call("apb_token_shift", *ptrs, _lib.ptr(tiles), _lib.ptr(count), tile, step, (ctypes.c_int * n)(*cols), dt)
    if simt:
        _call("apb_gemm_simt_grouped", _lib.ptr(mixed), _lib.ptr(w), _lib.ptr(out), n * T, N, W, W, w.stride(0), N, gemm.EPI_BF16, None, 0, 0.0,
              _lib.ptr(tiles), most, _lib.ptr(count), dt)
    else:
        _call("apb_gemm_bf16_grouped_dev", _lib.ptr(mixed), _lib.ptr(w), _lib.ptr(out), n * T, N, W, W, w.stride(0), N, gemm.EPI_BF16, 1.0, None,
              0, _lib.ptr(tiles), most, _lib.ptr(count), w.shape[0])
    return out


def tanh_rows(x: torch.Tensor) -> None:
    """``x [rows, n]`` (column slice) <- tanh(x), rounded to the activation type."""
    _call("apb_tanh_rows", _lib.ptr(x), x.stride(0), x.shape[0], x.shape[1], dtype_code(x.dtype))
