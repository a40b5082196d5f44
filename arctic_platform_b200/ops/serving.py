"""Operations of a serving step over a ragged batch (CUDA only).

A step advances several sequences at once, each by its own run of new tokens: a portion of a prompt of any length, or
one decoded token.  :class:`StepBatch` is the device-side description of such a step; the functions below launch the
kernels of ``serve_layers.cu``, ``serve_attention.cu``, ``serve_attention_tc.cu``, ``retention.cu`` and
``gemm_simt.cu`` on it.  They take bf16 or fp32 activations; the residual stream and all carried state are fp32.
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
            "apb_embed_hash": [vp] * 9 + [ll, ll, ll, i, i, vp, vp, ll, vp, i, vp, i, i, vp],
            "apb_loop_begin": [vp, vp, i, i, vp, ll, i, vp],
            "apb_norm_conv": [vp] * 13 + [i, i, i, f, i, vp],
            "apb_gain_norm_rows": [vp, vp, vp, vp, i, i, f, i, vp],
            "apb_qk_norm_cache": [vp, ll, i, i, i, vp, vp, vp, i, i, i, i, i, f, i, vp],
            "apb_serve_commit": [vp] * 5 + [i, vp, vp, vp],
            "apb_sigmoid_attn": [vp, ll, vp, vp, vp, vp, vp, vp, i, vp, vp, vp, vp, ll, i, i, i, i, i, f, f, i, vp],
            "apb_sigmoid_attn_mma": [vp, ll, vp, vp, vp, vp, i, vp, i, vp, vp, vp, vp, ll, vp] + [i] * 7 + [f, f, vp],
            "apb_sigmoid_attn_tc": [vp, ll, i, vp, i, vp, i, vp, vp, i, vp, vp, ll, i, i, i, i, f, f, vp],
            "apb_retention": [vp, ll, i, i, i, i, vp, vp, i, vp, f, vp, vp, vp, ll, f, f, vp, vp, vp, vp, vp] + [i] * 8 + [vp],
            "apb_retention_mma": [vp, ll, i, i, i, vp, vp, i, vp, f] + [vp] * 7 + [i, vp, vp, i, vp, vp, i, i, i, i, vp],
            "apb_retention_out": [vp, ll, i, vp, vp, ll, f, f, vp, vp, vp, vp, vp, i, i, i, i, vp],
            "apb_gemm_simt": [vp, vp, vp, i, i, i, ll, ll, ll, i, vp, vp, ll, i, vp],
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

    def entry_ptrs(self):
        return _lib.ptr(self.start), _lib.ptr(self.len), _lib.ptr(self.slot), _lib.ptr(self.pos0)


# --------------------------------------------------------------------------------------------- embedding and loop input
def embed(b: StepBatch, table: torch.Tensor, bigram: Optional[torch.Tensor], hash_spec: Optional[Tuple[int, int, int]],
          prev: torch.Tensor, x: torch.Tensor, x0: Optional[torch.Tensor] = None) -> None:
    """``x [rows, W]`` fp32 = token rows + hashed bigram rows (``hash_spec`` = buckets, multiplier of the previous and
    of the current token); ``x0`` receives them in the activation type.  Also fills ``b.kv_slot``."""
    V, W = table.shape
    buckets, mp, mc = hash_spec or (0, 0, 0)
    _call("apb_embed_hash", _lib.ptr(b.tokens), _lib.ptr(b.row_entry), *b.entry_ptrs(), _lib.ptr(prev), _lib.ptr(table),
          _lib.ptr(bigram), buckets, mp, mc, V, W, _lib.ptr(x), _lib.ptr(x0), 0 if x0 is None else x0.stride(0),
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


def gain_norm_rows(x: torch.Tensor, rows: Optional[torch.Tensor], gain: torch.Tensor, eps: float) -> torch.Tensor:
    n = x.shape[0] if rows is None else rows.shape[0]
    out = torch.empty((n, x.shape[1]), device=x.device, dtype=gain.dtype)
    _call("apb_gain_norm_rows", _lib.ptr(x), _lib.ptr(rows), _lib.ptr(gain), _lib.ptr(out), n, x.shape[1], float(eps),
          dtype_code(gain.dtype))
    return out


def qk_norm_cache(b: StepBatch, p: torch.Tensor, cols: Tuple[int, int, int], kcache: torch.Tensor, vcache: torch.Tensor,
                  heads: int, eps: float) -> None:
    """q and k columns of ``p`` divided by their root mean square per head (q in place), k and v into the page cache
    (``[pages, G, PAGE, D]`` and ``[pages, G, PAGE, E]``)."""
    G, D, E = kcache.shape[1], kcache.shape[3], vcache.shape[3]
    _call("apb_qk_norm_cache", _lib.ptr(p), p.stride(0), *cols, _lib.ptr(b.kv_slot), _lib.ptr(kcache), _lib.ptr(vcache),
          b.rows, heads, G, D, E, float(eps), dtype_code(p.dtype))


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


def gate_up_gelu(x: torch.Tensor, w_gu: torch.Tensor, out: torch.Tensor) -> None:
    """``out [M, ff]`` (may be a column slice) = gelu_tanh(gate) * up; gate and up rows interleaved in ``w_gu``."""
    M, K = x.shape
    N = w_gu.shape[0]
    if _simt(x, w_gu, out) or N % 16:
        _gemm_simt(x, w_gu, None, gemm.EPI_GEGLU, out2=out)
    else:
        gemm.gemm_raw(x, w_gu, None, M=M, N=N, K=K, epi=gemm.EPI_GEGLU, out2=out)


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


def _gemm_simt(a, w, out, epi, out2=None) -> None:
    _call("apb_gemm_simt", _lib.ptr(a), _lib.ptr(w), _lib.ptr(out), a.shape[0], w.shape[0], a.shape[1], a.stride(0),
          w.stride(0), 0 if out is None else out.stride(0), epi, None, _lib.ptr(out2),
          0 if out2 is None else out2.stride(0), dtype_code(a.dtype))


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
        key = ("retention", slices)
        if key not in b.host_tables:
            b.host_tables[key] = segment_plan(b.host, slices, 2 * _sm_count(p.device))
        plan = b.host_tables[key]
        seg = b.table(key + ("seg",), lambda: plan["seg"])
        chains = b.table(key + ("chains",), lambda: plan["chains"]) if len(plan["chains"]) else None
        qk = torch.empty((b.rows, H, 4, (D + 15) // 16 * 16), device=p.device, dtype=torch.bfloat16)
        carry = torch.empty((plan["states"], H, D, E), device=p.device, dtype=torch.float32) if plan["states"] else None
        _call("apb_retention_mma", _lib.ptr(p), p.stride(0), *cols[:3], _lib.ptr(rope[0]), _lib.ptr(rope[1]), rot_dims,
              _lib.ptr(log2_decay), float(k_scale), _lib.ptr(state), _lib.ptr(scratch), *b.entry_ptrs(), _lib.ptr(seg),
              len(plan["seg"]), _lib.ptr(carry), _lib.ptr(chains), len(plan["chains"]), _lib.ptr(b.row_entry), _lib.ptr(qk),
              b.rows, H, D, E)
        _call("apb_retention_out", _lib.ptr(p), p.stride(0), cols[3], _lib.ptr(scratch), _lib.ptr(out), out.stride(0),
              float(out_scale), float(eps), _lib.ptr(b.row_entry), *b.entry_ptrs(), b.rows, H, E, dtype_code(p.dtype))
