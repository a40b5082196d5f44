"""Serving speed of the stateful architectures beside the closest older model of equal layer size.

    python bench.py --workload serving [--serving-models reninex-2048,rigulorn-2048,...]
    python benchmarks/bench_serving.py [--models ...] [--kernels-only] [--only prefill|decode] [--step NAME] [--iters 20]

For every model (random weights, synthetic prompts) two parts are measured on one GPU:

* kernels: each step of ONE layer of every kind on a prefill batch (4 prompts x 2048 tokens) and on a decode batch (128
  sequences after 2048 tokens), next to the like kernel of the closest model: for Reninex a Qwen3-style layer of the same
  width, heads and feed-forward (for retention the gated delta rule of the hybrid family at the same heads and sizes); for
  Rigulorn a Reninex layer whose K/V rows, state and feed-forward have the same size; for Titatar the dense decoder's layer
  with the heads of its windowed attention, and the decoder family's mixture of experts with as many experts and (on average)
  as many routed rows; for Meronex the steps of a Titatar layer with its attention heads and its experts, for the recurrent mixers
  Rigulorn's state space with as many heads and states of the same size.  ``floor_ms`` is the slower of
  algorithmic bytes over the measured copy bandwidth and FLOPs over the measured bf16 GEMM peak, ``frac`` = floor / time.
  CUDA events around every launch, L2 overwritten before it, median over the iterations.
* engine: prefill and decode tokens/s through ``generate`` of the model, of the dense decoder with as many layers as the
  model has layer runs (for Titatar and Meronex: with a mixture of experts of the same size in every layer) and, for Rigulorn
  and Meronex, of the Reninex or Titatar preset of the same width.

Prints one JSON line per measurement.
"""
from __future__ import annotations

import argparse
import json
import statistics
import sys
import time
from pathlib import Path

import numpy as np
import torch

ROOT = Path(__file__).resolve().parents[1]
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))

SEQ, PREFILL_SEQS, DECODE_SEQS = 2048, 4, 128


def peaks():
    f = ROOT / "MEASURED_PEAKS.json"
    if f.is_file():
        d = json.loads(f.read_text())
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


class Timer:
    def __init__(self, iters: int):
        from arctic_platform_b200.ops import _lib
        self.iters, self.lib = iters, _lib
        self.flush = torch.empty(256 << 20, device="cuda", dtype=torch.uint8)

    def __call__(self, fn) -> float:
        """Median milliseconds of ``fn`` with a cold L2."""
        for _ in range(3):
            fn()
        marks = []
        for _ in range(self.iters):
            self.lib.cuda_lib().apb_fill_u32(self.lib.ptr(self.flush), self.flush.numel(), 1, self.lib.stream_ptr())
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            marks.append((e0, e1))
        torch.cuda.synchronize()
        return statistics.median(a.elapsed_time(b) for a, b in marks)


def _bf(*shape, std=1.0):
    return (torch.randn(*shape, device="cuda") * std).to(torch.bfloat16)


def phase_batch(phase):
    """``(batch, page tables, sequences, sum over the rows of the keys they see)``."""
    from arctic_platform_b200.ops import serving
    n = PREFILL_SEQS if phase == "prefill" else DECODE_SEQS
    per = SEQ // 16 + 1
    pages = np.random.default_rng(0).permutation(n * per).astype(np.int32).reshape(n, per)
    if phase == "prefill":
        b = serving.StepBatch.build([serving.StepEntry(i, np.arange(SEQ) % 1000, 0, pages[i]) for i in range(n)], "cuda")
        return b, n, n * per, SEQ * (SEQ + 1) // 2 * n
    i32 = dict(device="cuda", dtype=torch.int32)
    one = torch.arange(n, **i32)
    b = serving.StepBatch(n, n, one.clone(), None, one, torch.ones(n, **i32), one, torch.full((n,), SEQ, **i32),
                          torch.from_numpy(pages).cuda(), torch.empty(n, **i32))
    return b, n, n * per, (SEQ + 1) * n


def stateful_ops(cfg, phase):
    """``(name, fn, bytes, flops)`` of the steps of the model's layers on the phase's batch."""
    return {"Reninex": reninex_ops, "Rigulorn": rigulorn_ops, "Titatar": titatar_ops,
            "Meronex": meronex_ops}[cfg.architecture](cfg, phase)


def reninex_ops(cfg, phase):
    from arctic_platform_b200.engine.stateful_sampler import StateCache
    from arctic_platform_b200.models.reninex import ReninexLM
    from arctic_platform_b200.ops import serving
    import dataclasses
    one = dataclasses.replace(cfg, layers=cfg.layers[:1], loop=None, vocab_size=1024, bigram=None)
    model = ReninexLM(one, "cuda", torch.bfloat16).init_weights(0)
    model.prepare_serving(SEQ + 8)
    blk, s, W = model.blocks[0], one.layers[0], cfg.hidden_size
    L, R = s.left, s.right
    b, n, n_pages, keys = phase_batch(phase)
    cache = StateCache(model.cache_layout(), n_pages, n, "cuda", torch.bfloat16)
    for t in (cache.k[0], cache.v[0]):
        t.normal_()
    T = b.rows
    x = torch.randn(T, W, device="cuda")
    serving.embed(b, model.embed, None, None, cache.prev, torch.empty_like(x))
    h = _bf(T, W)
    p = serving.linear(h, blk.w_in)
    a = _bf(T, blk.w_out.shape[1])
    c, o = blk.in_cols, blk.out_cols
    Nin, K = blk.w_in.shape[0], blk.w_out.shape[1]
    ctx = T if phase == "prefill" else keys                  # K/V rows that have to be read once
    kv_row = L.kv_heads * (L.dim + L.vdim) * 2
    state = n * R.heads * R.dim * R.vdim * 4
    cols = tuple(c["right." + m][0] for m in "qkvg")
    rope = model._rope[R.rot_dims, R.rot_base]
    ret_flops = T * R.heads * (2 * 64 * (R.dim + R.vdim) / 2 + 4 * R.dim * R.vdim)
    return [
        ("norm + 2 input convolutions", lambda: serving.norm_conv(b, x, blk.norm1, blk.canon1, blk.canon2, True, cache.conv[0],
                                                                 cache.parity, cfg.conv_taps, cfg.norm_eps),
         T * W * 8 + (2 * n * (cfg.conv_taps - 1) * W * 4), 0),
        ("input projections (GEMM)", lambda: serving.linear(h, blk.w_in, p), 2 * (T * W + Nin * W + T * Nin), 2 * T * W * Nin),
        ("gate/up + GELU (GEMM)", lambda: serving.gate_up_gelu(h, blk.w_gu, a[:, o["down"][0]:]),
         2 * (T * W + 2 * s.ff * W + T * s.ff), 4 * T * W * s.ff),
        ("q/k norm + cache write", lambda: serving.qk_norm_cache(b, p, (c["left.q"][0], c["left.k"][0], c["left.v"][0]),
                                                               cache.k[0], cache.v[0], L.heads, cfg.norm_eps),
         2 * T * (2 * L.heads * L.dim) + 2 * T * kv_row, 0),
        ("attention", lambda: serving.sigmoid_attention(b, p[:, c["left.q"][0]:], L.heads, cache.k[0], cache.v[0], blk.pb,
                                                        L.scale, a[:, o["left.o"][0]:], s.left_scale),
         ctx * kv_row + 2 * T * L.heads * (L.dim + L.vdim), 2 * keys * L.heads * (L.dim + L.vdim)),
        ("recurrent mixer", lambda: serving.retention(b, p, cols, rope, R.rot_dims, blk.log2_decay, cache.state[0],
                                                      a[:, o["right.o"][0]:], cfg.norm_eps, R.dim ** -0.5, s.right_scale),
         2 * T * R.heads * (2 * R.dim + 3 * R.vdim) + state * (2 if phase == "decode" else 1), ret_flops),
        ("output projections (GEMM, += fp32)", lambda: serving.linear(a, blk.w_out, x, accumulate=True),
         2 * (T * K + K * W) + 8 * T * W, 2 * T * K * W),
    ]


def rigulorn_ops(cfg, phase):
    import dataclasses
    from arctic_platform_b200.engine.stateful_sampler import StateCache
    from arctic_platform_b200.models.rigulorn import RigulornLM
    from arctic_platform_b200.ops import serving
    attn = next(s for s in cfg.layers if s.attention and s.ff)
    ssm = next(s for s in cfg.layers if not s.attention)
    one = dataclasses.replace(cfg, layers=(attn, ssm), vocab_size=1024)
    model = RigulornLM(one, "cuda", torch.bfloat16).init_weights(0)
    model.prepare_serving(SEQ + 8)
    b, n, n_pages, keys = phase_batch(phase)
    cache = StateCache(model.cache_layout(), n_pages, n, "cuda", torch.bfloat16)
    for t in (cache.k[0], cache.v[0]):
        t.normal_()
    T, W, S, A, M = b.rows, cfg.hidden_size, cfg.streams, attn.mixer, ssm.mixer
    blk, mam = model.blocks
    x = torch.empty(T, S, W, device="cuda")
    serving.embed(b, model.embed, None, None, cache.prev, x)
    clear = serving.accumulates(T, W, x.device)
    y, h = torch.zeros(T, W, device="cuda"), _bf(T, W)
    p, pm = serving.linear(h, blk.mixer.w_in), serving.linear(h, mam.mixer.w_in)
    rope = model._rope[A.rot_dims, A.rot_base]
    ao, mo, fo = _bf(T, A.heads * A.vdim), _bf(T, M.inner), _bf(T, attn.ff)
    c, cm, mx = blk.mixer.in_cols, mam.mixer.in_cols, mam.mixer
    w = serving.SsmWeights(mx.conv, mx.conv_bias, mx.dt_bias, mx.a_log, mx.skip)
    kv_row = A.kv_heads * (2 * A.dim + A.vdim) * 2
    ctx = T if phase == "prefill" else keys
    state = n * M.inner * M.state * 4
    gemm = lambda N, K: (2 * (T * K + N * K + T * N), 2 * T * N * K)
    out = lambda K: (2 * (T * K + K * W) + (8 if clear else 4) * T * W, 2 * T * W * K)

    def recurrent():
        s = serving.state_space(b, pm, cm["xbc"][0], cm["dt"][0], w, M.groups, cache.conv[1], cache.parity, cache.state[1])
        serving.gated_group_norm(s, pm, mx.gain, M.norm_groups, cfg.norm_eps, mo)

    s1 = blk.sub1
    return [
        ("stream update + norm", lambda: serving.stream_step(x, y, s1.hc_mix, s1.hc_out, s1.hc_in, s1.norm, cfg.norm_eps, clear=clear),
         T * W * (8 * S + 4 + 2 + (4 if clear else 0)), 0),
        ("attention input projections (GEMM)", lambda: serving.linear(h, blk.mixer.w_in, p), *gemm(p.shape[1], W)),
        ("rotation + cache write", lambda: serving.rope_cache(b, p, tuple(c[m][0] for m in c), rope, A.rot_dims, 2 * A.heads, A.dim,
                                                             cache.k[0], cache.v[0]),
         2 * T * (2 * A.heads * 2 * A.dim) + 2 * T * kv_row, 0),
        ("attention", lambda: serving.softmax_attention(b, p, A.heads, cache.k[0], cache.v[0], blk.mixer.spec, blk.mixer.lam, ao),
         ctx * kv_row + 2 * T * A.heads * (2 * A.dim + A.vdim), 2 * keys * A.heads * (2 * A.dim + 2 * A.vdim)),
        ("attention output projection (GEMM)", lambda: serving.project(ao, blk.mixer.w_out, y), *out(ao.shape[1])),
        ("gate/up + clamped GLU (GEMM)", lambda: serving.gate_up_clamped(h, blk.mlp.w_gu, fo, attn.limit),
         2 * (T * W + 2 * attn.ff * W + T * attn.ff), 4 * T * W * attn.ff),
        ("down projection (GEMM)", lambda: serving.project(fo, blk.mlp.w_down, y), *out(attn.ff)),
        ("state-space input projections (GEMM)", lambda: serving.linear(h, mx.w_in, pm), *gemm(pm.shape[1], W)),
        ("recurrent mixer", recurrent,
         2 * T * (2 * M.inner + 2 * M.groups * M.state + M.heads + M.inner) + state * (2 if phase == "decode" else 1),
         T * M.heads * (2 * 64 * (M.state + M.vdim) / 2 + 4 * M.state * M.vdim)),
        ("state-space output projection (GEMM)", lambda: serving.project(mo, mx.w_out, y), *out(M.inner)),
    ]


def titatar_ops(cfg, phase):
    import dataclasses
    import math
    from arctic_platform_b200.engine.stateful_sampler import StateCache
    from arctic_platform_b200.models.titatar import MoeSpec, TitatarLM
    from arctic_platform_b200.ops import serving
    lat = next(s for s in cfg.layers if s.latent and isinstance(s.mlp, MoeSpec))
    win = next(s for s in cfg.layers if not s.latent)
    ff = next(s.mlp for s in cfg.layers if isinstance(s.mlp, int))
    one = dataclasses.replace(cfg, layers=(lat, dataclasses.replace(win, mlp=ff)), loop=None, vocab_size=1024)
    model = TitatarLM(one, "cuda", torch.bfloat16).init_weights(0)
    model.prepare_serving(SEQ + 8)
    b, n, n_pages, keys = phase_batch(phase)
    cache = StateCache(model.cache_layout(), n_pages, n, "cuda", torch.bfloat16)
    for t in cache._paged():
        t.normal_()
    T, W, L, A, M = b.rows, cfg.hidden_size, lat.mixer, win.mixer, lat.mlp
    lb, wb = model.blocks
    lm, wm, moe, glu = lb.mixer, wb.mixer, lb.mlp, wb.mlp
    x = torch.randn(T, W, device="cuda")
    serving.embed(b, model.embed, None, None, cache.prev, torch.empty_like(x))
    clear = serving.accumulates(T, W, x.device)
    y, h = torch.zeros(T, W, device="cuda"), _bf(T, W)
    pl, pw = serving.linear(h, lm.w_in), serving.linear(h, wm.w_in)
    lc, wc = lm.in_cols, wm.in_cols
    rl, rw = model._rope[L.rot], model._rope[A.rot]
    q = _bf(T, lm.w_q.shape[0])
    ql = pl[:, lc["dq"][0]:lc["dq"][0] + L.q_rank]
    lo, wo, fo = _bf(T, lm.n_out), _bf(T, wm.n_out), _bf(T, ff)
    z = serving.linear(h, moe.router, out_dtype=torch.float32)

    def experts():
        return serving.experts(b, h, z, moe.correction, moe.counters, moe.w_gu, moe.w_down, M.scores, M.experts, M.top, M.ff)

    mix = experts()
    pairs = T * M.top * M.experts / M.scores
    touched = M.experts * (1 - math.exp(-pairs / M.experts))
    C, R, D, E, H = L.kv_rank, L.rot_dim, L.dim, L.vdim, L.heads
    row = (C + R) * 2
    ctx = T if phase == "prefill" else keys
    seen = keys                                          # keys inside the window, summed over the rows
    if A.window:
        seen = n * sum(min(i + 1, A.window) for i in range(SEQ)) if phase == "prefill" else n * min(A.window, SEQ + 1)
    wctx = T if phase == "prefill" else seen
    kv_row = A.kv_heads * (A.dim + A.vdim) * 2
    expand = lm.w_expand.numel() * 2
    if phase == "prefill":
        lat_flops = 2 * keys * H * (D + R + E) + 2 * T * C * H * (D + E)
    else:
        lat_flops = 2 * keys * H * (2 * C + R) + 2 * T * C * H * (D + E)
    gemm = lambda N, K: (2 * (T * K + N * K + T * N), 2 * T * N * K)
    out = lambda K: (2 * (T * K + K * W) + (8 if clear else 4) * T * W, 2 * T * W * K)
    return [
        ("residual update + norms", lambda: serving.residual_step(x, y, lb.norm1b, lb.norm2, 1e-6, clear=clear),
         T * W * (8 + 4 + 2 + (4 if clear else 0)), 0),
        ("residual update + expert sum + norms", lambda: serving.residual_step(x, y, lb.norm1b, lb.norm2, 1e-6, clear=clear, mix=mix),
         T * W * (8 + 4 + 2 + (4 if clear else 0) + 2) + 2 * pairs * W, 0),
        ("latent input projections (GEMM)", lambda: serving.linear(h, lm.w_in, pl), *gemm(pl.shape[1], W)),
        ("latent norms + cache write", lambda: serving.latent_norm_cache(b, pl, lc["dq"][0], lc["dkv"][0], lm.q_norm, lm.kv_norm, rl,
                                                                        cache.k[0], 1e-6, R), 2 * T * (2 * L.q_rank + 2 * (C + R)), 0),
        ("query projection (GEMM)", lambda: serving.linear(ql, lm.w_q[:, :L.q_rank], q), *gemm(q.shape[1], L.q_rank)),
        ("latent attention", lambda: serving.latent_attention(b, q, lm.spec, cache.k[0], lm.w_absorb, lm.w_expand, lm.sink32,
                                                              pl[:, lc["g"][0]:], rl, lo),
         ctx * row + expand + 2 * T * H * (D + R + 2 * E), lat_flops),
        ("latent output projection (GEMM)", lambda: serving.project(lo, lm.w_out, y), *out(lm.n_out)),
        ("windowed input projections (GEMM)", lambda: serving.linear(h, wm.w_in, pw), *gemm(pw.shape[1], W)),
        ("q/k norm + rotation + cache write", lambda: serving.row_norm_rope_cache(b, pw, (wc["q"][0], wc["k"][0], wc["v"][0]), wm.q_norm,
                                                                                wm.k_norm, rw, A.rot.dims, A.heads, cache.k[1], cache.v[1], 1e-6),
         2 * T * (2 * A.heads * A.dim) + 2 * T * kv_row, 0),
        ("windowed attention", lambda: serving.softmax_attention(b, pw, A.heads, cache.k[1], cache.v[1], wm.spec, None, wo, sink=wm.sink,
                                                                 gate=pw[:, wc["g"][0]:]),
         wctx * kv_row + 2 * T * A.heads * (A.dim + A.vdim), 2 * seen * A.heads * (A.dim + A.vdim)),
        ("windowed output projection (GEMM)", lambda: serving.project(wo, wm.w_out, y), *out(wm.n_out)),
        ("router (GEMM)", lambda: serving.linear(h, moe.router, z), 2 * T * W + 2 * z.shape[1] * W + 4 * T * z.shape[1], 2 * T * W * z.shape[1]),
        ("routed experts", experts, touched * 6 * W * M.ff + 2 * T * W + 2 * pairs * W, 6 * pairs * W * M.ff),
        ("gate/up + SiLU (GEMM)", lambda: serving.gate_up_silu(h, glu.w_gu, fo), 2 * (T * W + 2 * ff * W + T * ff), 4 * T * W * ff),
        ("down projection (GEMM)", lambda: serving.project(fo, glu.w_down, y), *out(ff)),
    ]


def meronex_ops(cfg, phase):
    import dataclasses
    import math
    from arctic_platform_b200.engine.stateful_sampler import StateCache
    from arctic_platform_b200.models.meronex import MeronexLM
    from arctic_platform_b200.ops import gemm as gemm_ops, serving
    one = dataclasses.replace(cfg, layers=tuple(next(s for s in cfg.layers if s.type == t) for t in ("mlstm", "delta", "parallel")),
                              vocab_size=1024)
    model = MeronexLM(one, "cuda", torch.bfloat16).init_weights(0)
    model.prepare_serving(SEQ + 8)
    b, n, n_pages, keys = phase_batch(phase)
    cache = StateCache(model.cache_layout(), n_pages, n, "cuda", torch.bfloat16)
    for t in cache._paged():
        t.normal_()
    T, W, G = b.rows, cfg.hidden_size, cfg.norm_groups
    mem, dlt, par = (blk.mixer for blk in model.blocks)
    moe, M = model.blocks[0].mlp, one.layers[0].mlp
    x = torch.randn(T, W, device="cuda")
    serving.embed(b, model.embed, None, None, cache.prev, torch.empty_like(x))
    clear = serving.accumulates(T, W, x.device)
    y, y2, h = torch.zeros(T, W, device="cuda"), torch.zeros(T, W, device="cuda"), _bf(T, W)
    pm, pd, pp = (serving.linear(h, m.w_in) for m in (mem, dlt, par))
    om, od, ol, orr = (_bf(T, m) for m in (mem.n_out, dlt.n_out, par.n_left, par.n_right))
    L, R, K = par.m.left, par.m.right, par.rank
    c, rope = par.in_cols, model._rope[L.rot]
    spin = pp.clone()                                    # rotated in place again and again; attention reads queries rotated once
    serving.half_rope_cache(b, pp, (c["q"][0], c["k"][0], c["v"][0]), rope, L.rot.dims, L.heads, cache.k[2], cache.v[2], 1e-6)
    cols = [par.n_right] * 4 + [K]
    s = serving.token_shift(b, h, par.mu, cache.conv[2], cache.parity, par.w_shift, par.step, cols)
    low = s[4][:, :K]
    z = serving.linear(low, par.w_rank[:, :K], out_dtype=torch.float32)
    zz = serving.linear(h, moe.w_z, out_dtype=torch.float32)
    gate_col = moe.z_cols["rg"][0]

    def experts():
        return serving.experts(b, h, zz, None, moe.counters, moe.w_gu, moe.w_down, M.experts, M.experts, M.top, M.ff, sigmoid=True,
                               scale_input=True, epi=gemm_ops.EPI_CLAMP_GLU, limit=M.limit)

    def decay():
        serving.tanh_rows(low)
        serving.linear(low, par.w_rank[:, :K], z)

    mix = experts()
    pairs = T * M.top
    touched = M.experts * (1 - math.exp(-pairs / M.experts))
    ctx = T if phase == "prefill" else keys
    kv_row = L.kv_heads * (L.dim + L.vdim) * 2
    norms, bias = model.blocks[2], model.blocks[0]
    passes = 2 if phase == "decode" else 1
    state = lambda H, D, E: n * H * D * E * 4 * passes
    chunked = lambda H, D, E, f: T * H * (2 * 64 * (D + E) / 2 + f * D * E)
    gemm = lambda N, K: (2 * (T * K + N * K + T * N), 2 * T * N * K)
    out = lambda K: (2 * (T * K + K * W) + (8 if clear else 4) * T * W, 2 * T * W * K)
    res = T * W * (8 + 2 + (4 if clear else 0))
    how = dict(eps=1e-6, offset=0.0, groups=G, mult=0.7, clear=clear)
    d = mem.m
    q = dlt.m
    Hr, Dr = R.heads, R.dim
    return [
        ("gated residual update + norm", lambda: serving.residual_step(x, y, None, norms.norm1, gate=pm[:, mem.in_cols["rg"][0]:],
                                                                      gate_bias=bias.gate_bias1, **how), res + 6 * T * W, 0),
        ("gated residual update + expert sum + norm", lambda: serving.residual_step(x, None, None, norms.norm1, mix=mix, gate=zz[:, gate_col:],
                                                                                   gate_bias=bias.gate_bias2, **how),
         T * W * (8 + 2 + 4) + 2 * pairs * W, 0),
        ("gated residual update + two sides + norm", lambda: serving.residual_step(x, y, par.left_out, norms.norm2, y2=y2, post2=par.right_out,
                                                                                  gate=pp[:, c["rg"][0]:], gate_bias=norms.gate_bias1, **how),
         res + 6 * T * W + (8 if clear else 4) * T * W, 0),
        ("memory input projections (GEMM)", lambda: serving.linear(h, mem.w_in, pm), *gemm(pm.shape[1], W)),
        ("matrix memory", lambda: serving.recurrent(b, mem.spec, mem.inputs(pm), cache.state[0], om, aux=cache.aux[0]),
         2 * T * (2 * d.heads * d.dim + 3 * mem.n_out + 2 * d.heads) + state(d.heads, d.dim, d.vdim), chunked(d.heads, d.dim, d.vdim, 4)),
        ("memory output projection (GEMM)", lambda: serving.project(om, mem.w_out, y), *out(mem.n_out)),
        ("delta input projections (GEMM)", lambda: serving.linear(h, dlt.w_in, pd), *gemm(pd.shape[1], W)),
        ("convolution + delta rule", lambda: serving.recurrent(b, dlt.spec, dlt.inputs(pd), cache.state[1], od, hist=cache.conv[1],
                                                               parity=cache.parity),
         2 * T * (2 * q.kv_heads * q.dim + 3 * dlt.n_out + 2 * q.heads) + state(q.heads, q.dim, q.vdim), chunked(q.heads, q.dim, q.vdim, 6)),
        ("delta output projection (GEMM)", lambda: serving.project(od, dlt.w_out, y), *out(dlt.n_out)),
        ("parallel input projections (GEMM)", lambda: serving.linear(h, par.w_in, pp), *gemm(pp.shape[1], W)),
        ("rotation + value norm + cache write", lambda: serving.half_rope_cache(b, spin, (c["q"][0], c["k"][0], c["v"][0]), rope, L.rot.dims,
                                                                               L.heads, cache.k[2], cache.v[2], 1e-6),
         2 * T * (2 * L.heads * L.dim) + 2 * T * kv_row, 0),
        ("capped attention", lambda: serving.softmax_attention(b, pp, L.heads, cache.k[2], cache.v[2], par.softmax, None, ol),
         ctx * kv_row + 2 * T * L.heads * (L.dim + L.vdim), 2 * keys * L.heads * (L.dim + L.vdim)),
        ("attention output projection (GEMM)", lambda: serving.project(ol, par.w_left, y), *out(par.n_left)),
        ("token shift + its products (GEMM)", lambda: serving.token_shift(b, h, par.mu, cache.conv[2], cache.parity, par.w_shift, par.step, cols),
         2 * (T * W + sum(cols) * W + T * sum(cols)), 2 * T * W * sum(cols)),
        ("decay projection (GEMM)", decay, 2 * (2 * T * K + par.n_right * K) + 4 * T * par.n_right, 2 * T * K * par.n_right),
        ("time mixing", lambda: serving.recurrent(b, par.spec, par.inputs(s, z), cache.state[2], orr),
         2 * T * 5 * par.n_right + 4 * T * par.n_right + state(Hr, Dr, Dr), chunked(Hr, Dr, Dr, 4)),
        ("time mixing output projection (GEMM)", lambda: serving.project(orr, par.w_right, y2), *out(par.n_right)),
        ("router + gate (GEMM)", lambda: serving.linear(h, moe.w_z, zz), 2 * T * W + 2 * zz.shape[1] * W + 4 * T * zz.shape[1],
         2 * T * W * zz.shape[1]),
        ("routed experts", experts, touched * 6 * W * M.ff + 2 * T * W + 2 * pairs * W, 6 * pairs * W * M.ff),
    ]


# step of a Meronex layer -> (model, the like step of its layer)
MERONEX_LIKE = {
    "gated residual update + norm": ("titatar", "residual update + norms"),
    "gated residual update + expert sum + norm": ("titatar", "residual update + expert sum + norms"),
    "gated residual update + two sides + norm": ("titatar", "residual update + norms"),
    "memory input projections (GEMM)": ("titatar", "windowed input projections (GEMM)"), "matrix memory": ("memory", "recurrent mixer"),
    "memory output projection (GEMM)": ("titatar", "windowed output projection (GEMM)"),
    "delta input projections (GEMM)": ("titatar", "windowed input projections (GEMM)"), "convolution + delta rule": ("delta", "recurrent mixer"),
    "delta output projection (GEMM)": ("titatar", "windowed output projection (GEMM)"),
    "parallel input projections (GEMM)": ("titatar", "windowed input projections (GEMM)"),
    "rotation + value norm + cache write": ("titatar", "q/k norm + rotation + cache write"), "capped attention": ("titatar", "windowed attention"),
    "attention output projection (GEMM)": ("titatar", "windowed output projection (GEMM)"),
    "token shift + its products (GEMM)": ("titatar", "windowed input projections (GEMM)"),
    "decay projection (GEMM)": ("titatar", "router (GEMM)"), "time mixing": ("time_mix", "recurrent mixer"),
    "time mixing output projection (GEMM)": ("titatar", "windowed output projection (GEMM)"),
    "router + gate (GEMM)": ("titatar", "router (GEMM)"), "routed experts": ("titatar", "routed experts"),
}


def meronex_like(cfg, phase):
    """Steps of a Titatar layer with the attention heads (no window) and the experts of the Meronex model, and of Rigulorn's state
    space with the heads and state sizes of its recurrent mixers: ``model -> {name: (fn, bytes, flops)}``."""
    import dataclasses
    from arctic_platform_b200.models import rigulorn, titatar
    mem, dlt, par = (next(s for s in cfg.layers if s.type == t) for t in ("mlstm", "delta", "parallel"))
    L, M = par.mixer.left, mem.mlp
    t = titatar.PRESETS["titatar-2048"]
    latent = next(s for s in t.layers if s.latent)
    window = titatar.WindowAttnSpec(L.heads, L.kv_heads, L.dim, L.vdim, L.scale, 0, L.rot)
    layers = (dataclasses.replace(latent, mlp=titatar.MoeSpec(M.experts, 0, M.top, M.ff)), titatar.LayerSpec(window, 2 * cfg.hidden_size))
    ops = {"titatar": titatar_ops(dataclasses.replace(t, hidden_size=cfg.hidden_size, layers=layers, loop=None), phase)}
    r = rigulorn.PRESETS["rigulorn-2048"]
    attn = next(s for s in r.layers if s.attention and s.ff)
    sizes = {"memory": (mem.mixer.heads, mem.mixer.vdim, mem.mixer.dim, mem.mixer.heads),
             "delta": (dlt.mixer.heads, dlt.mixer.vdim, dlt.mixer.dim, dlt.mixer.kv_heads),
             "time_mix": (par.mixer.right.heads, par.mixer.right.dim, par.mixer.right.dim, par.mixer.right.heads)}
    for name, (heads, vdim, dim, groups) in sizes.items():
        ssm = rigulorn.LayerSpec(rigulorn.Mamba2Spec(heads, vdim, dim, groups, 4, heads), attn.ff, attn.limit)
        ops[name] = rigulorn_ops(dataclasses.replace(r, hidden_size=cfg.hidden_size, layers=(attn, ssm)), phase)
    return {k: {n: rest for n, *rest in v} for k, v in ops.items()}


# step of a Titatar layer -> the like step of the dense decoder's layer (experts: of its mixture)
TITATAR_LIKE = {
    "residual update + norms": "norm + 2 input convolutions", "residual update + expert sum + norms": "norm + 2 input convolutions",
    "latent input projections (GEMM)": "input projections (GEMM)", "latent norms + cache write": "q/k norm + cache write",
    "query projection (GEMM)": "attention output projection (GEMM)", "latent attention": "attention",
    "latent output projection (GEMM)": "attention output projection (GEMM)",
    "windowed input projections (GEMM)": "input projections (GEMM)", "q/k norm + rotation + cache write": "q/k norm + cache write",
    "windowed attention": "attention", "windowed output projection (GEMM)": "attention output projection (GEMM)",
    "router (GEMM)": "router (GEMM)", "routed experts": "routed experts", "gate/up + SiLU (GEMM)": "gate/up + GELU (GEMM)",
    "down projection (GEMM)": "output projections (GEMM, += fp32)",
}


def titatar_like(cfg):
    """The layer sizes of the windowed attention and the dense feed-forward, in the form ``dense_ops`` takes."""
    from arctic_platform_b200.models.reninex import ReninexConfig, _uniform
    A = next(s for s in cfg.layers if not s.latent).mixer
    ff = next(s.mlp for s in cfg.layers if isinstance(s.mlp, int))
    layers = _uniform(1, (A.heads, A.kv_heads, A.dim, A.vdim), (2, 64, 64, 64), ff)
    return ReninexConfig(cfg.vocab_size, cfg.hidden_size, layers, cfg.norm_eps, 4, None, None, f"titatar-like-{cfg.hidden_size}")


def moe_config(cfg):
    """The decoder family's mixture-of-experts model beside a Titatar model: its windowed attention's heads, its experts without
    the identity ones, as many of them per token as Titatar chooses on average, one layer per run."""
    import dataclasses
    m = next(s.mlp for s in cfg.layers if not isinstance(s.mlp, int) and s.mlp is not None)
    return dataclasses.replace(dense_config(titatar_like(cfg)), num_layers=len(cfg.layer_runs()), num_experts=m.experts,
                               num_experts_per_tok=round(m.top * m.experts / m.scores), moe_intermediate_size=m.ff,
                               name=f"moe-{cfg.hidden_size}")


def meronex_moe_config(cfg):
    """The decoder family's mixture-of-experts model with the attention heads and experts of a Meronex model, one layer per layer."""
    from arctic_platform_b200.models.config import DecoderConfig
    L = next(s for s in cfg.layers if s.type == "parallel").mixer.left
    M = next(s.mlp for s in cfg.layers if s.mlp is not None)
    return DecoderConfig(vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, intermediate_size=M.ff, num_layers=cfg.num_layers,
                         num_heads=L.heads, num_kv_heads=L.kv_heads, head_dim=L.dim, tie_word_embeddings=False, num_experts=M.experts,
                         num_experts_per_tok=M.top, moe_intermediate_size=M.ff, name=f"moe-{cfg.hidden_size}")


def moe_ops(cfg, phase):
    import math
    from arctic_platform_b200.models.moe import MoEFeedForward
    from arctic_platform_b200.ops import gemm
    d = moe_config(cfg)
    n = PREFILL_SEQS * SEQ if phase == "prefill" else DECODE_SEQS
    W, F, E = d.hidden_size, d.moe_intermediate_size, d.num_experts
    ff = MoEFeedForward(d, "cuda", torch.bfloat16)
    for t in ff.parameters():
        t.data.normal_(std=0.02)
    x = _bf(n, W)
    pairs = n * d.num_experts_per_tok
    touched = E * (1 - math.exp(-pairs / E))

    def run():
        with torch.no_grad():
            ff._routed(x)
    return {"routed experts": (run, touched * 6 * W * F + 4 * n * W, 6 * pairs * W * F),
            "router (GEMM)": (lambda: gemm.matmul_nt(x, ff.router.data), 2 * (n * W + E * W + n * E), 2 * n * W * E)}


# step of a Rigulorn layer -> (model, the like step of its layer); products next to the dense decoder's of the same shape
RIGULORN_LIKE = {
    "stream update + norm": ("reninex", "norm + 2 input convolutions"),
    "attention input projections (GEMM)": ("dense", "input projections (GEMM)"),
    "rotation + cache write": ("reninex", "q/k norm + cache write"), "attention": ("reninex", "attention"),
    "attention output projection (GEMM)": ("dense", "attention output projection (GEMM)"),
    "gate/up + clamped GLU (GEMM)": ("dense", "gate/up + GELU (GEMM)"),
    "down projection (GEMM)": ("dense", "output projections (GEMM, += fp32)"),
    "state-space input projections (GEMM)": ("reninex", "input projections (GEMM)"),
    "recurrent mixer": ("reninex", "recurrent mixer"),
    "state-space output projection (GEMM)": ("reninex", "output projections (GEMM, += fp32)"),
}


def reninex_like(cfg):
    """The Reninex model whose layer has the K/V rows, state and feed-forward of the Rigulorn model's layers."""
    from arctic_platform_b200.models.reninex import ReninexConfig, _uniform
    a = next(s for s in cfg.layers if s.attention and s.ff)
    A, M = a.mixer, next(s for s in cfg.layers if not s.attention).mixer
    layers = _uniform(1, (A.heads, A.kv_heads, 2 * A.dim, A.vdim), (M.heads, M.state, M.vdim, M.state), a.ff)
    return ReninexConfig(cfg.vocab_size, cfg.hidden_size, layers, cfg.norm_eps, 4, None, None, f"reninex-like-{cfg.hidden_size}")


def like_ops(cfg, phase):
    """Steps of the closest older model, keyed by the names of ``stateful_ops``: ``name -> (fn, bytes, flops)``."""
    if cfg.architecture == "Meronex":
        ops = meronex_like(cfg, phase)
        return {mine: ops[model][theirs] for mine, (model, theirs) in MERONEX_LIKE.items()}
    if cfg.architecture == "Titatar":
        ops = {**dense_ops(titatar_like(cfg), phase), **moe_ops(cfg, phase)}
        return {mine: ops[theirs] for mine, theirs in TITATAR_LIKE.items()}
    if cfg.architecture != "Rigulorn":
        return dense_ops(cfg, phase)
    like = reninex_like(cfg)
    ops = {"reninex": {name: rest for name, *rest in reninex_ops(like, phase)}, "dense": dense_ops(like, phase)}
    return {mine: ops[model][theirs] for mine, (model, theirs) in RIGULORN_LIKE.items()}


def dense_config(cfg):
    """The Qwen3-style decoder with the width, heads and feed-forward of the model's attention layers, one layer per run."""
    from arctic_platform_b200.models.config import DecoderConfig
    if cfg.architecture == "Rigulorn":
        s = next(s for s in cfg.layers if s.attention and s.ff)
        heads, kv_heads, dim = s.mixer.heads, s.mixer.kv_heads, 2 * s.mixer.dim
    else:
        s = cfg.layers[0]
        heads, kv_heads, dim = s.left.heads, s.left.kv_heads, s.left.dim
    return DecoderConfig(vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, intermediate_size=s.ff,
                         num_layers=len(cfg.layer_runs()), num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
                         tie_word_embeddings=False, name=f"dense-{cfg.hidden_size}")


def dense_ops(cfg, phase):
    """The like steps of the dense layer (and of the gated delta rule), keyed by the names of ``stateful_ops``."""
    import dataclasses
    from arctic_platform_b200.engine.sampler import SamplerEngine, _fn
    from arctic_platform_b200.models.decoder import DecoderLM
    from arctic_platform_b200.models.linear_attention import gated_delta_rule_chunked
    from arctic_platform_b200.ops import _lib, gemm, norm
    from arctic_platform_b200.ops.attention import AttnLayout, attention_fwd_cuda
    d = dataclasses.replace(dense_config(cfg), num_layers=1, vocab_size=1024)
    R = cfg.layers[0].right
    n = PREFILL_SEQS if phase == "prefill" else DECODE_SEQS
    T = SEQ * n if phase == "prefill" else n
    keys = SEQ * (SEQ + 1) // 2 * n if phase == "prefill" else (SEQ + 1) * n
    W, D, Hq, G, ff = d.hidden_size, d.head_dim, d.num_heads, d.num_kv_heads, d.intermediate_size
    model = DecoderLM(d, "cuda", torch.bfloat16).init_weights(0)
    blk = model.blocks[0]
    eng = SamplerEngine(d, "cuda", model=model, kv_cache_tokens=(SEQ + 32) * n, max_batch=max(8, n), max_seq_len=SEQ + 32,
                        cascade=False, use_cuda_graph=False)
    x, res = _bf(T, W), _bf(T, W)
    qkv = _bf(T, d.qkv_size)
    act, qo = _bf(T, ff), _bf(T, d.q_size)
    pos = torch.arange(T, device="cuda", dtype=torch.int32) % SEQ
    slots = torch.arange(T, device="cuda", dtype=torch.int32)
    rope = model.rope("cuda")
    q, k, v = norm.qknorm_rope(qkv, blk.q_norm, blk.k_norm, *rope, pos, Hq, G, D, 1e-6)
    kv_row = 2 * G * D * 2
    acc, accq = torch.zeros(T, W, device="cuda"), torch.zeros(T, d.qkv_size, device="cuda")
    tiles = lambda m: (m + 127) // 128

    def qk_and_cache():
        qq, kk, vv = norm.qknorm_rope(qkv, blk.q_norm, blk.k_norm, *rope, pos, Hq, G, D, 1e-6)
        _lib.check(_fn("kvw")(_lib.ptr(kk), kk.stride(0), _lib.ptr(vv), vv.stride(0), _lib.ptr(slots),
                              _lib.ptr(eng.kcache[0]), _lib.ptr(eng.vcache[0]), T, G, D, _lib.stream_ptr()), "kvw")

    ops = {}
    if phase == "prefill":
        layout = AttnLayout.from_cu_seqlens(np.arange(n + 1) * SEQ)
        ops["attention"] = (lambda: attention_fwd_cuda(q, k, v.contiguous(), layout, D ** -0.5, need_lse=False),
                            T * kv_row + 4 * T * Hq * D, 4 * keys * Hq * D)
        ops["output projections (GEMM, += fp32)"] = (lambda: gemm.matmul_nt(act, blk.wdown),
                                                     2 * (T * ff + ff * W + T * W), 2 * T * ff * W)
        ops["attention output projection (GEMM)"] = (lambda: gemm.matmul_nt(qo, blk.wo), 2 * (T * d.q_size + d.q_size * W + T * W),
                                                     2 * T * d.q_size * W)
        ops["q/k norm + cache write"] = (qk_and_cache, 2 * T * 2 * Hq * D + 2 * T * kv_row, 0)
        ops["norm + 2 input convolutions"] = (lambda: norm.rmsnorm(x, blk.ln1, 1e-6, res), T * W * 8, 0)
        qr, kr, vr = (torch.randn(SEQ, R.heads, m, device="cuda") for m in (R.dim, R.dim, R.vdim))
        gr, br = -torch.rand(SEQ, R.heads, device="cuda") * 0.1, torch.rand(SEQ, R.heads, device="cuda")

        def delta():
            with torch.no_grad():
                for _ in range(n):
                    gated_delta_rule_chunked(qr, kr, vr, gr, br)
        ops["recurrent mixer"] = (delta, 2 * T * R.heads * (2 * R.dim + 3 * R.vdim) + n * R.heads * R.dim * R.vdim * 4,
                                  T * R.heads * (2 * 64 * (R.dim + R.vdim) / 2 + 4 * R.dim * R.vdim))
        ops["input projections (GEMM)"] = (lambda: gemm.matmul_nt(x, blk.wqkv), 2 * (T * W + d.qkv_size * (W + T)),
                                           2 * T * W * d.qkv_size)
        ops["gate/up + GELU (GEMM)"] = (lambda: gemm.gate_up_swiglu(x, blk.wgu, keep_gu=False),
                                        2 * (T * W + 2 * ff * W + T * ff), 4 * T * W * ff)
    else:
        per = SEQ // 16 + 1
        eng.d_page_table[:n, :per] = torch.from_numpy(np.random.default_rng(0).permutation(n * per).astype(np.int32).reshape(n, per)).cuda()
        eng.d_len[:n], eng.d_active[:n] = SEQ + 1, 1
        eng.kcache.normal_()
        eng.vcache.normal_()
        sd, sq = max(1, min(148 // tiles(W), (ff + 63) // 64)), max(1, min(148 // tiles(d.qkv_size), (W + 63) // 64))
        qb = torch.empty(T, Hq, D, device="cuda", dtype=torch.bfloat16)
        ops["attention"] = (lambda: eng._decode_attention(0, q, n), keys * kv_row + 4 * T * Hq * D, 4 * keys * Hq * D)
        ops["output projections (GEMM, += fp32)"] = (
            lambda: gemm.gemm_raw(act, blk.wdown, acc, M=T, N=W, K=ff, epi=gemm.EPI_F32_ATOMIC, splits=sd, bn=128),
            2 * (T * ff + ff * W) + 8 * T * W, 2 * T * ff * W)
        so = max(1, min(148 // tiles(W), (d.q_size + 63) // 64))
        ops["attention output projection (GEMM)"] = (
            lambda: gemm.gemm_raw(qo, blk.wo, acc, M=T, N=W, K=d.q_size, epi=gemm.EPI_F32_ATOMIC, splits=so, bn=128),
            2 * (T * d.q_size + d.q_size * W) + 8 * T * W, 2 * T * d.q_size * W)
        ops["q/k norm + cache write"] = (lambda: _lib.check(_fn("qkv_post")(
            _lib.ptr(accq), accq.stride(0), _lib.ptr(blk.q_norm), _lib.ptr(blk.k_norm), _lib.ptr(rope[0]), _lib.ptr(rope[1]),
            _lib.ptr(pos), _lib.ptr(slots), _lib.ptr(qb), _lib.ptr(eng.kcache[0]), _lib.ptr(eng.vcache[0]), T, Hq, G, D, 1e-6,
            _lib.stream_ptr()), "qkv_post"), 8 * T * d.qkv_size + 2 * T * Hq * D + T * kv_row, 0)
        ops["norm + 2 input convolutions"] = (lambda: eng._norm_f32(acc, blk.ln1, res), T * W * 14, 0)
        ops["input projections (GEMM)"] = (
            lambda: gemm.gemm_raw(x, blk.wqkv, accq, M=T, N=d.qkv_size, K=W, epi=gemm.EPI_F32_ATOMIC, splits=sq, bn=128),
            2 * (T * W + d.qkv_size * W) + 8 * T * d.qkv_size, 2 * T * W * d.qkv_size)
        ops["gate/up + GELU (GEMM)"] = (lambda: gemm.gemm_raw(x, blk.wgu, None, M=T, N=2 * ff, K=W, epi=gemm.EPI_SWIGLU,
                                                              out2=act, bn=0), 2 * (T * W + 2 * ff * W + T * ff), 4 * T * W * ff)
        S = torch.randn(n, R.heads, R.dim, R.vdim, device="cuda")
        ks, qs, vs = (torch.randn(n, R.heads, m, device="cuda") for m in (R.dim, R.dim, R.vdim))
        al = torch.rand(n, R.heads, device="cuda")

        def delta_step():                                 # the state part of GatedDeltaNet.step
            s2 = S * al[:, :, None, None]
            pred = torch.einsum("bhkv,bhk->bhv", s2, ks)
            s2 = s2 + torch.einsum("bhk,bhv->bhkv", ks, vs - pred)
            torch.einsum("bhkv,bhk->bhv", s2, qs)
        ops["recurrent mixer"] = (delta_step, 2 * T * R.heads * (2 * R.dim + 3 * R.vdim) + 2 * S.numel() * 4,
                                  T * R.heads * 4 * R.dim * R.vdim)
    ops["_keep"] = eng
    return ops


def bench_kernels(name, cfg, phase, iters, step=None, compare=True):
    bw, peak, of = peaks()
    timer = Timer(iters)

    def measured(fn, nbytes, flops):
        ms = timer(fn)
        floor = max(nbytes / bw, flops / peak) * 1e3
        return ms, floor, floor / ms

    like = {k: measured(*v) for k, v in like_ops(cfg, phase).items() if k != "_keep" and (step is None or step in k)} \
        if compare else {}
    torch.cuda.empty_cache()
    for op, fn, nbytes, flops in stateful_ops(cfg, phase):
        if step is not None and step not in op:
            continue
        ms, floor, frac = measured(fn, nbytes, flops)
        row = {"model": name, "phase": phase, "step": op, "ms": round(ms, 4), "floor_ms": round(floor, 4),
               "frac": round(frac, 3), "of": of}
        if op in like:
            row.update(like_ms=round(like[op][0], 4), like_frac=round(like[op][2], 3), ratio=round(frac / like[op][2], 2))
        print(json.dumps(row), flush=True)


def bench_engine(name, cfg, seqs, new_tokens):
    from arctic_platform_b200.engine.sampler import SamplerEngine
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.models import registry
    from arctic_platform_b200.models.config import resolve_config
    prompts = [np.random.default_rng(i).integers(1, cfg.vocab_size, SEQ).tolist() for i in range(seqs)]
    limits = dict(kv_cache_tokens=seqs * (SEQ + new_tokens + 32), max_batch=seqs, max_seq_len=SEQ + new_tokens + 16)
    older = {"Rigulorn": f"reninex-{cfg.hidden_size}", "Meronex": f"titatar-{cfg.hidden_size}"}.get(cfg.architecture)
    if cfg.architecture == "Meronex":
        models = [cfg, meronex_moe_config(cfg)]
    else:
        models = [cfg, moe_config(cfg) if cfg.architecture == "Titatar" else dense_config(cfg)]
    if older in registry.presets():
        models.append(resolve_config(older))
    for m in models:
        model = registry.new_model(m, "cuda", torch.bfloat16).init_weights(0)
        if registry.is_stateful(m):
            eng = StatefulSampler(m, "cuda", model=model, **limits)
        else:
            eng = SamplerEngine(m, "cuda", model=model, cascade=False, **limits)

        def run(n):
            torch.cuda.synchronize()
            t = time.perf_counter()
            eng.generate(prompts, {"temperature": 1.0, "max_tokens": n, "ignore_eos": True})
            torch.cuda.synchronize()
            return time.perf_counter() - t

        for n in (1, new_tokens):
            run(n)
        pre = statistics.median(run(1) for _ in range(3))
        full = statistics.median(run(new_tokens) for _ in range(3))
        params = sum(p.numel() for p in eng.model.parameters())
        print(json.dumps({
            "model": m.name, "engine": type(eng).__name__, "sequences": seqs, "prompt_len": SEQ, "new_tokens": new_tokens,
            "parameters": params, "layer_runs": len(m.layer_runs()) if registry.is_stateful(m) else m.num_layers,
            "prefill_tokens_per_s": round(seqs * SEQ / pre), "decode_tokens_per_s": round(seqs * (new_tokens - 1) / (full - pre)),
            "decode_ms_per_step": round((full - pre) * 1e3 / (new_tokens - 1), 3),
            "gflop_per_token": round(m.flops_per_token(SEQ, backward=False) / 1e9, 3),
            "prefill_tflops": round(seqs * SEQ / pre * (m.flops_per_token(SEQ, backward=False) - 2.0 * cfg.vocab_size * cfg.hidden_size) / 1e12, 1)}),
            flush=True)
        del eng, model
        torch.cuda.empty_cache()


def main(models, kernels_only=False, only=None, iters=20, seqs=64, new_tokens=129, step=None, compare=True) -> None:
    from arctic_platform_b200.models.config import resolve_config
    from arctic_platform_b200.ops import _lib
    for name in models:
        cfg = resolve_config(name)
        for phase in ("prefill", "decode"):
            if only in (None, phase):
                bench_kernels(name, cfg, phase, iters, step, compare)
                torch.cuda.empty_cache()
        if not kernels_only:
            bench_engine(name, cfg, seqs, new_tokens)
    _lib.check_status("serving benchmark")


if __name__ == "__main__":
    ap = argparse.ArgumentParser()
    ap.add_argument("--models", default="reninex-2048,reninex-4096,rigulorn-2048,rigulorn-4096,titatar-2048,titatar-4096,"
                                         "meronex-2048,meronex-4096")
    ap.add_argument("--kernels-only", action="store_true")
    ap.add_argument("--only", choices=["prefill", "decode", "none"], help="which kernels are timed")
    ap.add_argument("--step", help="only the steps whose name contains this")
    ap.add_argument("--no-compare", action="store_true", help="leave the dense kernels out")
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--seqs", type=int, default=64)
    ap.add_argument("--new-tokens", type=int, default=129)
    a = ap.parse_args()
    main(a.models.split(","), a.kernels_only, a.only, a.iters, a.seqs, a.new_tokens, a.step, not a.no_compare)
