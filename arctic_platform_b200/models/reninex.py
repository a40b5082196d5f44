"""Reninex: a decoder whose layers run two mixers side by side, beside the feed-forward, on one norm.

Per layer, with ``h = norm(x)`` (one gain per norm):

    x <- x + a_l * Left(h1) + a_r * Right(h1) + FF(h2),      h_k = h + causal depth-wise convolution_k(h)

* Left: attention with sigmoid weights (q and k normalised per head, a bias per head, no softmax, no rotation) over a
  paged K/V cache, grouped query heads;
* Right: retention -- linear attention with a fixed decay per head, rotary q and k, a per-head norm and a silu gate --
  with a constant-size fp32 state;
* FF: a gated tanh-GELU feed-forward (may be absent).

The embedding adds a hashed bigram row.  A range of layers can be run several times in a row with the same weights; a
pass starts from a projection of (stream, embedding output) plus a step vector, and keeps caches and states of its own.

The projections that read ``h1`` are one fused weight ``w_in`` (q, k, v of the left mixer, q, k, v, g of the right one),
gate and up are interleaved in ``w_gu``, and the three output projections are one weight ``w_out`` over the concatenated
activations, so a layer is three GEMMs; the mixers' scales are applied where the activations are produced and the last
GEMM accumulates onto the fp32 residual stream.  Every column group starts at a multiple of 8 (16-byte rows).
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Optional, Tuple

import torch
from torch import nn

from ..ops import norm, serving


@dataclass(frozen=True)
class SigmoidAttnSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float


@dataclass(frozen=True)
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class LayerSpec:
    left: SigmoidAttnSpec
    right: RetentionSpec
    left_scale: float
    right_scale: float
    ff: int                      # 0: no feed-forward


@dataclass
class ReninexConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    conv_taps: int = 0                                       # 0: no input convolutions
    bigram: Optional[Tuple[int, int, int]] = None            # buckets, multiplier of the previous / current token
    loop: Optional[Tuple[int, int, int]] = None              # start, stop, times
    name: str = "reninex"

    architecture = "Reninex"
    model_type = "reninex"
    # what the rest of the package asks a configuration for
    is_moe = False
    vlm_layout = False
    layer_types = None
    tie_word_embeddings = False

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def rms_norm_eps(self) -> float:
        return self.norm_eps

    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """Execution order: ``(layer, pass)`` with the pass number on the first layer of every pass, else ``None``."""
        a, b, times = self.loop if self.loop else (0, 0, 0)
        runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(a)]
        for t in range(times):
            runs += [(i, t if i == a else None) for i in range(a, b)]
        return runs + [(i, None) for i in range(b, self.num_layers)]

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(d: Dict[str, Any], name: str = "") -> "ReninexConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != "parallel":
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            m, mlp = e["mixer"], e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            L, R = m["left"], m["right"]
            if L["heads"] % L["kv_heads"]:
                raise ValueError(f"layer {i}: {L['heads']} query heads do not share {L['kv_heads']} key heads evenly")
            if len(R["decay"]) != R["heads"]:
                raise ValueError(f"layer {i}: {len(R['decay'])} decays for {R['heads']} heads")
            rot = R["rot"]
            if rot["dims"] % 2 or not 0 <= rot["dims"] <= R["dim"]:
                raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions of {R['dim']}")
            layers.append(LayerSpec(
                SigmoidAttnSpec(L["heads"], L["kv_heads"], L["dim"], L["vdim"], float(L["scale"])),
                RetentionSpec(R["heads"], R["dim"], R["vdim"], tuple(float(x) for x in R["decay"]), int(rot["dims"]),
                              float(rot["base"])),
                float(m["left_scale"]), float(m["right_scale"]), int(mlp["ff"]) if mlp is not None else 0))
        bg = (d.get("embedding") or {}).get("bigram")
        lp = d.get("loop")
        if lp and not (0 <= lp["start"] < lp["stop"] <= len(layers) and lp["times"] >= 1):
            raise ValueError(f"loop {lp} does not fit {len(layers)} layers")
        canon = d.get("canon")
        return ReninexConfig(
            vocab_size=d["vocab"], hidden_size=d["width"], layers=tuple(layers), norm_eps=float(d["norm"]["eps"]),
            conv_taps=int(canon["taps"]) if canon else 0,
            bigram=(int(bg["buckets"]), int(bg["mul_prev"]), int(bg["mul_cur"])) if bg else None,
            loop=(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None,
            name=name or "reninex")

    def to_hf_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "layers": []}
        if self.conv_taps:
            d["canon"] = {"taps": self.conv_taps}
        if self.bigram:
            d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))}
        if self.loop:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        for s in self.layers:
            L, R = s.left, s.right
            d["layers"].append({
                "type": "parallel",
                "mixer": {"left": {"heads": L.heads, "kv_heads": L.kv_heads, "dim": L.dim, "vdim": L.vdim,
                                   "scale": L.scale},
                          "right": {"heads": R.heads, "dim": R.dim, "vdim": R.vdim, "decay": list(R.decay),
                                    "rot": {"base": R.rot_base, "dims": R.rot_dims}},
                          "left_scale": s.left_scale, "right_scale": s.right_scale},
                "mlp": {"kind": "dense", "ff": s.ff} if s.ff else None})
        return d

    to_dict = to_hf_dict

    def tensor_names(self) -> List[str]:
        """Every tensor of a checkpoint, in the order of the layers."""
        names = ["embed"] + (["bigram"] if self.bigram else []) + (["loop.in", "loop.step"] if self.loop else [])
        for i, s in enumerate(self.layers):
            p = f"l{i}."
            names += [p + "norm1"] + [p + "mix.left." + n for n in ("q", "k", "v", "pb", "o")]
            names += [p + "mix.right." + n for n in ("q", "k", "v", "g", "o")]
            if s.ff:
                names += [p + "mlp." + n for n in ("gate", "up", "down")]
            if self.conv_taps:
                names += [p + "canon1"] + ([p + "canon2"] if s.ff else [])
        return names + ["final.norm", "head"]

    # ------------------------------------------------------------------ sizes
    def num_parameters(self, include_embeddings: bool = True) -> int:
        W, n = self.hidden_size, 1
        for s in self.layers:
            L, R = s.left, s.right
            n += W * (L.heads * (L.dim + L.vdim) + L.kv_heads * (L.dim + L.vdim)) + L.heads + 1
            n += W * R.heads * (2 * R.dim + 3 * R.vdim) + 3 * W * s.ff + W * self.conv_taps * (2 if s.ff else 1)
        if self.loop:
            n += 2 * W * W + self.loop[2] * W
        if include_embeddings:
            n += 2 * self.vocab_size * W + ((self.bigram[0] + 1) * W if self.bigram else 0)
        return n

    def flops_per_token(self, seq_len: int = 0, backward: bool = False) -> float:
        """Matmul FLOPs of one token (2 x weights, looped layers once per pass), attention over ``seq_len / 2`` keys on
        average and the retention update."""
        W, f = self.hidden_size, 2.0 * self.vocab_size * self.hidden_size
        for i, t in self.layer_runs():
            s = self.layers[i]
            L, R = s.left, s.right
            f += 2.0 * W * ((L.heads + L.kv_heads) * (L.dim + L.vdim) + R.heads * (2 * R.dim + 3 * R.vdim) + 3 * s.ff)
            f += 2.0 * L.heads * (L.dim + L.vdim) * seq_len / 2.0 + 4.0 * R.heads * R.dim * R.vdim
            f += 4.0 * W * W if t is not None else 0.0
        return f * (3.0 if backward else 1.0)


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _columns(sizes: Dict[str, int]) -> Tuple[Dict[str, Tuple[int, int]], int]:
    """Column groups laid side by side, each starting at a multiple of 8: name -> (first column, size), total."""
    out, o = {}, 0
    for n, s in sizes.items():
        out[n] = (o, s)
        o += _pad8(s)
    return out, o


class ReninexBlock(nn.Module):
    """Weights of one layer in the fused layouts, and the layer itself on a ragged serving batch."""

    def __init__(self, cfg: ReninexConfig, spec: LayerSpec, device, dtype):
        super().__init__()
        self.cfg, self.spec = cfg, spec
        L, R, W = spec.left, spec.right, cfg.hidden_size
        self.in_cols, n_in = _columns({
            "left.q": L.heads * L.dim, "left.k": L.kv_heads * L.dim, "left.v": L.kv_heads * L.vdim,
            "right.q": R.heads * R.dim, "right.k": R.heads * R.dim, "right.v": R.heads * R.vdim,
            "right.g": R.heads * R.vdim})
        self.out_cols, n_out = _columns({"left.o": L.heads * L.vdim, "right.o": R.heads * R.vdim, "down": spec.ff})
        self.padded = n_out != sum(s for _, s in self.out_cols.values())
        mk = lambda *s: nn.Parameter(torch.zeros(*s, device=device, dtype=dtype), requires_grad=False)
        self.norm1 = mk(1)
        self.w_in = mk(n_in, W)
        self.w_out = mk(W, n_out)
        self.pb = mk(L.heads)
        self.w_gu = mk(2 * spec.ff, W) if spec.ff else None
        self.canon1 = mk(cfg.conv_taps, W) if cfg.conv_taps else None       # [taps, W]
        self.canon2 = mk(cfg.conv_taps, W) if cfg.conv_taps and spec.ff else None
        self.register_buffer("log2_decay", torch.tensor(
            [math.log2(x) if x > 0 else float("-inf") for x in R.decay], dtype=torch.float32, device=device),
            persistent=False)

    def serve(self, b: serving.StepBatch, x: torch.Tensor, cache, run: int, rope) -> None:
        """Adds this layer's output onto the fp32 residual stream ``x [rows, W]``."""
        s, eps = self.spec, self.cfg.norm_eps
        L, R = s.left, s.right
        h1, h2 = serving.norm_conv(b, x, self.norm1, self.canon1, self.canon2, bool(s.ff), cache.conv[run],
                                   cache.parity, max(1, self.cfg.conv_taps), eps)
        p = serving.linear(h1, self.w_in)
        c, o = self.in_cols, self.out_cols
        alloc = torch.zeros if self.padded else torch.empty
        a = alloc((b.rows, self.w_out.shape[1]), device=x.device, dtype=h1.dtype)
        if s.ff:
            serving.gate_up_gelu(h2, self.w_gu, a[:, o["down"][0]:o["down"][0] + s.ff])
        serving.qk_norm_cache(b, p, (c["left.q"][0], c["left.k"][0], c["left.v"][0]), cache.k[run], cache.v[run],
                              L.heads, eps)
        serving.sigmoid_attention(b, p[:, c["left.q"][0]:], L.heads, cache.k[run], cache.v[run], self.pb, L.scale,
                                  a[:, o["left.o"][0]:], s.left_scale)
        serving.retention(b, p, tuple(c["right." + n][0] for n in "qkvg"), rope[R.rot_dims, R.rot_base], R.rot_dims,
                          self.log2_decay, cache.state[run], a[:, o["right.o"][0]:], eps, R.dim ** -0.5,
                          s.right_scale)
        serving.linear(a, self.w_out, x, accumulate=True)


class ReninexLM(nn.Module):
    def __init__(self, cfg: ReninexConfig, device="cuda", dtype=torch.bfloat16):
        super().__init__()
        self.cfg = cfg
        W = cfg.hidden_size
        mk = lambda *s: nn.Parameter(torch.zeros(*s, device=device, dtype=dtype), requires_grad=False)
        self.embed = mk(cfg.vocab_size, W)
        self.bigram = mk(cfg.bigram[0] + 1, W) if cfg.bigram else None
        self.loop_in = mk(W, 2 * W) if cfg.loop else None
        self.loop_step = mk(cfg.loop[2], W) if cfg.loop else None
        self.blocks = nn.ModuleList([ReninexBlock(cfg, s, device, dtype) for s in cfg.layers])
        self.final_norm = mk(1)
        self.head = mk(cfg.vocab_size, W)
        self._rope: Dict[Tuple[int, float], Tuple[torch.Tensor, torch.Tensor]] = {}
        self._rope_len = 0

    @property
    def dtype(self) -> torch.dtype:
        return self.embed.dtype

    @property
    def output_weight(self) -> torch.Tensor:
        return self.head

    # ------------------------------------------------------------------ weights
    def _place(self, name: str):
        """``(destination, transform)``: where the checkpoint tensor ``name`` lives inside the fused parameters."""
        top = {"embed": self.embed, "bigram": self.bigram, "loop.in": self.loop_in, "loop.step": self.loop_step,
               "head": self.head, "final.norm": self.final_norm}
        if name in top and top[name] is not None:
            return top[name].data, None
        parts = name.split(".")
        if parts[0][:1] != "l" or not parts[0][1:].isdigit() or int(parts[0][1:]) >= len(self.blocks):
            raise KeyError(f"unexpected tensor name {name!r}")
        blk, rest = self.blocks[int(parts[0][1:])], ".".join(parts[1:])
        if rest == "norm1":
            return blk.norm1.data, None
        if rest == "mix.left.pb":
            return blk.pb.data, None
        if rest in ("canon1", "canon2") and getattr(blk, rest) is not None:
            return getattr(blk, rest).data, "t"
        if rest in ("mlp.gate", "mlp.up") and blk.w_gu is not None:
            return blk.w_gu.data[(0 if rest == "mlp.gate" else 1)::2], None
        if rest == "mlp.down" and blk.w_gu is not None:
            o, n = blk.out_cols["down"]
            return blk.w_out.data[:, o:o + n], None
        if rest.startswith("mix."):
            key = rest[4:]
            for cols, w, dim in ((blk.in_cols, blk.w_in, 0), (blk.out_cols, blk.w_out, 1)):
                if key in cols:
                    o, n = cols[key]
                    return w.data.narrow(dim, o, n), None
        raise KeyError(f"unexpected tensor name {name!r}")

    @torch.no_grad()
    def load_named_tensor(self, name: str, t: torch.Tensor) -> None:
        dst, how = self._place(name)
        src = t.t() if how == "t" else (t.reshape(1) if t.dim() == 0 else t)
        if dst.shape != src.shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit")
        dst.copy_(src.to(device=dst.device, dtype=dst.dtype))

    def iter_named_tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        for name in self.cfg.tensor_names():
            t, how = self._place(name)
            yield name, (t.t() if how == "t" else t.reshape(()) if name.endswith("norm1") or name == "final.norm" else t)

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: float = 0.02) -> "ReninexLM":
        """Deterministic random weights keyed by tensor name (gains are ones, the head biases are -4)."""
        from .decoder import hash_name
        for name, t in self.iter_named_tensors():
            leaf = name.split(".")[-1]
            if leaf in ("norm1", "norm"):
                v = torch.ones(())
            elif leaf == "pb":
                v = torch.full(t.shape, -4.0)
            else:
                g = torch.Generator(device=t.device)
                g.manual_seed((hash_name(name) + seed) % (2 ** 31))
                v = torch.randn(t.shape, generator=g, dtype=torch.float32, device=t.device)
                v *= 0.1 if leaf.startswith("canon") else std
            self.load_named_tensor(name, v.to(self.dtype))
        return self

    # ------------------------------------------------------------------ serving protocol
    def cache_layout(self) -> List[Dict[str, tuple]]:
        """What every layer run keeps per sequence: paged K/V ``(kv heads, dim, vdim)``, recurrent state ``(heads, dim,
        vdim)``, convolution history ``(rows, width)``."""
        out = []
        for i, _ in self.cfg.layer_runs():
            L, R = self.cfg.layers[i].left, self.cfg.layers[i].right
            out.append({"kv": (L.kv_heads, L.dim, L.vdim), "state": (R.heads, R.dim, R.vdim),
                        "conv": (max(0, self.cfg.conv_taps - 1), self.cfg.hidden_size)})
        return out

    def prepare_serving(self, max_positions: int) -> None:
        """Position tables (one per distinct rotation), computed in float64."""
        dev = self.embed.device
        if self._rope_len < max_positions or any(t[0].device != dev for t in self._rope.values()):
            self._rope = {}
            for s in self.cfg.layers:
                key = (s.right.rot_dims, s.right.rot_base)
                if key not in self._rope:
                    self._rope[key] = norm.rope_tables(max_positions, max(2, key[0]), key[1], dev)
            self._rope_len = max_positions

    def serve_rows(self, b: serving.StepBatch, cache, on_layer=None) -> torch.Tensor:
        """Runs the layers over the batch, advancing caches and states; returns the residual stream ``[rows, W]`` fp32.
        ``on_layer(run, x)`` sees the stream after every layer run."""
        cfg, dev = self.cfg, self.embed.device
        W = cfg.hidden_size
        x = torch.empty((b.rows, W), device=dev, dtype=torch.float32)
        xx0 = torch.empty((b.rows, 2 * W), device=dev, dtype=self.dtype) if cfg.loop else None
        serving.embed(b, self.embed, self.bigram, cfg.bigram, cache.prev, x, xx0[:, W:] if cfg.loop else None)
        for run, (i, t) in enumerate(cfg.layer_runs()):
            if t is not None:
                serving.loop_begin(x, self.loop_step[t], xx0)
                serving.linear(xx0, self.loop_in, x, accumulate=True)
            self.blocks[i].serve(b, x, cache, run, self._rope)
            if on_layer is not None:
                on_layer(run, x)
        serving.commit(b, cache.prev, cache.parity)
        return x

    def output_rows(self, x: torch.Tensor, rows: Optional[torch.Tensor]) -> torch.Tensor:
        """Final norm of the chosen rows (None: all), in the activation type."""
        return serving.gain_norm_rows(x, rows, self.final_norm, self.cfg.norm_eps)

    def logits(self, h: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        return serving.linear(h, self.head, out, out_dtype=torch.float32)


def _decays(n: int) -> Tuple[float, ...]:
    return tuple(1.0 - 2.0 ** (-5 - 4.0 * i / max(1, n - 1)) for i in range(n))


def _uniform(n_layers: int, left, right, ff: int, left_scale: float = 0.7, right_scale: float = 0.6) -> Tuple[LayerSpec, ...]:
    H, G, D, E = left
    h, d, e, rot = right
    return (LayerSpec(SigmoidAttnSpec(H, G, D, E, D ** -0.5), RetentionSpec(h, d, e, _decays(h), rot, 10000.0),
                      left_scale, right_scale, ff),) * n_layers


PRESETS: Dict[str, ReninexConfig] = {
    "reninex-tiny": ReninexConfig(320, 128, _uniform(3, (4, 2, 64, 32), (2, 32, 64, 16), 256), 1e-5, 4, (101, 31, 5),
                                  (1, 2, 2), "reninex-tiny"),
    # layers of the size of a 1.7B / 8B dense decoder's
    "reninex-2048": ReninexConfig(151936, 2048, _uniform(8, (16, 8, 128, 128), (8, 128, 256, 128), 6144), 1e-6, 4,
                                  (65521, 1009, 37), (2, 6, 2), "reninex-2048"),
    "reninex-4096": ReninexConfig(151936, 4096, _uniform(8, (32, 8, 128, 128), (16, 128, 256, 128), 12288), 1e-6, 4,
                                  (65521, 1009, 37), (2, 6, 2), "reninex-4096"),
}
