"""Meronex: recurrent mixers of three kinds beside softmax attention, gated sublayers, mixtures of experts.

    x <- x + m sigmoid(G h + b) * sublayer(h),     h = norm(x) in equal groups of the width, one m for the model

Mixers:

* mlstm: matrix memory with exponential input and forget gates (soft-capped), a normaliser and a running maximum;
* delta: gated delta rule; q, k, v behind a short convolution, q and k unit vectors shared by groups of value heads;
* parallel: attention (rotary positions on half-split pairs with YaRN frequencies, normed values, capped scores) and time mixing
  (blends with the previous token, a decay per key channel from a low-rank projection, a bonus for the current token) on the same
  input; half the sum of their normed outputs.

Feed-forward: a mixture of clamped GLU experts with sigmoid scores; a token's weight multiplies the expert's input.

The projections that read one input are one fused weight, the sublayer's gate among them (for the mixture beside the router, in
fp32), gate and up are interleaved, and every column group starts at a multiple of 8 (16-byte rows).  The sum of the chosen experts
or the norms of two sides, the gate, the residual update and the next norm are one kernel.  The rank of the decay projection is
that of the checkpoint's tensors.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Optional, Tuple, Union

import torch
from torch import nn

from ..ops import gemm, norm, serving
from .reninex import _columns, _pad8
from .rigulorn import _activations
from .titatar import RotSpec, _read_rot, _write_rot

DEFAULT_RANK = 64                        # of a decay projection, until a checkpoint says otherwise


@dataclass(frozen=True)
class MemorySpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class CappedAttnSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float                       # 0: none
    rot: RotSpec


@dataclass(frozen=True)
class TimeMixSpec:
    heads: int
    dim: int


@dataclass(frozen=True)
class ParallelSpec:
    left: CappedAttnSpec
    right: TimeMixSpec


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    ff: int
    limit: float


MixerSpec = Union[MemorySpec, DeltaSpec, ParallelSpec]
_TYPES = {"mlstm": MemorySpec, "delta": DeltaSpec, "parallel": ParallelSpec}


@dataclass(frozen=True)
class LayerSpec:
    mixer: MixerSpec
    mlp: Optional[MoeSpec] = None

    @property
    def type(self) -> str:
        return next(n for n, c in _TYPES.items() if isinstance(self.mixer, c))


def _read_mixer(kind: str, m: Dict[str, Any], where: str) -> MixerSpec:
    if kind == "mlstm":
        return MemorySpec(m["heads"], m["dim"], m["vdim"], float(m["gate_cap"]))
    if kind == "delta":
        if m["heads"] % m["kv_heads"] or int(m["conv"]) < 1:
            raise ValueError(f"{where}: {m} does not divide evenly")
        return DeltaSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], int(m["conv"]))
    if kind != "parallel":
        raise ValueError(f"{where}: unknown mixer type {kind!r}")
    a, r = m["left"], m["right"]
    rot = _read_rot(a["rot"])
    if a["heads"] % a["kv_heads"]:
        raise ValueError(f"{where}: {a['heads']} query heads do not share {a['kv_heads']} key heads evenly")
    if rot.dims % 2 or not 0 <= rot.dims <= a["dim"]:
        raise ValueError(f"{where}: {rot.dims} rotated dimensions of {a['dim']}")
    return ParallelSpec(CappedAttnSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), float(a.get("softcap") or 0.0), rot),
                        TimeMixSpec(r["heads"], r["dim"]))


def _write_mixer(m: MixerSpec) -> Dict[str, Any]:
    if isinstance(m, MemorySpec):
        return {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
    if isinstance(m, DeltaSpec):
        return {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps}
    a = m.left
    left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale, "rot": _write_rot(a.rot)}
    if a.softcap:
        left["softcap"] = a.softcap
    return {"left": left, "right": {"heads": m.right.heads, "dim": m.right.dim}}


@dataclass
class MeronexConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    norm_groups: int = 1
    residual_mult: float = 1.0
    name: str = "meronex"

    architecture = "Meronex"
    model_type = "meronex"
    # what the rest of the package asks a configuration for (the engine's own expert switches are the dense decoder's)
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
        return [(i, None) for i in range(self.num_layers)]

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(d: Dict[str, Any], name: str = "") -> "MeronexConfig":
        layers: List[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            mixer, mlp, ff = _read_mixer(e["type"], e["mixer"], f"layer {i}"), e.get("mlp"), None
            if mlp is not None:
                if mlp.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
                r, x = mlp["router"], mlp["expert"]
                ff = MoeSpec(int(r["experts"]), int(r["top"]), int(x["ff"]), float(x["limit"]))
                if not 1 <= ff.top <= min(32, ff.experts) or ff.experts > 512 or ff.limit <= 0:
                    raise ValueError(f"layer {i}: {ff.top} of {ff.experts} experts, limit {ff.limit}")
            layers.append(LayerSpec(mixer, ff))
        groups = int(d["norm"].get("groups") or 1)
        if groups < 1 or d["width"] % groups:
            raise ValueError(f"{groups} norm groups do not divide a width of {d['width']}")
        return MeronexConfig(vocab_size=d["vocab"], hidden_size=d["width"], layers=tuple(layers), norm_eps=float(d["norm"]["eps"]),
                             norm_groups=groups, residual_mult=float(d.get("residual_mult", 1.0)), name=name or "meronex")

    def to_hf_dict(self) -> Dict[str, Any]:
        layers = [{"type": s.type, "mixer": _write_mixer(s.mixer),
                   "mlp": None if s.mlp is None else {"kind": "moe", "expert": {"ff": s.mlp.ff, "limit": s.mlp.limit},
                                                      "router": {"experts": s.mlp.experts, "top": s.mlp.top}}} for s in self.layers]
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "residual_mult": self.residual_mult, "layers": layers}

    to_dict = to_hf_dict

    def tensor_names(self) -> List[str]:
        """Every tensor of a checkpoint, in the order of the layers."""
        names = ["embed"]
        for i, s in enumerate(self.layers):
            p = f"l{i}."
            names += [p + n for n in (("norm1",) if s.mlp is None else ("norm1", "norm2"))]
            names += [p + "mix." + n for n in _MIXERS[s.type].NAMES]
            if s.mlp is not None:
                names += [p + f"mlp.e{e}.{n}" for e in range(s.mlp.experts) for n in ("gate", "up", "down")] + [p + "mlp.router"]
            names += [p + f"rg{n}{leaf}" for n in ((1,) if s.mlp is None else (1, 2)) for leaf in ("", ".b")]
        return names + ["final.norm", "head"]

    # ------------------------------------------------------------------ sizes
    def _mixer_weights(self, s: LayerSpec) -> Tuple[int, int]:
        """Weights of the mixer's products (the sublayer's gate included), and of its vectors."""
        W, m = self.hidden_size, s.mixer
        if isinstance(m, MemorySpec):
            out = m.heads * m.vdim
            return W * (2 * m.heads * m.dim + 3 * out + 2 * m.heads + W), 2 * m.heads + out + W
        if isinstance(m, DeltaSpec):
            qk, out = 2 * m.kv_heads * m.dim, m.heads * m.vdim
            return W * (qk + 3 * out + 2 * m.heads + W), (qk + out) * m.taps + 2 * m.heads + m.vdim + W
        a, inner = m.left, m.right.heads * m.right.dim
        return (W * (a.heads * (a.dim + a.vdim) + a.kv_heads * (a.dim + a.vdim) + 5 * inner + W) + DEFAULT_RANK * (W + inner),
                3 * inner + 8 * W)

    def num_parameters(self, include_embeddings: bool = True) -> int:
        W = n = self.hidden_size
        for s in self.layers:
            n += sum(self._mixer_weights(s)) + W
            if s.mlp is not None:
                n += W * (s.mlp.experts * (3 * s.mlp.ff + 1) + W + 2)
        return n + (2 * self.vocab_size * W if include_embeddings else 0)

    def flops_per_token(self, seq_len: int = 0, backward: bool = False) -> float:
        """Matmul FLOPs of one token (2 x the weights it meets), attention over the keys it sees on average, the state updates."""
        W, out = self.hidden_size, 2.0 * self.vocab_size * self.hidden_size
        for s in self.layers:
            m = s.mixer
            out += 2.0 * self._mixer_weights(s)[0]
            if isinstance(m, ParallelSpec):
                out += 2.0 * m.left.heads * (m.left.dim + m.left.vdim) * seq_len / 2.0 + 4.0 * m.right.heads * m.right.dim ** 2
            else:
                out += (6.0 if isinstance(m, DeltaSpec) else 4.0) * m.heads * m.dim * m.vdim
            if s.mlp is not None:
                out += 2.0 * W * (3.0 * s.mlp.ff * s.mlp.top + s.mlp.experts + W)
        return out * (3.0 if backward else 1.0)


Placed = Optional[torch.Tensor]


class _MemoryMixer(nn.Module):
    NAMES = ("q", "k", "v", "g", "o", "norm", "i", "i.b", "f", "f.b")

    def __init__(self, cfg: MeronexConfig, m: MemorySpec, mk):
        super().__init__()
        W, H = cfg.hidden_size, m.heads
        self.m, self.n_out = m, H * m.vdim
        self.in_cols, n_in = _columns({"q": H * m.dim, "k": H * m.dim, "v": self.n_out, "g": self.n_out, "i": H, "f": H, "rg": W})
        self.w_in, self.w_out = mk(n_in, W), mk(W, _pad8(self.n_out))
        self.gain, self.i_bias, self.f_bias = mk(self.n_out), mk(H), mk(H)
        self.spec = serving.RecurrentSpec("memory", H, H, m.dim, m.vdim, cfg.norm_eps, cap=m.gate_cap, silu=False)

    def place(self, key: str) -> Placed:
        if key in self.in_cols:
            return self.w_in.data.narrow(0, *self.in_cols[key])
        return {"o": self.w_out.data.narrow(1, 0, self.n_out), "norm": self.gain.data, "i.b": self.i_bias.data,
                "f.b": self.f_bias.data}.get(key)

    def cache_layout(self) -> Dict[str, Any]:
        return {"state": (self.m.heads, self.m.dim, self.m.vdim), "aux": (self.m.heads, self.m.dim + 1)}

    def inputs(self, p: torch.Tensor) -> serving.RecurrentInputs:
        c = {n: o for n, (o, _) in self.in_cols.items()}
        return serving.RecurrentInputs(p, c["q"], c["k"], c["v"], c["g"], self.i_bias, self.f_bias, self.gain, c["i"], c["f"])

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y, cache, run: int, rope) -> Dict[str, Any]:
        p = serving.linear(h, self.w_in)
        a = _activations(b.rows, self.n_out, h)
        serving.recurrent(b, self.spec, self.inputs(p), cache.state[run], a, aux=cache.aux[run])
        serving.project(a, self.w_out, y[0])
        return {"y": y[0], "gate": p[:, self.in_cols["rg"][0]:]}


class _DeltaMixer(nn.Module):
    NAMES = ("q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "A_log", "norm", "a", "dt_bias", "g", "o")

    def __init__(self, cfg: MeronexConfig, m: DeltaSpec, mk):
        super().__init__()
        W, H, n_qk = cfg.hidden_size, m.heads, m.kv_heads * m.dim
        self.m, self.n_out = m, H * m.vdim
        self.qkv = {"q": (0, n_qk), "k": (n_qk, n_qk), "v": (2 * n_qk, self.n_out)}          # side by side, as the convolution reads them
        self.in_cols, n_in = _columns({"qkv": 2 * n_qk + self.n_out, "g": self.n_out, "a": H, "b": H, "rg": W})
        self.w_in, self.w_out = mk(n_in, W), mk(W, _pad8(self.n_out))
        self.conv = mk(m.taps, 2 * n_qk + self.n_out)
        self.gain, self.a_log, self.dt_bias = mk(m.vdim), mk(H), mk(H)
        self.spec = serving.RecurrentSpec("delta", H, m.kv_heads, m.dim, m.vdim, cfg.norm_eps, shared_gain=True)

    def place(self, key: str) -> Placed:
        head, _, leaf = key.partition(".")
        if head in self.qkv and leaf in ("", "conv"):
            o, n = self.qkv[head]
            return self.conv.data.narrow(1, o, n).t() if leaf else self.w_in.data.narrow(0, o, n)
        if key in ("g", "a", "b", "rg"):
            return self.w_in.data.narrow(0, *self.in_cols[key])
        return {"o": self.w_out.data.narrow(1, 0, self.n_out), "norm": self.gain.data, "A_log": self.a_log.data,
                "dt_bias": self.dt_bias.data}.get(key)

    def cache_layout(self) -> Dict[str, Any]:
        return {"state": (self.m.heads, self.m.dim, self.m.vdim), "conv": (self.m.taps - 1, self.spec.channels)}

    def inputs(self, p: torch.Tensor) -> serving.RecurrentInputs:
        c = {n: o for n, (o, _) in self.in_cols.items()}
        q, k, v = (self.qkv[n][0] for n in "qkv")
        return serving.RecurrentInputs(p, q, k, v, c["g"], self.a_log, self.dt_bias, self.gain, c["a"], c["b"], conv=self.conv)

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y, cache, run: int, rope) -> Dict[str, Any]:
        p = serving.linear(h, self.w_in)
        a = _activations(b.rows, self.n_out, h)
        serving.recurrent(b, self.spec, self.inputs(p), cache.state[run], a, hist=cache.conv[run], parity=cache.parity)
        serving.project(a, self.w_out, y[0])
        return {"y": y[0], "gate": p[:, self.in_cols["rg"][0]:]}


class _ParallelMixer(nn.Module):
    """Attention and time mixing on one input.  Leaves their outputs in the two buffers of ``y``, not yet normed."""
    SHIFTS = "rkvgw"
    NAMES = tuple("left." + n for n in "qkvo") + tuple("right.mu." + s for s in SHIFTS) + \
        tuple("right." + n for n in ("r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o")) + ("left.out", "right.out")

    def __init__(self, cfg: MeronexConfig, m: ParallelSpec, mk):
        super().__init__()
        W, L, R = cfg.hidden_size, m.left, m.right
        self.m, self.eps, self.mk = m, cfg.norm_eps, mk
        self.in_cols, n_in = _columns({"q": L.heads * L.dim, "k": L.kv_heads * L.dim, "v": L.kv_heads * L.vdim, "rg": W})
        self.n_left, self.n_right = L.heads * L.vdim, R.heads * R.dim
        self.w_in, self.w_left, self.w_right = mk(n_in, W), mk(W, _pad8(self.n_left)), mk(W, _pad8(self.n_right))
        self.mu = mk(len(self.SHIFTS), W)
        self.w0, self.bonus, self.gain = mk(self.n_right), mk(self.n_right), mk(self.n_right)
        self.left_out, self.right_out = mk(W), mk(W)
        self.step = _pad8(self.n_right)                    # rows per product of the shifted inputs
        self.w_shift = self.w_rank = None
        self.set_rank(DEFAULT_RANK)
        self.softmax = serving.SoftmaxSpec(L.scale, cap=L.softcap)
        self.spec = serving.RecurrentSpec("time_mix", R.heads, R.heads, R.dim, R.dim, cfg.norm_eps)

    def set_rank(self, rank: int) -> None:
        """Room for a decay projection of this rank; the other weights stay.  The last product's rows fill whole tiles."""
        old, self.rank = self.w_shift, rank
        self.w_shift = self.mk(4 * self.step + (rank + 127) // 128 * 128, self.mu.shape[1])
        self.w_rank = self.mk(self.n_right, _pad8(rank))
        if old is not None:
            self.w_shift.data[:4 * self.step].copy_(old.data[:4 * self.step])

    def place(self, key: str, shape=None) -> Placed:
        side, _, name = key.partition(".")
        if key in ("rg",) or (side == "left" and name in ("q", "k", "v")):
            return self.w_in.data.narrow(0, *self.in_cols[name or key])
        if side == "right" and name in ("w1", "w2"):
            if shape is not None and shape[0 if name == "w1" else 1] != self.rank:
                self.set_rank(shape[0 if name == "w1" else 1])
            return self.w_shift.data.narrow(0, 4 * self.step, self.rank) if name == "w1" else self.w_rank.data.narrow(1, 0, self.rank)
        if side == "right" and name in ("r", "k", "v", "g"):
            return self.w_shift.data.narrow(0, self.SHIFTS.index(name) * self.step, self.n_right)
        if side == "right" and name[:3] == "mu." and name[3:] and name[3:] in self.SHIFTS:
            return self.mu.data[self.SHIFTS.index(name[3:])]
        R = self.m.right
        return {"left.o": self.w_left.data.narrow(1, 0, self.n_left), "right.o": self.w_right.data.narrow(1, 0, self.n_right),
                "right.w0": self.w0.data, "right.u": self.bonus.data.view(R.heads, R.dim), "right.norm": self.gain.data,
                "left.out": self.left_out.data, "right.out": self.right_out.data}.get(key)

    def cache_layout(self) -> Dict[str, Any]:
        L, R = self.m.left, self.m.right
        return {"kv": (L.kv_heads, L.dim, L.vdim), "state": (R.heads, R.dim, R.dim), "conv": (1, self.mu.shape[1])}

    def inputs(self, s: torch.Tensor, z: torch.Tensor) -> serving.RecurrentInputs:
        n = s.stride(0)
        return serving.RecurrentInputs(s[0], 0, n, 2 * n, 3 * n, self.w0, self.bonus, self.gain, z=z)

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y, cache, run: int, rope) -> Dict[str, Any]:
        L, c = self.m.left, self.in_cols
        p = serving.linear(h, self.w_in)
        kc, vc = cache.k[run], cache.v[run]
        serving.half_rope_cache(b, p, (c["q"][0], c["k"][0], c["v"][0]), rope[L.rot], L.rot.dims, L.heads, kc, vc, self.eps)
        a = _activations(b.rows, self.n_left, h)
        serving.softmax_attention(b, p, L.heads, kc, vc, self.softmax, None, a)
        serving.project(a, self.w_left, y[0])
        s = serving.token_shift(b, h, self.mu, cache.conv[run], cache.parity, self.w_shift, self.step, [self.n_right] * 4 + [self.rank])
        low = s[4][:, :self.rank]
        serving.tanh_rows(low)
        z = serving.linear(low, self.w_rank[:, :self.rank], out_dtype=torch.float32)
        a = _activations(b.rows, self.n_right, h)
        serving.recurrent(b, self.spec, self.inputs(s, z), cache.state[run], a)
        serving.project(a, self.w_right, y[1])
        return {"y": y[0], "post": self.left_out, "y2": y[1], "post2": self.right_out, "gate": p[:, c["rg"][0]:], "share": 0.5}


_MIXERS = {"mlstm": _MemoryMixer, "delta": _DeltaMixer, "parallel": _ParallelMixer}


class _Mixture(nn.Module):
    """Routed experts that weigh their input; the router and the sublayer's gate are one product.  Returns the experts unsummed."""

    def __init__(self, cfg: MeronexConfig, s: MoeSpec, mk):
        super().__init__()
        W = cfg.hidden_size
        self.s = s
        self.z_cols, n_z = _columns({"router": s.experts, "rg": W})
        self.w_z, self.w_gu, self.w_down = mk(n_z, W), mk(s.experts * 2 * s.ff, W), mk(s.experts * W, _pad8(s.ff))
        self.register_buffer("counters", torch.zeros(s.experts + 1, dtype=torch.int32, device=self.w_z.device), persistent=False)

    def place(self, key: str) -> Placed:
        s = self.s
        if key in self.z_cols:
            return self.w_z.data.narrow(0, *self.z_cols[key])
        head, _, leaf = key.partition(".")
        if head[:1] == "e" and head[1:].isdigit() and int(head[1:]) < s.experts:
            e, W = int(head[1:]), self.w_gu.shape[1]
            if leaf in ("gate", "up"):
                return self.w_gu.data[2 * s.ff * e:2 * s.ff * (e + 1)][(0 if leaf == "gate" else 1)::2]
            if leaf == "down":
                return self.w_down.data[W * e:W * (e + 1), :s.ff]
        return None

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y, cache, run: int, rope) -> Dict[str, Any]:
        s = self.s
        z = serving.linear(h, self.w_z, out_dtype=torch.float32)
        mix = serving.experts(b, h, z, None, self.counters, self.w_gu, self.w_down, s.experts, s.experts, s.top, s.ff, sigmoid=True,
                              scale_input=True, epi=gemm.EPI_CLAMP_GLU, limit=s.limit)
        return {"mix": mix, "gate": z[:, self.z_cols["rg"][0]:]}


class MeronexBlock(nn.Module):
    """Weights of one layer in the fused layouts."""

    def __init__(self, cfg: MeronexConfig, spec: LayerSpec, mk):
        super().__init__()
        self.spec = spec
        W, two = cfg.hidden_size, spec.mlp is not None
        self.mixer = _MIXERS[spec.type](cfg, spec.mixer, mk)
        self.mlp = _Mixture(cfg, spec.mlp, mk) if two else None
        self.norm1, self.gate_bias1 = mk(W), mk(W)
        self.norm2, self.gate_bias2 = (mk(W), mk(W)) if two else (None, None)

    def place(self, rest: str, shape=None) -> Placed:
        head, _, key = rest.partition(".")
        bodies = {"1": self.mixer, "2": self.mlp}
        if head in ("rg1", "rg2") and bodies[head[2]] is not None:
            return bodies[head[2]].place("rg") if not key else getattr(self, "gate_bias" + head[2]).data if key == "b" else None
        if rest in ("norm1", "norm2"):
            w = getattr(self, rest)
            return None if w is None else w.data
        if head == "mix" and key != "rg":
            return self.mixer.place(key, shape) if isinstance(self.mixer, _ParallelMixer) else self.mixer.place(key)
        return self.mlp.place(key) if head == "mlp" and key != "rg" and self.mlp is not None else None

    def sublayers(self):
        """``(norm ahead, body, bias of its gate)``"""
        yield self.norm1, self.mixer, self.gate_bias1
        if self.mlp is not None:
            yield self.norm2, self.mlp, self.gate_bias2


class MeronexLM(nn.Module):
    def __init__(self, cfg: MeronexConfig, device="cuda", dtype=torch.bfloat16):
        super().__init__()
        self.cfg = cfg
        mk = lambda *s: nn.Parameter(torch.zeros(*s, device=device, dtype=dtype), requires_grad=False)
        self.embed = mk(cfg.vocab_size, cfg.hidden_size)
        self.blocks = nn.ModuleList([MeronexBlock(cfg, s, mk) for s in cfg.layers])
        self.final_norm = mk(cfg.hidden_size)
        self.head = mk(cfg.vocab_size, cfg.hidden_size)
        self._rope: Dict[RotSpec, Tuple[torch.Tensor, torch.Tensor]] = {}
        self._rope_len = 0

    @property
    def dtype(self) -> torch.dtype:
        return self.embed.dtype

    @property
    def output_weight(self) -> torch.Tensor:
        return self.head

    # ------------------------------------------------------------------ weights
    def _place(self, name: str, shape=None) -> torch.Tensor:
        """Where the checkpoint tensor ``name`` (of this shape) lives inside the fused parameters."""
        top = {"embed": self.embed, "head": self.head, "final.norm": self.final_norm}
        if name in top:
            return top[name].data
        layer, _, rest = name.partition(".")
        found = None
        if layer[:1] == "l" and layer[1:].isdigit() and int(layer[1:]) < len(self.blocks):
            found = self.blocks[int(layer[1:])].place(rest, shape)
        if found is None:
            raise KeyError(f"unexpected tensor name {name!r}")
        return found

    @torch.no_grad()
    def load_named_tensor(self, name: str, t: torch.Tensor) -> None:
        dst = self._place(name, t.shape)
        if dst.shape != t.shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit")
        dst.copy_(t.to(device=dst.device, dtype=dst.dtype))

    def iter_named_tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        for name in self.cfg.tensor_names():
            yield name, self._place(name)

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: float = 0.02) -> "MeronexLM":
        """Deterministic random weights keyed by tensor name (gains are ones, gates start half open, decays spread over heads and
        channels)."""
        from .decoder import hash_name
        for name, t in self.iter_named_tensors():
            leaf, n = name.split(".", 1)[-1], t.numel()
            if leaf in ("norm", "norm1", "norm2", "mix.norm", "mix.right.norm", "mix.left.out", "mix.right.out"):
                v = torch.ones(t.shape)
            elif leaf in ("rg1.b", "rg2.b", "mix.i.b"):
                v = torch.zeros(t.shape)
            elif leaf == "mix.f.b":
                v = torch.linspace(3.0, 6.0, n)
            elif leaf == "mix.A_log":
                v = torch.log(torch.linspace(1.0, 16.0, n))
            elif leaf in ("mix.dt_bias", "mix.right.w0"):
                v = torch.linspace(-6.0, -1.0, n)
            elif leaf[:13] == "mix.right.mu." or leaf == "mix.right.u":
                v = torch.full(t.shape, 0.5)
            else:
                g = torch.Generator(device=t.device)
                g.manual_seed((hash_name(name) + seed) % (2 ** 31))
                v = torch.randn(t.shape, generator=g, dtype=torch.float32, device=t.device) * (0.3 if leaf.endswith(".conv") else std)
            self.load_named_tensor(name, v.to(self.dtype))
        return self

    # ------------------------------------------------------------------ serving protocol
    def cache_layout(self) -> List[Dict[str, Any]]:
        """What every layer keeps per sequence: paged K/V ``(kv heads, key row, value row)``, recurrent state ``(heads, dim, vdim)`` and
        its companions (``aux``), the inputs of the tokens before (``conv``) of a convolution or a blend."""
        return [blk.mixer.cache_layout() for blk in self.blocks]

    def prepare_serving(self, max_positions: int) -> None:
        """Position tables (one per distinct rotation), computed in float64."""
        dev = self.embed.device
        if self._rope_len < max_positions or any(t[0].device != dev for t in self._rope.values()):
            self._rope = {}
            for s in self.cfg.layers:
                r = s.mixer.left.rot if isinstance(s.mixer, ParallelSpec) else None
                if r is not None and r not in self._rope:
                    self._rope[r] = norm.rope_tables(max_positions, max(2, r.dims), r.base, dev, r.yarn if r.dims else None)
            self._rope_len = max_positions

    def serve_rows(self, b: serving.StepBatch, cache, on_layer=None) -> torch.Tensor:
        """Runs the layers over the batch, advancing caches and states; returns the residual ``[rows, W]`` fp32.  ``on_layer(run, x)``
        sees it after every layer."""
        cfg, dev = self.cfg, self.embed.device
        W = cfg.hidden_size
        x = torch.empty((b.rows, W), device=dev, dtype=torch.float32)
        serving.embed(b, self.embed, None, None, cache.prev, x)
        clear = serving.accumulates(b.rows, W, dev)            # products of few rows are added onto a zeroed y
        sides = 2 if any(isinstance(s.mixer, ParallelSpec) for s in cfg.layers) else 1
        y = [(torch.zeros if clear else torch.empty)((b.rows, W), device=dev, dtype=torch.float32) for _ in range(sides)]
        how = dict(eps=cfg.norm_eps, offset=0.0, groups=cfg.norm_groups)
        left: Dict[str, Any] = dict(y=None, post=None)         # the last sublayer's output, not yet in x
        for run, blk in enumerate(self.blocks):
            for pre, body, bias in blk.sublayers():
                h = serving.residual_step(x, pre=pre, clear=clear, **how, **left)
                out = body.serve(b, h, y, cache, run, self._rope)
                left = dict(dict(y=None, post=None), gate_bias=bias, mult=cfg.residual_mult * out.pop("share", 1.0))
                left.update(out)
            if on_layer is not None:
                on_layer(run, serving.residual_step(x, pre=None, write=False, **how, **left))
        serving.commit(b, cache.prev, cache.parity)
        return serving.residual_step(x, pre=None, write=False, dtype=self.dtype, **how, **left)

    def output_rows(self, x: torch.Tensor, rows: Optional[torch.Tensor]) -> torch.Tensor:
        """Final norm of the chosen rows (None: all), in the activation type."""
        return serving.gain_norm_rows(x, rows, self.final_norm, self.cfg.norm_eps, groups=self.cfg.norm_groups)

    def logits(self, h: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        return serving.linear(h, self.head, out, out_dtype=torch.float32)


def _stack(n: int, memory: MemorySpec, delta: DeltaSpec, parallel: ParallelSpec, moe: MoeSpec) -> Tuple[LayerSpec, ...]:
    """``n`` layers, the three mixers in turn."""
    return tuple(LayerSpec((memory, delta, parallel)[i % 3], moe) for i in range(n))


_YARN = norm.Yarn(4.0, 4096.0, 32.0, 1.0)

PRESETS: Dict[str, MeronexConfig] = {
    "meronex-tiny": MeronexConfig(320, 128, _stack(4, MemorySpec(3, 32, 48, 8.0), DeltaSpec(4, 2, 32, 40, 3), ParallelSpec(
        CappedAttnSpec(4, 2, 32, 48, 0.18, 25.0, RotSpec(16, 10000.0, _YARN)), TimeMixSpec(4, 24)), MoeSpec(6, 2, 64, 2.0)), 1e-5, 4, 0.6,
        "meronex-tiny"),
    # layers of the size of a 1.7B / 8B dense decoder's
    "meronex-2048": MeronexConfig(151936, 2048, _stack(12, MemorySpec(16, 128, 128, 15.0), DeltaSpec(16, 8, 128, 128, 4), ParallelSpec(
        CappedAttnSpec(16, 8, 128, 128, 128 ** -0.5, 30.0, RotSpec(128, 10000.0, _YARN)), TimeMixSpec(32, 64)), MoeSpec(64, 5, 768, 7.0)),
        1e-6, 2, 0.7, "meronex-2048"),
    "meronex-4096": MeronexConfig(151936, 4096, _stack(12, MemorySpec(32, 128, 128, 15.0), DeltaSpec(32, 16, 128, 128, 4), ParallelSpec(
        CappedAttnSpec(32, 8, 128, 128, 128 ** -0.5, 30.0, RotSpec(128, 10000.0, _YARN)), TimeMixSpec(64, 64)), MoeSpec(64, 5, 1536, 7.0)),
        1e-6, 2, 0.7, "meronex-4096"),
}
