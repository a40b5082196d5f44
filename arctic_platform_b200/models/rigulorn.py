"""Rigulorn: a decoder with parallel residual streams over differential attention and state-space (Mamba-2) mixers.

The residual is ``streams`` fp32 copies ``x_t`` of the scaled embedding.  A layer has a mixer and, optionally, a
feed-forward; each sublayer reads one combination of the streams and writes back into all of them:

    u = sum_t in[t] x_t;    y = sublayer(norm(u));    x_t <- sum_s mix[s, t] x_s + out[t] y

and the model's output is the norm of the streams' sum.  Mixers:

* attention: two softmax maps per head over the same values, combined as ``a1 - lambda a2`` and normalised per head; rotary
  positions on neighbouring pairs, capped scores, and chunks of positions outside of which nothing is visible.  A layer
  may read the keys and values of an earlier one (``kv_from``), which it then shares the cache with;
* mamba2: causal short convolution, selective state space with one decay per head and token, gate before a norm in groups.

The feed-forward is a clamped GLU, ``g sigmoid(1.702 g) (u + 1)``.

The projections that read one input are one fused weight (q, k, v; z, x, B, C, dt), gate and up are interleaved, and every
column group starts at a multiple of 8 (16-byte rows).  The update of the streams, the next sublayer's combination and its
norm are one kernel.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Optional, Tuple, Union

import torch
from torch import nn

from ..ops import norm, serving
from .reninex import _columns, _pad8


@dataclass(frozen=True)
class DiffAttnSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    diff: float
    chunk: int
    rot_dims: int
    rot_base: float
    kv_from: Optional[int] = None       # the layer whose keys and values this one reads


@dataclass(frozen=True)
class Mamba2Spec:
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[DiffAttnSpec, Mamba2Spec]
    ff: int = 0                          # 0: no feed-forward
    limit: float = 0.0

    @property
    def attention(self) -> bool:
        return isinstance(self.mixer, DiffAttnSpec)


@dataclass
class RigulornConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    streams: int = 1
    embed_scale: float = 1.0
    name: str = "rigulorn"

    architecture = "Rigulorn"
    model_type = "rigulorn"
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
        return [(i, None) for i in range(self.num_layers)]

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(d: Dict[str, Any], name: str = "") -> "RigulornConfig":
        layers: List[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            m, mlp = e["mixer"], e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            if e["type"] == "attention":
                rot, src = m["rot"], m.get("kv_from")
                if m["heads"] % m["kv_heads"]:
                    raise ValueError(f"layer {i}: {m['heads']} query heads do not share {m['kv_heads']} key heads evenly")
                if rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"]:
                    raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions of {m['dim']}")
                mixer: Union[DiffAttnSpec, Mamba2Spec] = DiffAttnSpec(
                    m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), float(m.get("softcap") or 0.0),
                    float(m["diff"]), int((m.get("mask") or {}).get("size", 0)), int(rot["dims"]), float(rot["base"]), src)
                if src is not None:
                    o = layers[src].mixer if 0 <= src < i else None
                    if not isinstance(o, DiffAttnSpec) or o.kv_from is not None or \
                            (o.kv_heads, o.dim, o.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                        raise ValueError(f"layer {i}: layer {src} has no keys and values that fit")
            elif e["type"] == "mamba2":
                mixer = Mamba2Spec(m["heads"], m["vdim"], m["state"], m["groups"], int(m["conv"]), m["norm_groups"])
                if mixer.heads % mixer.groups or mixer.inner % mixer.norm_groups or mixer.taps < 1:
                    raise ValueError(f"layer {i}: {m} does not divide evenly")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            layers.append(LayerSpec(mixer, int(mlp["ff"]) if mlp else 0, float(mlp["limit"]) if mlp else 0.0))
        if d["streams"] < 1:
            raise ValueError(f"{d['streams']} residual streams")
        return RigulornConfig(vocab_size=d["vocab"], hidden_size=d["width"], layers=tuple(layers),
                              norm_eps=float(d["norm"]["eps"]), streams=int(d["streams"]),
                              embed_scale=float(d["embedding"]["scale"]), name=name or "rigulorn")

    def to_hf_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "streams": self.streams,
                             "embedding": {"scale": self.embed_scale}, "layers": []}
        for s in self.layers:
            m = s.mixer
            if s.attention:
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                         "softcap": m.softcap, "diff": m.diff, "mask": {"size": m.chunk},
                         "rot": {"base": m.rot_base, "dims": m.rot_dims}}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            else:
                mixer = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.taps,
                         "norm_groups": m.norm_groups}
            d["layers"].append({"type": "attention" if s.attention else "mamba2", "mixer": mixer,
                                "mlp": {"kind": "dense", "ff": s.ff, "limit": s.limit} if s.ff else None})
        return d

    to_dict = to_hf_dict

    def tensor_names(self) -> List[str]:
        """Every tensor of a checkpoint, in the order of the layers."""
        names = ["embed"]
        for i, s in enumerate(self.layers):
            p = f"l{i}."
            names += [p + "norm1"] + ([p + "norm2"] if s.ff else [])
            if s.attention:
                own = () if s.mixer.kv_from is not None else ("k", "v")
                mix = ("q",) + own + ("lq1", "lk1", "lq2", "lk2", "o")
            else:
                mix = ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")
            names += [p + "mix." + n for n in mix]
            if s.ff:
                names += [p + "mlp." + n for n in ("gate", "up", "down")]
            names += [p + f"hc{q}.{n}" for q in ((1, 2) if s.ff else (1,)) for n in ("in", "out", "mix")]
        return names + ["final.norm", "head"]

    # ------------------------------------------------------------------ sizes
    def _layer_weights(self, s: LayerSpec) -> int:
        W, m = self.hidden_size, s.mixer
        if s.attention:
            own = 0 if m.kv_from is not None else m.kv_heads * (2 * m.dim + m.vdim)
            return W * (2 * m.heads * m.dim + own + m.heads * m.vdim + 3 * s.ff)
        return W * (2 * m.inner + 2 * m.groups * m.state + m.heads + m.inner + 3 * s.ff)

    def num_parameters(self, include_embeddings: bool = True) -> int:
        W, S, n = self.hidden_size, self.streams, self.hidden_size
        for s in self.layers:
            m = s.mixer
            n += self._layer_weights(s) + (2 if s.ff else 1) * (W + S * (S + 2))
            n += 4 * m.dim if s.attention else m.channels * (m.taps + 1) + 3 * m.heads + m.inner
        return n + (2 * self.vocab_size * W if include_embeddings else 0)

    def flops_per_token(self, seq_len: int = 0, backward: bool = False) -> float:
        """Matmul FLOPs of one token (2 x weights), attention over the keys its chunk leaves on average, the state update."""
        f = 2.0 * self.vocab_size * self.hidden_size
        for s in self.layers:
            m = s.mixer
            f += 2.0 * self._layer_weights(s)
            if s.attention:
                f += 2.0 * m.heads * (2 * m.dim + 2 * m.vdim) * min(seq_len, m.chunk or seq_len) / 2.0
            else:
                f += 4.0 * m.inner * m.state
        return f * (3.0 if backward else 1.0)


class _Sublayer(nn.Module):
    """Norm and stream weights in front of and behind a mixer or a feed-forward."""

    def __init__(self, cfg: RigulornConfig, mk):
        super().__init__()
        S = cfg.streams
        self.norm, self.hc_in, self.hc_out, self.hc_mix = mk(cfg.hidden_size), mk(S), mk(S), mk(S, S)


class _AttentionMixer(nn.Module):
    def __init__(self, cfg: RigulornConfig, m: DiffAttnSpec, mk):
        super().__init__()
        self.m = m
        own = {"k": m.kv_heads * 2 * m.dim, "v": m.kv_heads * m.vdim} if m.kv_from is None else {}
        self.in_cols, n_in = _columns({"q": m.heads * 2 * m.dim, **own})
        self.n_out = m.heads * m.vdim
        self.w_in, self.w_out = mk(n_in, cfg.hidden_size), mk(cfg.hidden_size, _pad8(self.n_out))
        self.lq1, self.lk1, self.lq2, self.lk2 = mk(m.dim), mk(m.dim), mk(m.dim), mk(m.dim)
        self.register_buffer("lam", torch.zeros(1, dtype=torch.float32, device=self.lq1.device), persistent=False)
        self.spec = serving.SoftmaxSpec(m.scale, m.softcap, m.chunk, 2, 1.0 - m.diff, cfg.norm_eps)

    def refresh(self) -> None:
        """The second map's weight, after its four vectors changed."""
        dot = lambda a, b: torch.exp((a.data.float() * b.data.float()).sum())
        self.lam.copy_(dot(self.lq1, self.lk1) - dot(self.lq2, self.lk2) + self.m.diff)

    def place(self, key: str):
        if key in self.in_cols:
            o, n = self.in_cols[key]
            return self.w_in.data.narrow(0, o, n), None
        if key == "o":
            return self.w_out.data.narrow(1, 0, self.n_out), None
        if key in ("lq1", "lk1", "lq2", "lk2"):
            return getattr(self, key).data, None
        return None

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y: torch.Tensor, cache, run: int, rope) -> None:
        m, c = self.m, self.in_cols
        p = serving.linear(h, self.w_in)
        kc, vc = cache.k[run], cache.v[run]
        serving.rope_cache(b, p, tuple(c[n][0] for n in c), rope[m.rot_dims, m.rot_base], m.rot_dims, 2 * m.heads, m.dim, kc, vc,
                           write=m.kv_from is None)
        a = _activations(b.rows, self.n_out, h)
        serving.softmax_attention(b, p, m.heads, kc, vc, self.spec, self.lam, a)
        serving.project(a, self.w_out, y)


class _Mamba2Mixer(nn.Module):
    def __init__(self, cfg: RigulornConfig, m: Mamba2Spec, mk):
        super().__init__()
        self.m, self.eps = m, cfg.norm_eps
        self.in_cols, n_in = _columns({"z": m.inner, "xbc": m.channels, "dt": m.heads})
        self.w_in, self.w_out = mk(n_in, cfg.hidden_size), mk(cfg.hidden_size, _pad8(m.inner))
        self.conv, self.conv_bias = mk(m.taps, m.channels), mk(m.channels)
        self.dt_bias, self.a_log, self.skip, self.gain = mk(m.heads), mk(m.heads), mk(m.heads), mk(m.inner)

    def place(self, key: str):
        plain = {"conv.b": self.conv_bias, "dt_bias": self.dt_bias, "A_log": self.a_log, "D": self.skip, "norm": self.gain}
        if key in plain:
            return plain[key].data, None
        if key == "conv":
            return self.conv.data, "t"
        if key == "in":
            return [self.w_in.data.narrow(0, o, n) for o, n in self.in_cols.values()], None
        if key == "o":
            return self.w_out.data.narrow(1, 0, self.m.inner), None
        return None

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y: torch.Tensor, cache, run: int, rope) -> None:
        m, c = self.m, self.in_cols
        p = serving.linear(h, self.w_in)
        w = serving.SsmWeights(self.conv, self.conv_bias, self.dt_bias, self.a_log, self.skip)
        s = serving.state_space(b, p, c["xbc"][0], c["dt"][0], w, m.groups, cache.conv[run], cache.parity, cache.state[run])
        a = _activations(b.rows, m.inner, h)
        serving.gated_group_norm(s, p, self.gain, m.norm_groups, self.eps, a)
        serving.project(a, self.w_out, y)


class _FeedForward(nn.Module):
    def __init__(self, cfg: RigulornConfig, ff: int, limit: float, mk):
        super().__init__()
        self.ff, self.limit = ff, limit
        self.w_gu, self.w_down = mk(2 * ff, cfg.hidden_size), mk(cfg.hidden_size, _pad8(ff))

    def place(self, key: str):
        if key in ("gate", "up"):
            return self.w_gu.data[(0 if key == "gate" else 1)::2], None
        return (self.w_down.data.narrow(1, 0, self.ff), None) if key == "down" else None

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y: torch.Tensor, cache, run: int, rope) -> None:
        a = _activations(b.rows, self.ff, h)
        serving.gate_up_clamped(h, self.w_gu, a[:, :self.ff], self.limit)
        serving.project(a, self.w_down, y)


def _activations(rows: int, n: int, like: torch.Tensor) -> torch.Tensor:
    """Room for ``n`` columns, padded to a multiple of 8 with zeros (the padding meets zero weights)."""
    alloc = torch.zeros if n % 8 else torch.empty
    return alloc((rows, _pad8(n)), device=like.device, dtype=like.dtype)


class RigulornBlock(nn.Module):
    """Weights of one layer in the fused layouts."""

    def __init__(self, cfg: RigulornConfig, spec: LayerSpec, mk):
        super().__init__()
        self.spec = spec
        self.sub1 = _Sublayer(cfg, mk)
        self.mixer = (_AttentionMixer if spec.attention else _Mamba2Mixer)(cfg, spec.mixer, mk)
        self.sub2 = _Sublayer(cfg, mk) if spec.ff else None
        self.mlp = _FeedForward(cfg, spec.ff, spec.limit, mk) if spec.ff else None

    def place(self, rest: str):
        head, _, key = rest.partition(".")
        subs = {"1": self.sub1, "2": self.sub2}
        if rest in ("norm1", "norm2") and subs[rest[-1]] is not None:
            return subs[rest[-1]].norm.data, None
        if head in ("hc1", "hc2") and key in ("in", "out", "mix") and subs[head[-1]] is not None:
            return getattr(subs[head[-1]], "hc_" + key).data, None
        if head == "mix":
            return self.mixer.place(key)
        return self.mlp.place(key) if head == "mlp" and self.mlp is not None else None

    def sublayers(self):
        yield self.sub1, self.mixer
        if self.mlp is not None:
            yield self.sub2, self.mlp


class RigulornLM(nn.Module):
    def __init__(self, cfg: RigulornConfig, device="cuda", dtype=torch.bfloat16):
        super().__init__()
        self.cfg = cfg
        mk = lambda *s: nn.Parameter(torch.zeros(*s, device=device, dtype=dtype), requires_grad=False)
        self.embed = mk(cfg.vocab_size, cfg.hidden_size)
        self.blocks = nn.ModuleList([RigulornBlock(cfg, s, mk) for s in cfg.layers])
        self.final_norm = mk(cfg.hidden_size)
        self.head = mk(cfg.vocab_size, cfg.hidden_size)
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
        """``(destination or list of row ranges, transform)``: where the checkpoint tensor ``name`` lives."""
        top = {"embed": self.embed, "head": self.head, "final.norm": self.final_norm}
        if name in top:
            return top[name].data, None
        layer, _, rest = name.partition(".")
        found = None
        if layer[:1] == "l" and layer[1:].isdigit() and int(layer[1:]) < len(self.blocks):
            found = self.blocks[int(layer[1:])].place(rest)
        if found is None:
            raise KeyError(f"unexpected tensor name {name!r}")
        return found

    @torch.no_grad()
    def load_named_tensor(self, name: str, t: torch.Tensor) -> None:
        dst, how = self._place(name)
        parts = dst if isinstance(dst, list) else [dst]
        src = t.t() if how == "t" else t
        rows = sum(p.shape[0] for p in parts)
        if src.dim() != parts[0].dim() or src.shape[0] != rows or src.shape[1:] != parts[0].shape[1:]:
            raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit")
        for p, s in zip(parts, src.split([p.shape[0] for p in parts])):
            p.copy_(s.to(device=p.device, dtype=p.dtype))
        if name.rsplit(".", 1)[-1] in ("lq1", "lk1", "lq2", "lk2"):
            self.blocks[int(name.split(".")[0][1:])].mixer.refresh()

    def iter_named_tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        for name in self.cfg.tensor_names():
            t, how = self._place(name)
            t = torch.cat(t) if isinstance(t, list) else t
            yield name, t.t() if how == "t" else t

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: float = 0.02) -> "RigulornLM":
        """Deterministic random weights keyed by tensor name (gains are ones, streams start as an average that is written
        back to all of them, decays spread over the heads)."""
        from .decoder import hash_name
        S = self.cfg.streams
        for name, t in self.iter_named_tensors():
            leaf = name.split(".", 1)[-1]
            if leaf in ("norm1", "norm2", "mix.norm") or name == "final.norm" or leaf == "mix.D":
                v = torch.ones(t.shape)
            elif leaf in ("hc1.in", "hc2.in"):
                v = torch.full(t.shape, 1.0 / S)
            elif leaf in ("hc1.out", "hc2.out"):
                v = torch.ones(t.shape)
            elif leaf in ("hc1.mix", "hc2.mix"):
                v = torch.eye(S)
            elif leaf == "mix.A_log":
                v = torch.log(torch.linspace(1.0, 16.0, t.numel()))
            elif leaf == "mix.dt_bias":
                v = torch.linspace(-6.0, -2.0, t.numel())
            else:
                g = torch.Generator(device=t.device)
                g.manual_seed((hash_name(name) + seed) % (2 ** 31))
                v = torch.randn(t.shape, generator=g, dtype=torch.float32, device=t.device)
                v *= 0.3 if leaf == "mix.conv" else 0.1 if leaf[4:6] in ("lq", "lk") else std
            self.load_named_tensor(name, v.to(self.dtype))
        return self

    # ------------------------------------------------------------------ serving protocol
    def cache_layout(self) -> List[Dict[str, Any]]:
        """What every layer keeps per sequence: paged K/V ``(kv heads, key row, value row)`` or the layer it borrows them from,
        or recurrent state ``(heads, state, vdim)`` and convolution history ``(rows, channels)``."""
        out: List[Dict[str, Any]] = []
        for s in self.cfg.layers:
            m = s.mixer
            if not s.attention:
                out.append({"state": (m.heads, m.state, m.vdim), "conv": (m.taps - 1, m.channels)})
            elif m.kv_from is not None:
                out.append({"kv_from": m.kv_from})
            else:
                out.append({"kv": (m.kv_heads, 2 * m.dim, m.vdim)})
        return out

    def prepare_serving(self, max_positions: int) -> None:
        """Position tables (one per distinct rotation), computed in float64."""
        dev = self.embed.device
        if self._rope_len < max_positions or any(t[0].device != dev for t in self._rope.values()):
            self._rope = {}
            for s in self.cfg.layers:
                key = (s.mixer.rot_dims, s.mixer.rot_base) if s.attention else None
                if key is not None and key not in self._rope:
                    self._rope[key] = norm.rope_tables(max_positions, max(2, key[0]), key[1], dev)
            self._rope_len = max_positions

    def serve_rows(self, b: serving.StepBatch, cache, on_layer=None) -> torch.Tensor:
        """Runs the layers over the batch, advancing caches and states; returns the sum of the residual streams ``[rows, W]``
        fp32.  ``on_layer(run, x)`` sees that sum after every layer."""
        cfg, dev = self.cfg, self.embed.device
        W, eps = cfg.hidden_size, cfg.norm_eps
        x = torch.empty((b.rows, cfg.streams, W), device=dev, dtype=torch.float32)
        serving.embed(b, self.embed, None, None, cache.prev, x, scale=cfg.embed_scale)
        clear = serving.accumulates(b.rows, W, dev)            # products of few rows are added onto a zeroed y
        y = (torch.zeros if clear else torch.empty)((b.rows, W), device=dev, dtype=torch.float32)
        last: Optional[_Sublayer] = None
        for run, blk in enumerate(self.blocks):
            for sub, body in blk.sublayers():
                h = serving.stream_step(x, y if last else None, last.hc_mix if last else None, last.hc_out if last else None,
                                        sub.hc_in, sub.norm, eps, clear=clear)
                body.serve(b, h, y, cache, run, self._rope)
                last = sub
            if on_layer is not None:
                on_layer(run, serving.stream_step(x, y, last.hc_mix, last.hc_out, None, None, eps, write=False))
        serving.commit(b, cache.prev, cache.parity)
        return serving.stream_step(x, y if last else None, last.hc_mix if last else None, last.hc_out if last else None, None,
                                   None, eps, write=False, dtype=self.dtype)

    def output_rows(self, x: torch.Tensor, rows: Optional[torch.Tensor]) -> torch.Tensor:
        """Final norm of the chosen rows (None: all), in the activation type."""
        return serving.gain_norm_rows(x, rows, self.final_norm, self.cfg.norm_eps)

    def logits(self, h: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        return serving.linear(h, self.head, out, out_dtype=torch.float32)


def _stack(n: int, attn: DiffAttnSpec, ssm: Mamba2Spec, ff: int, limit: float = 7.0, ssm_ff: bool = False) -> Tuple[LayerSpec, ...]:
    """``n`` layers: state-space mixers in front of every third attention layer; the last attention layer borrows its keys."""
    import dataclasses
    out: List[LayerSpec] = []
    for i in range(n):
        if i % 3 == 0:
            out.append(LayerSpec(ssm, ff if ssm_ff else 0, limit if ssm_ff else 0.0))
        else:
            src = max((j for j, s in enumerate(out) if s.attention and s.mixer.kv_from is None), default=None)
            borrow = i == n - 1 and src is not None
            out.append(LayerSpec(dataclasses.replace(attn, kv_from=src) if borrow else attn, ff, limit))
    return tuple(out)


PRESETS: Dict[str, RigulornConfig] = {
    "rigulorn-tiny": RigulornConfig(320, 128, _stack(4, DiffAttnSpec(4, 2, 16, 32, 0.25, 30.0, 0.2, 96, 16, 10000.0),
                                                     Mamba2Spec(6, 32, 16, 2, 4, 3), 256), 1e-5, 2, 4.0, "rigulorn-tiny"),
    # layers of the size of a 1.7B / 8B dense decoder's
    "rigulorn-2048": RigulornConfig(151936, 2048, _stack(12, DiffAttnSpec(16, 8, 64, 128, 0.125, 30.0, 0.2, 8192, 64, 10000.0),
                                                         Mamba2Spec(64, 64, 128, 8, 4, 8), 6144, ssm_ff=True), 1e-6, 4, 2.0,
                                    "rigulorn-2048"),
    "rigulorn-4096": RigulornConfig(151936, 4096, _stack(12, DiffAttnSpec(32, 8, 64, 128, 0.125, 30.0, 0.2, 8192, 64, 10000.0),
                                                         Mamba2Spec(128, 64, 128, 8, 4, 8), 12288, ssm_ff=True), 1e-6, 4, 2.0,
                                    "rigulorn-4096"),
}
