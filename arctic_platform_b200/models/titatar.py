"""Titatar: latent attention and windowed attention layers with sinks and output gates, mixtures of experts, norms on both sides
of every sublayer.

    x <- x + norm_b(sublayer(norm_a(x)))             norm(x) = x / rms(x) * (1 + w)

Mixers:

* attention: grouped query heads over a sliding window; q and k normed over the whole projection, rotary positions (dimension i
  with i + dims/2), a softmax whose denominator contains one more ``exp(0)``, and one output gate per head;
* latent attention: queries through a normed latent, keys and values as projections of one normed latent per token that is all
  the cache keeps, beside one rotated key part shared by the heads (neighbouring pairs, YaRN frequencies); a learned sink per
  head and an output gate per column.

Feed-forward: a gated SiLU layer, or a mixture of such experts with softmax scores, a correction that only the choice sees,
identity experts and a shared expert.  A range of layers can run several times in a row with the same weights, each pass with
caches of its own; the embedding output is added to the residual ahead of every pass but the first.

The projections that read one input are one fused weight, gate and up are interleaved, and every column group starts at a
multiple of 8 (16-byte rows).  The sum of the chosen experts, the second norm of a sublayer, the residual update and the first
norm of the next sublayer are one kernel.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Iterator, List, Optional, Tuple, Union

import torch
from torch import nn

from ..ops import norm, serving
from .reninex import _columns, _pad8
from .rigulorn import _activations


@dataclass(frozen=True)
class RotSpec:
    dims: int
    base: float
    yarn: Optional[norm.Yarn] = None


@dataclass(frozen=True)
class WindowAttnSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                          # 0: none
    rot: RotSpec


@dataclass(frozen=True)
class LatentAttnSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotSpec


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    identity: int
    top: int
    ff: int
    shared_ff: int = 0                   # 0: no shared expert

    @property
    def scores(self) -> int:
        return self.experts + self.identity


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[WindowAttnSpec, LatentAttnSpec]
    mlp: Union[int, MoeSpec, None] = None         # dense feed-forward of that width, or a mixture, or none

    @property
    def latent(self) -> bool:
        return isinstance(self.mixer, LatentAttnSpec)


def _read_rot(d: Dict[str, Any]) -> RotSpec:
    sc = d.get("scaling")
    return RotSpec(int(d["dims"]), float(d["base"]),
                   norm.Yarn(*(float(sc[n]) for n in ("factor", "original", "fast", "slow"))) if sc else None)


def _write_rot(r: RotSpec) -> Dict[str, Any]:
    d: Dict[str, Any] = {"dims": r.dims, "base": r.base}
    if r.yarn:
        d["scaling"] = {n: getattr(r.yarn, n) for n in ("factor", "original", "fast", "slow")}
    return d


@dataclass
class TitatarConfig:
    vocab_size: int
    hidden_size: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float
    embed_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None              # start, stop, times
    name: str = "titatar"

    architecture = "Titatar"
    model_type = "titatar"
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
        """Execution order: ``(layer, pass)`` with the pass number on the first layer of every pass, else ``None``."""
        a, b, times = self.loop if self.loop else (0, 0, 0)
        runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(a)]
        for t in range(times):
            runs += [(i, t if i == a else None) for i in range(a, b)]
        return runs + [(i, None) for i in range(b, self.num_layers)]

    # ------------------------------------------------------------------ config.json
    @staticmethod
    def from_dict(d: Dict[str, Any], name: str = "") -> "TitatarConfig":
        layers: List[LayerSpec] = []
        for i, e in enumerate(d["layers"]):
            m, mlp = e["mixer"], e.get("mlp")
            rot = _read_rot(m["rot"])
            if e["type"] == "attention":
                if m["heads"] % m["kv_heads"]:
                    raise ValueError(f"layer {i}: {m['heads']} query heads do not share {m['kv_heads']} key heads evenly")
                if rot.dims % 2 or not 0 <= rot.dims <= m["dim"]:
                    raise ValueError(f"layer {i}: {rot.dims} rotated dimensions of {m['dim']}")
                mixer: Union[WindowAttnSpec, LatentAttnSpec] = WindowAttnSpec(
                    m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), int((m.get("mask") or {}).get("size", 0)), rot)
                if mixer.window < 0:
                    raise ValueError(f"layer {i}: a window of {mixer.window} positions")
            elif e["type"] == "latent_attention":
                mixer = LatentAttnSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]), rot)
                if rot.dims != mixer.rot_dim or rot.dims % 2:
                    raise ValueError(f"layer {i}: {rot.dims} rotated dimensions of a rotated part of {mixer.rot_dim}")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            ff: Union[int, MoeSpec, None] = None
            if mlp is not None:
                kind = mlp.get("kind", "dense")
                if kind == "dense":
                    ff = int(mlp["ff"])
                elif kind == "moe":
                    r, shared = mlp["router"], mlp.get("shared")
                    ff = MoeSpec(int(r["experts"]), int(r.get("identity") or 0), int(r["top"]), int(mlp["expert"]["ff"]),
                                 int(shared["ff"]) if shared else 0)
                    if not 1 <= ff.top <= min(32, ff.scores) or ff.experts < 1 or ff.scores > 512:
                        raise ValueError(f"layer {i}: {ff.top} of {ff.experts} + {ff.identity} experts")
                else:
                    raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
            layers.append(LayerSpec(mixer, ff))
        lp = d.get("loop")
        if lp and not (0 <= lp["start"] < lp["stop"] <= len(layers) and lp["times"] >= 1):
            raise ValueError(f"loop {lp} does not fit {len(layers)} layers")
        return TitatarConfig(vocab_size=d["vocab"], hidden_size=d["width"], layers=tuple(layers), norm_eps=float(d["norm"]["eps"]),
                             embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                             loop=(int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else None, name=name or "titatar")

    def to_hf_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale}, "layers": []}
        if self.loop:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        for s in self.layers:
            m, f = s.mixer, s.mlp
            mixer: Dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": _write_rot(m.rot)}
            if s.latent:
                mixer.update(rot_dim=m.rot_dim, q_rank=m.q_rank, kv_rank=m.kv_rank)
            else:
                mixer["kv_heads"] = m.kv_heads
                if m.window:
                    mixer["mask"] = {"size": m.window}
            mlp: Optional[Dict[str, Any]] = None
            if isinstance(f, MoeSpec):
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "identity": f.identity, "top": f.top}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            elif f is not None:
                mlp = {"kind": "dense", "ff": f}
            d["layers"].append({"type": "latent_attention" if s.latent else "attention", "mixer": mixer, "mlp": mlp})
        return d

    to_dict = to_hf_dict

    def tensor_names(self) -> List[str]:
        """Every tensor of a checkpoint, in the order of the layers."""
        names = ["embed"]
        glu = ("gate", "up", "down")
        for i, s in enumerate(self.layers):
            p, f = f"l{i}.", s.mlp
            names += [p + n for n in (("norm1", "norm1b") if f is None else ("norm1", "norm2", "norm1b", "norm2b"))]
            names += [p + "mix." + n for n in (("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "sink", "g", "o") if s.latent
                                               else ("q", "k", "v", "q.norm", "k.norm", "g", "o"))]
            if isinstance(f, MoeSpec):
                names += [p + f"mlp.e{e}.{n}" for e in range(f.experts) for n in glu]
                names += [p + "mlp.router", p + "mlp.correction"]
                names += [p + "mlp.shared." + n for n in glu] if f.shared_ff else []
            elif f is not None:
                names += [p + "mlp." + n for n in glu]
        return names + ["final.norm", "head"]

    # ------------------------------------------------------------------ sizes
    def _mixer_weights(self, s: LayerSpec) -> Tuple[int, int]:
        """Weights of the mixer's products, and of its vectors."""
        W, m = self.hidden_size, s.mixer
        out = m.heads * m.vdim
        if s.latent:
            return (W * (m.q_rank + m.kv_rank + m.rot_dim + 2 * out) + m.heads * (m.q_rank * (m.dim + m.rot_dim)
                    + m.kv_rank * (m.dim + m.vdim)), m.q_rank + m.kv_rank + m.heads)
        return W * (m.heads * m.dim + m.kv_heads * (m.dim + m.vdim) + m.heads + out), (m.heads + m.kv_heads) * m.dim

    def num_parameters(self, include_embeddings: bool = True) -> int:
        W = n = self.hidden_size
        for s in self.layers:
            f = s.mlp
            n += sum(self._mixer_weights(s)) + (2 if f is None else 4) * W
            if isinstance(f, MoeSpec):
                n += 3 * W * (f.experts * f.ff + f.shared_ff) + f.scores * (W + 1)
            elif f is not None:
                n += 3 * W * f
        return n + (2 * self.vocab_size * W if include_embeddings else 0)

    def flops_per_token(self, seq_len: int = 0, backward: bool = False) -> float:
        """Matmul FLOPs of one token (2 x the weights it meets, looped layers once per pass; of the chosen experts on average the
        share that is no identity) and attention over the keys it sees on average."""
        W, out = self.hidden_size, 2.0 * self.vocab_size * self.hidden_size
        for i, _ in self.layer_runs():
            s = self.layers[i]
            m, f = s.mixer, s.mlp
            out += 2.0 * self._mixer_weights(s)[0]
            keys = seq_len / 2.0 if s.latent or not m.window else min(seq_len / 2.0, m.window)
            out += 2.0 * m.heads * (m.dim + (m.rot_dim if s.latent else 0) + m.vdim) * keys
            if isinstance(f, MoeSpec):
                out += 2.0 * W * (3.0 * f.ff * f.top * f.experts / f.scores + 3.0 * f.shared_ff + f.scores)
            elif f is not None:
                out += 6.0 * W * f
        return out * (3.0 if backward else 1.0)


Placed = Optional[torch.Tensor]


class _AttentionMixer(nn.Module):
    def __init__(self, cfg: TitatarConfig, m: WindowAttnSpec, mk):
        super().__init__()
        self.m, self.eps = m, cfg.norm_eps
        self.in_cols, n_in = _columns({"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim, "g": m.heads})
        self.n_out = m.heads * m.vdim
        self.w_in, self.w_out = mk(n_in, cfg.hidden_size), mk(cfg.hidden_size, _pad8(self.n_out))
        self.q_norm, self.k_norm = mk(m.heads * m.dim), mk(m.kv_heads * m.dim)
        self.spec = serving.SoftmaxSpec(m.scale, window=m.window)
        self.register_buffer("sink", torch.zeros(m.heads, dtype=torch.float32, device=self.q_norm.device), persistent=False)

    def place(self, key: str) -> Placed:
        if key in self.in_cols:
            o, n = self.in_cols[key]
            return self.w_in.data.narrow(0, o, n)
        return {"o": self.w_out.data.narrow(1, 0, self.n_out), "q.norm": self.q_norm.data, "k.norm": self.k_norm.data}.get(key)

    def cache_layout(self) -> Dict[str, Any]:
        return {"kv": (self.m.kv_heads, self.m.dim, self.m.vdim)}

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y: torch.Tensor, cache, run: int, rope) -> None:
        m, c = self.m, self.in_cols
        p = serving.linear(h, self.w_in)
        kc, vc = cache.k[run], cache.v[run]
        serving.row_norm_rope_cache(b, p, (c["q"][0], c["k"][0], c["v"][0]), self.q_norm, self.k_norm, rope[m.rot], m.rot.dims, m.heads,
                                    kc, vc, self.eps)
        a = _activations(b.rows, self.n_out, h)
        serving.softmax_attention(b, p, m.heads, kc, vc, self.spec, None, a, sink=self.sink, gate=p[:, c["g"][0]:])
        serving.project(a, self.w_out, y)


class _LatentMixer(nn.Module):
    def __init__(self, cfg: TitatarConfig, m: LatentAttnSpec, mk):
        super().__init__()
        self.m, self.eps = m, cfg.norm_eps
        self.n_out = m.heads * m.vdim
        self.in_cols, n_in = _columns({"dq": m.q_rank, "dkv": m.kv_rank + m.rot_dim, "g": self.n_out})
        self.exp_cols, n_exp = _columns({"uk": m.heads * m.dim, "uv": self.n_out})
        self.w_in, self.w_out = mk(n_in, cfg.hidden_size), mk(cfg.hidden_size, _pad8(self.n_out))
        self.w_q = mk(m.heads * (m.dim + m.rot_dim), _pad8(m.q_rank))
        self.w_expand = mk(n_exp, _pad8(m.kv_rank))                      # keys and values of all heads from the latent
        self.q_norm, self.kv_norm, self.sink = mk(m.q_rank), mk(m.kv_rank), mk(m.heads)
        self.spec = serving.LatentSpec(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale)
        dev = self.sink.device
        # what serving derives from the weights: the key projection transposed per head, the sinks in fp32
        self.register_buffer("w_absorb", torch.zeros(m.heads * m.kv_rank, _pad8(m.dim), device=dev, dtype=self.sink.dtype), persistent=False)
        self.register_buffer("sink32", torch.zeros(m.heads, device=dev, dtype=torch.float32), persistent=False)

    def place(self, key: str) -> Placed:
        m = self.m
        if key in self.in_cols:
            o, n = self.in_cols[key]
            return self.w_in.data.narrow(0, o, n)
        if key in self.exp_cols:
            o, n = self.exp_cols[key]
            return self.w_expand.data.narrow(0, o, n).narrow(1, 0, m.kv_rank)
        return {"uq": self.w_q.data.narrow(1, 0, m.q_rank), "o": self.w_out.data.narrow(1, 0, self.n_out), "dq.norm": self.q_norm.data,
                "dkv.norm": self.kv_norm.data, "sink": self.sink.data}.get(key)

    def refresh(self, key: str) -> None:
        m = self.m
        if key == "uk":
            self.w_absorb.view(m.heads, m.kv_rank, -1)[:, :, :m.dim].copy_(self.place("uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2))
        elif key == "sink":
            self.sink32.copy_(self.sink.data)

    def cache_layout(self) -> Dict[str, Any]:
        return {"kv": (1, serving.shared_row(self.m.kv_rank + self.m.rot_dim, self.m.kv_rank, self.sink.dtype), 0)}

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y: torch.Tensor, cache, run: int, rope) -> None:
        m, c = self.m, self.in_cols
        p = serving.linear(h, self.w_in)
        latents = cache.k[run]
        serving.latent_norm_cache(b, p, c["dq"][0], c["dkv"][0], self.q_norm, self.kv_norm, rope[m.rot], latents, self.eps, m.rot_dim)
        q = serving.linear(p[:, c["dq"][0]:c["dq"][0] + m.q_rank], self.w_q[:, :m.q_rank])
        a = _activations(b.rows, self.n_out, h)
        serving.latent_attention(b, q, self.spec, latents, self.w_absorb, self.w_expand, self.sink32, p[:, c["g"][0]:], rope[m.rot], a)
        serving.project(a, self.w_out, y)


class _GatedLayer(nn.Module):
    """W_down (silu(W_gate h) * (W_up h))"""

    def __init__(self, cfg: TitatarConfig, ff: int, mk):
        super().__init__()
        self.ff = ff
        self.w_gu, self.w_down = mk(2 * ff, cfg.hidden_size), mk(cfg.hidden_size, _pad8(ff))

    def place(self, key: str) -> Placed:
        if key in ("gate", "up"):
            return self.w_gu.data[(0 if key == "gate" else 1)::2]
        return self.w_down.data.narrow(1, 0, self.ff) if key == "down" else None

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y: torch.Tensor, cache, run: int, rope) -> None:
        a = _activations(b.rows, self.ff, h)
        serving.gate_up_silu(h, self.w_gu, a[:, :self.ff])
        serving.project(a, self.w_down, y)


class _Mixture(nn.Module):
    """Routed, identity and shared experts.  Leaves the shared expert's output in ``y`` and returns the rest unsummed."""

    def __init__(self, cfg: TitatarConfig, s: MoeSpec, mk):
        super().__init__()
        W = cfg.hidden_size
        self.s = s
        self.router, self.correction = mk(_pad8(s.scores), W), mk(s.scores)
        self.w_gu, self.w_down = mk(s.experts * 2 * s.ff, W), mk(s.experts * W, _pad8(s.ff))
        self.shared = _GatedLayer(cfg, s.shared_ff, mk) if s.shared_ff else None
        self.register_buffer("counters", torch.zeros(s.experts + 1, dtype=torch.int32, device=self.router.device), persistent=False)

    def place(self, key: str) -> Placed:
        s = self.s
        head, _, leaf = key.partition(".")
        if key == "router":
            return self.router.data[:s.scores]
        if key == "correction":
            return self.correction.data
        if head == "shared" and self.shared is not None:
            return self.shared.place(leaf)
        if head[:1] == "e" and head[1:].isdigit() and int(head[1:]) < s.experts:
            e, W = int(head[1:]), self.w_gu.shape[1]
            if leaf in ("gate", "up"):
                return self.w_gu.data[2 * s.ff * e:2 * s.ff * (e + 1)][(0 if leaf == "gate" else 1)::2]
            if leaf == "down":
                return self.w_down.data[W * e:W * (e + 1), :s.ff]
        return None

    def serve(self, b: serving.StepBatch, h: torch.Tensor, y: torch.Tensor, cache, run: int, rope) -> serving.ExpertMix:
        s = self.s
        z = serving.linear(h, self.router, out_dtype=torch.float32)
        mix = serving.experts(b, h, z, self.correction, self.counters, self.w_gu, self.w_down, s.scores, s.experts, s.top, s.ff)
        if self.shared is not None:
            self.shared.serve(b, h, y, cache, run, rope)
        return mix


class TitatarBlock(nn.Module):
    """Weights of one layer in the fused layouts."""

    def __init__(self, cfg: TitatarConfig, spec: LayerSpec, mk):
        super().__init__()
        self.spec = spec
        W, f = cfg.hidden_size, spec.mlp
        self.norm1, self.norm1b = mk(W), mk(W)
        self.mixer = (_LatentMixer if spec.latent else _AttentionMixer)(cfg, spec.mixer, mk)
        self.norm2, self.norm2b = (mk(W), mk(W)) if f is not None else (None, None)
        self.mlp = None if f is None else _Mixture(cfg, f, mk) if isinstance(f, MoeSpec) else _GatedLayer(cfg, f, mk)

    def place(self, rest: str) -> Placed:
        head, _, key = rest.partition(".")
        if rest in ("norm1", "norm1b", "norm2", "norm2b"):
            w = getattr(self, rest)
            return None if w is None else w.data
        if head == "mix":
            return self.mixer.place(key)
        return self.mlp.place(key) if head == "mlp" and self.mlp is not None else None

    def sublayers(self):
        """``(norm ahead, body, norm behind)``"""
        yield self.norm1, self.mixer, self.norm1b
        if self.mlp is not None:
            yield self.norm2, self.mlp, self.norm2b


class TitatarLM(nn.Module):
    def __init__(self, cfg: TitatarConfig, device="cuda", dtype=torch.bfloat16):
        super().__init__()
        self.cfg = cfg
        mk = lambda *s: nn.Parameter(torch.zeros(*s, device=device, dtype=dtype), requires_grad=False)
        self.embed = mk(cfg.vocab_size, cfg.hidden_size)
        self.blocks = nn.ModuleList([TitatarBlock(cfg, s, mk) for s in cfg.layers])
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
    def _place(self, name: str) -> torch.Tensor:
        """Where the checkpoint tensor ``name`` lives inside the fused parameters."""
        top = {"embed": self.embed, "head": self.head, "final.norm": self.final_norm}
        if name in top:
            return top[name].data
        layer, _, rest = name.partition(".")
        found = None
        if layer[:1] == "l" and layer[1:].isdigit() and int(layer[1:]) < len(self.blocks):
            found = self.blocks[int(layer[1:])].place(rest)
        if found is None:
            raise KeyError(f"unexpected tensor name {name!r}")
        return found

    @torch.no_grad()
    def load_named_tensor(self, name: str, t: torch.Tensor) -> None:
        dst = self._place(name)
        if dst.shape != t.shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)} does not fit")
        dst.copy_(t.to(device=dst.device, dtype=dst.dtype))
        layer, _, rest = name.partition(".")
        if rest in ("mix.uk", "mix.sink"):
            self.blocks[int(layer[1:])].mixer.refresh(rest[4:])

    def iter_named_tensors(self) -> Iterator[Tuple[str, torch.Tensor]]:
        for name in self.cfg.tensor_names():
            yield name, self._place(name)

    @torch.no_grad()
    def init_weights(self, seed: int = 0, std: float = 0.02) -> "TitatarLM":
        """Deterministic random weights keyed by tensor name (gains neutral, sinks and corrections zero)."""
        from .decoder import hash_name
        for name, t in self.iter_named_tensors():
            leaf = name.split(".", 1)[-1]
            if leaf in ("mix.q.norm", "mix.k.norm", "mix.dq.norm", "mix.dkv.norm"):
                v = torch.ones(t.shape)
            elif leaf in ("norm", "norm1", "norm2", "norm1b", "norm2b", "mix.sink", "mlp.correction"):
                v = torch.zeros(t.shape)
            else:
                g = torch.Generator(device=t.device)
                g.manual_seed((hash_name(name) + seed) % (2 ** 31))
                v = torch.randn(t.shape, generator=g, dtype=torch.float32, device=t.device) * std
            self.load_named_tensor(name, v.to(self.dtype))
        return self

    # ------------------------------------------------------------------ serving protocol
    def cache_layout(self) -> List[Dict[str, Any]]:
        """What every layer run keeps per sequence: paged K/V ``(kv heads, key row, value row)``; a latent layer's row is the
        latent and the rotated key part, and it has no value row."""
        return [self.blocks[i].mixer.cache_layout() for i, _ in self.cfg.layer_runs()]

    def prepare_serving(self, max_positions: int) -> None:
        """Position tables (one per distinct rotation), computed in float64."""
        dev = self.embed.device
        if self._rope_len < max_positions or any(t[0].device != dev for t in self._rope.values()):
            self._rope = {}
            for s in self.cfg.layers:
                r = s.mixer.rot
                if r not in self._rope:
                    self._rope[r] = norm.rope_tables(max_positions, max(2, r.dims), r.base, dev, r.yarn if r.dims else None)
            self._rope_len = max_positions

    def serve_rows(self, b: serving.StepBatch, cache, on_layer=None) -> torch.Tensor:
        """Runs the layers over the batch, advancing the caches; returns the residual ``[rows, W]`` fp32.  ``on_layer(run, x)``
        sees it after every layer run."""
        cfg, dev = self.cfg, self.embed.device
        W, eps = cfg.hidden_size, cfg.norm_eps
        x = torch.empty((b.rows, W), device=dev, dtype=torch.float32)
        serving.embed(b, self.embed, None, None, cache.prev, x, scale=cfg.embed_scale)
        clear = serving.accumulates(b.rows, W, dev)            # products of few rows are added onto a zeroed y
        y = (torch.zeros if clear else torch.empty)((b.rows, W), device=dev, dtype=torch.float32)
        left: Dict[str, Any] = dict(y=None, post=None, mix=None)          # the last sublayer's output, not yet in x
        for run, (i, t) in enumerate(cfg.layer_runs()):
            again = (b.tokens, self.embed, cfg.embed_scale) if t else None
            for pre, body, post in self.blocks[i].sublayers():
                h = serving.residual_step(x, pre=pre, eps=eps, again=again, clear=clear, **left)
                again = None
                mix = body.serve(b, h, y, cache, run, self._rope)
                only_mix = mix is not None and body.shared is None
                left = dict(y=None if only_mix else y, post=post, mix=mix)
            if on_layer is not None:
                on_layer(run, serving.residual_step(x, pre=None, eps=eps, write=False, **left))
        serving.commit(b, cache.prev, cache.parity)
        return serving.residual_step(x, pre=None, eps=eps, write=False, **left)

    def output_rows(self, x: torch.Tensor, rows: Optional[torch.Tensor]) -> torch.Tensor:
        """Final norm of the chosen rows (None: all), in the activation type."""
        return serving.gain_norm_rows(x, rows, self.final_norm, self.cfg.norm_eps, 1.0)

    def logits(self, h: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        return serving.linear(h, self.head, out, out_dtype=torch.float32)


def _stack(n: int, latent: LatentAttnSpec, window: WindowAttnSpec, ff: int, moe: MoeSpec) -> Tuple[LayerSpec, ...]:
    """``n`` layers: the first dense, every third one windowed, the others latent."""
    return tuple(LayerSpec(window if i % 3 == 2 else latent, moe if i else ff) for i in range(n))


_YARN = norm.Yarn(4.0, 4096.0, 32.0, 1.0)

PRESETS: Dict[str, TitatarConfig] = {
    "titatar-tiny": TitatarConfig(320, 128, _stack(4, LatentAttnSpec(4, 32, 16, 32, 48, 64, 0.15, RotSpec(16, 10000.0, _YARN)),
                                                   WindowAttnSpec(4, 2, 32, 48, 0.18, 50, RotSpec(16, 10000.0)), 256,
                                                   MoeSpec(6, 2, 2, 64, 32)), 1e-5, 2.0, (1, 3, 2), "titatar-tiny"),
    # layers of the size of a 1.7B / 8B dense decoder's
    "titatar-2048": TitatarConfig(151936, 2048, _stack(8, LatentAttnSpec(16, 128, 64, 128, 768, 512, 192 ** -0.5, RotSpec(64, 10000.0, _YARN)),
                                                       WindowAttnSpec(16, 8, 128, 128, 128 ** -0.5, 1024, RotSpec(128, 10000.0)), 6144,
                                                       MoeSpec(64, 16, 6, 768, 1024)), 1e-6, 1.0, (2, 6, 2), "titatar-2048"),
    "titatar-4096": TitatarConfig(151936, 4096, _stack(8, LatentAttnSpec(32, 128, 64, 128, 1536, 512, 192 ** -0.5, RotSpec(64, 10000.0, _YARN)),
                                                       WindowAttnSpec(32, 8, 128, 128, 128 ** -0.5, 1024, RotSpec(128, 10000.0)), 12288,
                                                       MoeSpec(64, 16, 6, 1536, 2048)), 1e-6, 1.0, (2, 6, 2), "titatar-4096"),
}
