"""Plain, slow Reninex decoder: the oracle of the kernel and engine tests.

One function per mechanism, each written as the textbook expression over ONE whole sequence (no cache, no state
hand-over, no chunks, no batching), in the dtype of its inputs -- the tests use float64 on the CPU.  It shares no code
with the package.  ``forward(cfg, tensors, tokens)`` takes the parsed config.json and the checkpoint's tensors by name
and returns ``(logits [T, V], residual stream after every layer run [runs, T, width])``.

``faults`` (a set of names) plants a deliberate mistake, so that a test can show that its inputs would reveal one:
``no_bigram_start``, ``conv_shift``, ``window:<n>`` (keys more than n-1 back are dropped), ``state_reset:<n>`` (the
recurrent state is lost before position n), ``no_bias``."""
from __future__ import annotations

import math

import torch


def embedding(embed, tokens, bigram=None, spec=None, faults=()):
    """Token rows plus, when the model has one, the hashed row of (previous token, token)."""
    x = embed[tokens].clone()
    if bigram is not None:
        b = int(spec["buckets"])
        rows = []
        for t, tok in enumerate(tokens.tolist()):
            if t == 0 and "no_bigram_start" not in faults:
                rows.append(b)
            else:
                prev = int(tokens[t - 1]) if t else 0
                rows.append((prev * int(spec["mul_prev"]) + tok * int(spec["mul_cur"])) % b)
        x = x + bigram[torch.tensor(rows)]
    return x


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_conv(h, w, faults=()):
    """Depth-wise convolution: out[t] = sum_j w[:, j] * h[t - taps + 1 + j], zeros before the first row."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for j in range(taps):
        back = taps - 1 - j
        if "conv_shift" in faults and back:
            back += 1
        if back < T:
            out[back:] += h[:T - back] * w[:, j]
    return out


def rotate(x, positions, dims, base):
    """Rotary embedding of ``x [T, H, D]``: dimension i pairs with i + dims/2, the rest is untouched."""
    half = dims // 2
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * freq[None]
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def sigmoid_attention(q, k, v, bias, scale, faults=()):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]``: every key j <= i enters with weight
    sigmoid(scale * q_i . k_j + bias_h); the weights are not normalised."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    seen = j <= i
    for f in faults:
        if f.startswith("window:"):
            seen = seen & (i - j < int(f.split(":")[1]))
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].t() * scale + (0.0 if "no_bias" in faults else bias[h])
        p = torch.where(seen, 1.0 / (1.0 + torch.exp(-s)), torch.zeros_like(s))
        out.append(p @ v[:, h // rep])
    return torch.stack(out, 1)


def retention(q, k, v, decay, faults=()):
    """``q, k [T, H, D]``, ``v [T, H, E]``: S <- decay_h S + k v^T, o = S^T q, token by token from S = 0."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    d = torch.tensor(list(decay), dtype=torch.float64).to(q.dtype)[:, None, None]
    out = []
    for t in range(T):
        if f"state_reset:{t}" in faults:
            S = torch.zeros_like(S)
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + torch.exp(-z))


def left_mixer(m, W, p, h, eps, faults=()):
    T = h.shape[0]
    H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ W[p + "q"].t()).view(T, H, D), eps)
    k = rms((h @ W[p + "k"].t()).view(T, G, D), eps)
    v = (h @ W[p + "v"].t()).view(T, G, E)
    o = sigmoid_attention(q, k, v, W[p + "pb"], m["scale"], faults)
    return o.reshape(T, H * E) @ W[p + "o"].t()


def right_mixer(m, W, p, h, eps, faults=()):
    T = h.shape[0]
    H, D, E = m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rotate((h @ W[p + "q"].t()).view(T, H, D), pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotate((h @ W[p + "k"].t()).view(T, H, D), pos, m["rot"]["dims"], m["rot"]["base"]) * D ** -0.5
    v = (h @ W[p + "v"].t()).view(T, H, E)
    o = rms(retention(q, k, v, m["decay"], faults), eps).reshape(T, H * E)
    return (o * silu(h @ W[p + "g"].t())) @ W[p + "o"].t()


def feed_forward(W, p, h):
    return (gelu_tanh(h @ W[p + "gate"].t()) * (h @ W[p + "up"].t())) @ W[p + "down"].t()


def layer(cfg, spec, W, p, x, faults=()):
    """Parallel layer: both sublayers read the same norm, each through its own input convolution."""
    eps = cfg["norm"]["eps"]
    h = rms(x, eps) * W[p + "norm1"]

    def conv_in(name):
        return h + causal_conv(h, W[p + name], faults) if cfg.get("canon") else h

    mx = spec["mixer"]
    h1 = conv_in("canon1")
    y = mx["left_scale"] * left_mixer(mx["left"], W, p + "mix.left.", h1, eps, faults) \
        + mx["right_scale"] * right_mixer(mx["right"], W, p + "mix.right.", h1, eps, faults)
    if spec.get("mlp") is not None:
        y = y + feed_forward(W, p + "mlp.", conv_in("canon2"))
    return x + y


def layer_order(cfg):
    """``(layer, pass or None)`` in the order of execution; the pass number is set on a pass's first layer."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n)]


@torch.no_grad()
def forward(cfg, tensors, tokens, dtype=torch.float64, faults=()):
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    tokens = torch.as_tensor(tokens)
    bg = (cfg.get("embedding") or {}).get("bigram")
    x0 = embedding(W["embed"], tokens, W.get("bigram") if bg else None, bg, faults)
    x, runs = x0, []
    for i, t in layer_order(cfg):
        if t is not None:
            x = torch.cat([x, x0], -1) @ W["loop.in"].t() + W["loop.step"][t]
        x = layer(cfg, cfg["layers"][i], W, f"l{i}.", x, faults)
        runs.append(x)
    h = rms(x, cfg["norm"]["eps"]) * W["final.norm"]
    return h @ W["head"].t(), torch.stack(runs)
