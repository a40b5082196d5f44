"""Plain, slow Meronex decoder: the oracle of the kernel and engine tests.

One function per mechanism, each written as the textbook expression over ONE whole sequence (recurrences token by token, no cache,
no chunks, no batching, experts one by one), in the dtype of its inputs -- the tests use float64 on the CPU.  It shares no code
with the package.  ``forward(cfg, tensors, tokens)`` takes the parsed config.json and the checkpoint's tensors by name and returns
``(logits [T, V], residual after every layer [layers, T, width])``.

``faults`` (a set of names) plants a deliberate mistake, so that a test can show that its inputs would reveal one:
norms ``one_group``, ``one_plus``; sublayers ``no_gate``, ``gate_without_bias``, ``gate_of_residual``, ``no_mult``; matrix memory
``no_input_cap``, ``no_forget_cap``, ``no_floor`` (the denominator without its lower bound), ``signed_denominator``, ``silu_out``
(silu in place of the sigmoid), ``unscaled_q``; delta rule ``read_before_write``, ``decay_after_write``, ``no_unit``,
``no_conv_state`` (the convolution starts anew every 5 tokens), ``reversed_taps``,
``spread_heads`` (query head h reads h mod kv_heads), ``no_dt_bias``; attention ``neighbour_pairs``, ``no_yarn``, ``no_yarn_gain``,
``no_softcap``, ``cap_before_scale``, ``raw_values``, ``values_rotated``; time mixing ``shift_two``, ``no_shift_state`` (no previous
token every 5 tokens), ``no_bonus``, ``read_after_write``, ``scalar_decay``, ``linear_rank`` (no tanh); side by side ``sum_of_sides``,
``sides_not_normed``; experts ``softmax_scores``, ``renormed``, ``weighted_output``, ``silu_glu``, ``no_limit``."""
from __future__ import annotations

import math

import torch

RECENT = 5          # tokens after which the faulty variants forget


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def group_norm(x, w, groups, eps, faults=()):
    groups = 1 if "one_group" in faults else groups
    parts = x.reshape(*x.shape[:-1], groups, -1)
    return rms(parts, eps).reshape(x.shape) * (1.0 + w if "one_plus" in faults else w)


# ------------------------------------------------------------------------------------------------ matrix memory
def memory_gates(zi, zf, cap, faults=()):
    """Log input and forget gates from their projections (biases included)."""
    soft = lambda z: cap * torch.tanh(z / cap)
    return (zi if "no_input_cap" in faults else soft(zi)), -softplus(-(zf if "no_forget_cap" in faults else soft(zf)))


def matrix_memory(q, k, v, log_i, log_f, faults=()):
    """``q, k [T, H, D]`` (q scaled), ``v [T, H, E]``, log gates ``[T, H]`` -> ``[T, H, E]``."""
    T, H, D = q.shape
    S, n = q.new_zeros(H, D, v.shape[2]), q.new_zeros(H, D)
    m = q.new_zeros(H)
    out = []
    for t in range(T):
        new = torch.maximum(log_f[t] + m, log_i[t])
        a, b = torch.exp(log_f[t] + m - new), torch.exp(log_i[t] - new)
        m = new
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        den = (n * q[t]).sum(-1)
        den = den if "signed_denominator" in faults else den.abs()
        den = den if "no_floor" in faults else torch.maximum(den, torch.exp(-m))
        out.append((S * q[t][:, :, None]).sum(1) / (den + 1e-6)[:, None])
    return torch.stack(out)


def mlstm(m, W, h, eps, faults=()):
    H, D, E, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = (h @ W["q"].T).reshape(T, H, D) * (1.0 if "unscaled_q" in faults else D ** -0.5)
    k, v = (h @ W["k"].T).reshape(T, H, D), (h @ W["v"].T).reshape(T, H, E)
    log_i, log_f = memory_gates(h @ W["i"].T + W["i.b"], h @ W["f"].T + W["f.b"], m["gate_cap"], faults)
    o = rms(matrix_memory(q, k, v, log_i, log_f, faults), eps).reshape(T, H * E) * W["norm"]
    g = h @ W["g"].T
    return (o * (silu(g) if "silu_out" in faults else sigmoid(g))) @ W["o"].T


# ------------------------------------------------------------------------------------------------ gated delta rule
def short_conv(x, w, faults=()):
    """Causal convolution per channel, ``w [channels, taps]``, last column the current token's; then silu."""
    T, taps = x.shape[0], w.shape[1]
    w = w.flip(1) if "reversed_taps" in faults else w
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s < 0 or ("no_conv_state" in faults and s < t - t % RECENT):
                continue
            y[t] = y[t] + w[:, j] * x[s]
    return silu(y)


def delta_rule(q, k, v, beta, g, faults=()):
    """``q, k [T, H, D]`` (unit vectors, q scaled), ``v [T, H, E]``, ``beta, g [T, H]`` -> ``[T, H, E]``."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        late = "decay_after_write" in faults
        S = S if late else g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        before = (S * q[t][:, :, None]).sum(1)
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(before if "read_before_write" in faults else (S * q[t][:, :, None]).sum(1))
        S = g[t][:, None, None] * S if late else S
    return torch.stack(out)


def delta(m, W, h, eps, faults=()):
    H, G, D, E, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (short_conv(h @ W[n].T, W[n + ".conv"], faults) for n in "qkv")
    of = torch.arange(H) % G if "spread_heads" in faults else torch.arange(H) // (H // G)
    unit = (lambda x: x) if "no_unit" in faults else (lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6))
    q = unit(q.reshape(T, G, D))[:, of] * D ** -0.5
    k = unit(k.reshape(T, G, D))[:, of]
    beta = sigmoid(h @ W["b"].T)
    a = h @ W["a"].T + (0.0 if "no_dt_bias" in faults else W["dt_bias"])
    g = torch.exp(-torch.exp(W["A_log"]) * softplus(a))
    o = rms(delta_rule(q, k, v.reshape(T, H, E), beta, g, faults), eps) * W["norm"]
    return (o.reshape(T, H * E) * silu(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ attention
def yarn_frequencies(rot, faults=()):
    """Angle per position of every pair, and the factor on cos and sin."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    if not sc or "no_yarn" in faults:
        return f, 1.0
    turns = lambda t: dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(turns(sc["fast"])), 0), min(math.ceil(turns(sc["slow"])), dims - 1)
    ramp = torch.tensor([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)], dtype=torch.float64)
    gain = 1.0 if "no_yarn_gain" in faults else 0.1 * math.log(sc["factor"]) + 1.0
    return f / sc["factor"] * ramp + f * (1.0 - ramp), gain


def rotate(x, rot, faults=()):
    """``x [T, heads, >= dims]``: the first ``dims`` dimensions turned by the position's angles, pairs (i, i + dims / 2)."""
    n = rot["dims"]
    if n == 0:
        return x
    f, gain = yarn_frequencies(rot, faults)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * f[None, :]
    c, s = (a.cos() * gain).to(x.dtype)[:, None], (a.sin() * gain).to(x.dtype)[:, None]
    if "neighbour_pairs" in faults:
        u, v = x[..., 0:n:2], x[..., 1:n:2]
        turned = torch.stack([u * c - v * s, v * c + u * s], -1).reshape(*x.shape[:-1], n)
    else:
        u, v = x[..., :n // 2], x[..., n // 2:n]
        turned = torch.cat([u * c - v * s, v * c + u * s], -1)
    return torch.cat([turned, x[..., n:]], -1)


def capped_attention(q, k, v, scale, cap, faults=()):
    """Causal softmax attention, ``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]`` -> ``[T, H * E]``."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        kv = h // (H // G)
        s = q[:, h] @ k[:, kv].T
        if cap and "no_softcap" not in faults:
            s = cap * torch.tanh(s / cap) * scale if "cap_before_scale" in faults else cap * torch.tanh(s * scale / cap)
        else:
            s = s * scale
        s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, kv])
    return torch.stack(out, 1).reshape(T, -1)


def attention(m, W, h, eps, faults=()):
    H, G, T = m["heads"], m["kv_heads"], h.shape[0]
    q = rotate((h @ W["q"].T).reshape(T, H, m["dim"]), m["rot"], faults)
    k = rotate((h @ W["k"].T).reshape(T, G, m["dim"]), m["rot"], faults)
    v = (h @ W["v"].T).reshape(T, G, m["vdim"])
    v = v if "raw_values" in faults else rms(v, eps)
    v = rotate(v, m["rot"], faults) if "values_rotated" in faults and m["vdim"] >= m["rot"]["dims"] else v
    return capped_attention(q, k, v, m["scale"], m.get("softcap"), faults) @ W["o"].T


# ------------------------------------------------------------------------------------------------ time mixing
def token_shift(h, mu, faults=()):
    """h + (previous token's h - h) * mu."""
    before = torch.zeros_like(h)
    by = 2 if "shift_two" in faults else 1
    before[by:] = h[:-by] if h.shape[0] > by else h[:0]
    if "no_shift_state" in faults:
        before[::RECENT] = 0
    return h + (before - h) * mu


def channel_decay_recurrence(r, k, v, w, u, faults=()):
    """``r, k, w [T, H, D]``, ``v [T, H, E]``, bonus ``u [H, D]`` -> ``[T, H, E]``."""
    S = r.new_zeros(r.shape[1], r.shape[2], v.shape[2])
    w = w.mean(-1, keepdim=True).expand_as(w) if "scalar_decay" in faults else w
    u = torch.zeros_like(u) if "no_bonus" in faults else u
    out = []
    for t in range(r.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        new = w[t][:, :, None] * S + kv
        seen = new if "read_after_write" in faults else S + u[:, :, None] * kv
        out.append((seen * r[t][:, :, None]).sum(1))
        S = new
    return torch.stack(out)


def time_mixing(m, W, h, eps, faults=()):
    H, D, T = m["heads"], m["dim"], h.shape[0]
    mix = {s: token_shift(h, W["mu." + s], faults) for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[s].T).reshape(T, H, D) for s in "rkv")
    low = mix["w"] @ W["w1"].T
    z = (low if "linear_rank" in faults else torch.tanh(low)) @ W["w2"].T + W["w0"]
    o = channel_decay_recurrence(r, k, v, torch.exp(-torch.exp(z)).reshape(T, H, D), W["u"].reshape(H, D), faults)
    return (rms(o, eps).reshape(T, H * D) * W["norm"] * silu(mix["g"] @ W["g"].T)) @ W["o"].T


def parallel(m, W, h, eps, faults=()):
    sides = []
    for name, f in (("left", attention), ("right", time_mixing)):
        sub = {k[len(name) + 1:]: v for k, v in W.items() if k.startswith(name + ".")}
        y = f(m[name], sub, h, eps, faults)
        sides.append(y * sub["out"] if "sides_not_normed" in faults else rms(y, eps) * sub["out"])
    return (sides[0] + sides[1]) * (1.0 if "sum_of_sides" in faults else 0.5)


# ------------------------------------------------------------------------------------------------ experts
def clamped_glu(h, gate, up, down, limit, faults=()):
    g, u = h @ gate.T, h @ up.T
    if "no_limit" not in faults:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    y = silu(g) * u if "silu_glu" in faults else g * sigmoid(1.702 * g) * (u + 1.0)
    return y @ down.T


def mixture(m, W, h, faults=()):
    top, limit = m["router"]["top"], m["expert"]["limit"]
    z = h @ W["router"].T
    s = torch.softmax(z, -1) if "softmax_scores" in faults else sigmoid(z)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = sorted(range(s.shape[1]), key=lambda e: -float(s[t, e]))[:top]
        total = sum(s[t, e] for e in chosen) if "renormed" in faults else 1.0
        for e in chosen:
            w = s[t, e] / total
            glu = lambda x: clamped_glu(x, *(W[f"e{e}.{n}"] for n in ("gate", "up", "down")), limit, faults)
            out[t] = out[t] + (w * glu(h[t]) if "weighted_output" in faults else glu(w * h[t]))
    return out


# ------------------------------------------------------------------------------------------------ the decoder
MIXERS = {"mlstm": mlstm, "delta": delta, "parallel": parallel}


def forward(cfg, tensors, tokens, dtype=torch.float64, faults=()):
    W = {k: v.to(dtype) for k, v in tensors.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    mult = 1.0 if "no_mult" in faults else cfg["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    after = []
    for i, e in enumerate(cfg["layers"]):
        sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}

        def add(x, n, f):
            h = group_norm(x, W[f"l{i}.norm{n}"], groups, eps, faults)
            src = x if "gate_of_residual" in faults else h
            z = src @ W[f"l{i}.rg{n}"].T + (0.0 if "gate_without_bias" in faults else W[f"l{i}.rg{n}.b"])
            return x + mult * f(h) * (1.0 if "no_gate" in faults else sigmoid(z))

        x = add(x, 1, lambda h: MIXERS[e["type"]](e["mixer"], sub(f"l{i}.mix."), h, eps, faults))
        if e.get("mlp"):
            x = add(x, 2, lambda h: mixture(e["mlp"], sub(f"l{i}.mlp."), h, faults))
        after.append(x)
    return group_norm(x, W["final.norm"], groups, eps, faults) @ W["head"].T, torch.stack(after) if after else x[None][:0]


def generate(cfg, tensors, prompt, n):
    """Greedy continuation of ``prompt`` by ``n`` tokens."""
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(forward(cfg, tensors, seq)[0][-1].argmax()))
    return seq[len(prompt):]
