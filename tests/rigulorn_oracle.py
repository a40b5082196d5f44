"""Plain, slow Rigulorn decoder: the oracle of the kernel and engine tests.

One function per mechanism, each written as the textbook expression over ONE whole sequence (no cache, no state
hand-over, no blocks, no batching), in the dtype of its inputs -- the tests use float64 on the CPU.  It shares no code
with the package.  ``forward(cfg, tensors, tokens)`` takes the parsed config.json and the checkpoint's tensors by name
and returns ``(logits [T, V], sum of the residual streams after every layer [layers, T, width])``.

``faults`` (a set of names) plants a deliberate mistake, so that a test can show that its inputs would reveal one:
``chunk_early`` / ``chunk_late`` (chunks one token shorter / longer), ``no_chunks``, ``chunks_from:<n>`` (chunks counted
from position n), ``no_softcap``, ``one_map`` (the second attention map is dropped), ``no_diff_scale``, ``half_rotation``
(pairs (i, i + dims/2)), ``own_keys`` (a layer that borrows keys reads the first layer's), ``conv_shift``,
``state_reset:<n>`` (the recurrent state is lost before position n), ``late_gate`` (the gate after the norm), ``one_norm``
(one group), ``no_limit``, ``mix_transposed``, ``in_order_mix`` (a stream is mixed from the ones already replaced)."""
from __future__ import annotations

import torch


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def rotate_pairs(x, positions, dims, base, faults=()):
    """Rotary embedding of ``x [T, H, D]``: dimension 2i pairs with 2i + 1 for the first ``dims``, the rest is untouched."""
    y = x.clone()
    half = dims // 2
    for i in range(half):
        a = positions.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        m, n = (i, i + half) if "half_rotation" in faults else (2 * i, 2 * i + 1)
        y[..., m] = x[..., m] * c - x[..., n] * s
        y[..., n] = x[..., n] * c + x[..., m] * s
    return y


def chunk_visible(T, size, faults=()):
    """``[T, T]`` bool: key j of query i, same chunk of ``size`` positions and not later (size 0: plain causal)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    seen = j <= i
    size = size - ("chunk_early" in faults) + ("chunk_late" in faults)
    shift = sum(int(f.split(":")[1]) for f in faults if f.startswith("chunks_from:"))
    if size and "no_chunks" not in faults:
        seen = seen & ((i - shift).div(size, rounding_mode="floor") == (j - shift).div(size, rounding_mode="floor"))
    return seen


def softcapped_attention(q, k, v, scale, softcap, seen, faults=()):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, E]``: softmax over the visible keys of cap * tanh(scale q.k / cap)."""
    rep = q.shape[1] // k.shape[1]
    out = []
    for h in range(q.shape[1]):
        s = q[:, h] @ k[:, h // rep].t() * scale
        if softcap and "no_softcap" not in faults:
            s = softcap * torch.tanh(s / softcap)
        s = torch.where(seen, s, torch.full_like(s, float("-inf")))
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append((p / p.sum(-1, keepdim=True)) @ v[:, h // rep])
    return torch.stack(out, 1)


def map_weight(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def two_map_attention(q, k, v, lam, diff, scale, softcap, seen, eps, faults=()):
    """``q [T, H, 2, D]``, ``k [T, G, 2, D]``, ``v [T, G, E]``: first map minus ``lam`` times the second, normalised per
    head and scaled by ``1 - diff``."""
    a1 = softcapped_attention(q[:, :, 0], k[:, :, 0], v, scale, softcap, seen, faults)
    a2 = softcapped_attention(q[:, :, 1], k[:, :, 1], v, scale, softcap, seen, faults)
    o = rms(a1 if "one_map" in faults else a1 - lam * a2, eps)
    return o if "no_diff_scale" in faults else o * (1.0 - diff)


def causal_conv(x, w, b, faults=()):
    """Depth-wise: out[t] = b + sum_j w[:, j] * x[t - taps + 1 + j], zeros before the first row."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x) + b
    for j in range(taps):
        back = taps - 1 - j + (1 if "conv_shift" in faults and j < taps - 1 else 0)
        if back < T:
            out[back:] += x[:T - back] * w[:, j]
    return out


def state_space(x, B, C, dt, A_log, D, faults=()):
    """``x [T, H, E]``, ``B, C [T, G, N]``, ``dt [T, H]`` (after the softplus): token by token from S = 0."""
    T, H, E = x.shape
    G, N = B.shape[1:]
    rep = H // G
    S = torch.zeros(H, N, E, dtype=x.dtype)
    out = torch.zeros_like(x)
    for t in range(T):
        if f"state_reset:{t}" in faults:
            S = torch.zeros_like(S)
        for h in range(H):
            decay = torch.exp(-torch.exp(A_log[h]) * dt[t, h])
            S[h] = decay * S[h] + dt[t, h] * torch.outer(B[t, h // rep], x[t, h])
            out[t, h] = S[h].t() @ C[t, h // rep] + D[h] * x[t, h]
    return out


def gated_group_norm(y, z, w, groups, eps, faults=()):
    """The gate first, then every one of ``groups`` equal parts by its own root mean square, then the weight."""
    T, n = y.shape
    parts = 1 if "one_norm" in faults else groups
    if "late_gate" in faults:
        return rms(y.view(T, parts, -1), eps).reshape(T, n) * w * silu(z)
    return rms((y * silu(z)).view(T, parts, -1), eps).reshape(T, n) * w


def clamped_glu(g, u, limit, faults=()):
    if "no_limit" not in faults:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, min=-limit, max=limit)
    return g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)


# ---------------------------------------------------------------------------- layers
def attention_keys(m, W, p, h):
    T = h.shape[0]
    k = (h @ W[p + "k"].t()).view(T, 2 * m["kv_heads"], m["dim"])
    k = rotate_pairs(k, torch.arange(T), m["rot"]["dims"], m["rot"]["base"])
    return k.view(T, m["kv_heads"], 2, m["dim"]), (h @ W[p + "v"].t()).view(T, m["kv_heads"], m["vdim"])


def attention_mixer(m, W, p, h, kv, eps, faults=()):
    T = h.shape[0]
    q = (h @ W[p + "q"].t()).view(T, 2 * m["heads"], m["dim"])
    q = rotate_pairs(q, torch.arange(T), m["rot"]["dims"], m["rot"]["base"], faults).view(T, m["heads"], 2, m["dim"])
    lam = map_weight(*(W[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    seen = chunk_visible(T, m["mask"]["size"], faults)
    o = two_map_attention(q, *kv, lam, m["diff"], m["scale"], m["softcap"], seen, eps, faults)
    return o.reshape(T, -1) @ W[p + "o"].t()


def mamba_mixer(m, W, p, h, eps, faults=()):
    T = h.shape[0]
    H, E, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    z, xbc, dt = torch.split(h @ W[p + "in"].t(), [H * E, H * E + 2 * G * N, H], -1)
    xbc = silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"], faults))
    x, B, C = torch.split(xbc, [H * E, G * N, G * N], -1)
    y = state_space(x.reshape(T, H, E), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + W[p + "dt_bias"]),
                    W[p + "A_log"], W[p + "D"], faults)
    return gated_group_norm(y.reshape(T, -1), z, W[p + "norm"], m["norm_groups"], eps, faults) @ W[p + "o"].t()


def feed_forward(m, W, p, h, faults=()):
    return clamped_glu(h @ W[p + "gate"].t(), h @ W[p + "up"].t(), m["limit"], faults) @ W[p + "down"].t()


def streams_in(x, w_in):
    """``x [s, T, W]``: the sublayer's input."""
    return torch.einsum("s,stw->tw", w_in, x)


def streams_out(x, y, mix, w_out, faults=()):
    """``mix [from, to]``; every stream is replaced from the old ones."""
    new = []
    src = list(x)
    for t in range(len(x)):
        col = mix[t] if "mix_transposed" in faults else mix[:, t]
        new.append(sum(col[s] * src[s] for s in range(len(x))) + w_out[t] * y)
        if "in_order_mix" in faults:
            src[t] = new[-1]
    return torch.stack(new)


@torch.no_grad()
def forward(cfg, tensors, tokens, dtype=torch.float64, faults=()):
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x0 = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x = torch.stack([x0] * cfg["streams"])
    held, after = {}, []
    for i, s in enumerate(cfg["layers"]):
        p, m = f"l{i}.", s["mixer"]
        h = rms(streams_in(x, W[p + "hc1.in"]), eps) * W[p + "norm1"]
        if s["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                held[i] = attention_keys(m, W, p + "mix.", h)
                src = i
            elif "own_keys" in faults:
                src = min(held)
            y = attention_mixer(m, W, p + "mix.", h, held[src], eps, faults)
        else:
            y = mamba_mixer(m, W, p + "mix.", h, eps, faults)
        x = streams_out(x, y, W[p + "hc1.mix"], W[p + "hc1.out"], faults)
        if s.get("mlp") is not None:
            h = rms(streams_in(x, W[p + "hc2.in"]), eps) * W[p + "norm2"]
            x = streams_out(x, feed_forward(s["mlp"], W, p + "mlp.", h, faults), W[p + "hc2.mix"], W[p + "hc2.out"], faults)
        after.append(x.sum(0))
    return (rms(x.sum(0), eps) * W["final.norm"]) @ W["head"].t(), torch.stack(after)
