"""Tubevik in plain PyTorch on the CPU, float64, one function per mechanism, one token sequence at a time and nothing kept
between calls: what the engine's kernels, caches and state slots are compared with.

Notation: x is the residual stream [T, width]; positions count from 0; weights are stored [out, in]; w maps tensor names to
float64 tensors; p is a prefix of tensor names ("l3", "l3.mix").
"""

import math

import torch

F64 = torch.float64


def layer_norm(x, weight, bias, eps):
    """Mean taken off, over the root of the mean square of what is left, gain and bias."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * weight + bias


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def capped(z, cap):
    return cap * torch.tanh(z / cap)


# ------------------------------------------------------------------------------------------ rotation

def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims, base, s):
    """(frequencies, factor on cos and sin).  A pair that turns more than ``fast`` times within the original context keeps its
    frequency, one that turns fewer than ``slow`` times is slowed by ``factor``, those between go from one to the other."""
    def pair_that_turns(times):
        return dims * math.log(s["original"] / (2.0 * math.pi * times)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_that_turns(s["fast"])), 0)
    hi = min(math.ceil(pair_that_turns(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotation(rot):
    """(rotated entries, frequencies, factor) of a configuration's ``rot`` (None: no rotation)."""
    if not rot or not rot["dims"]:
        return 0, [], 1.0
    if rot.get("scaling"):
        f, factor = yarn_frequencies(rot["dims"], rot["base"], rot["scaling"])
        return rot["dims"], f, factor
    return rot["dims"], plain_frequencies(rot["dims"], rot["base"]), 1.0


def rotate(x, positions, turn, layout):
    """x [T, heads, dim]: the pairs of the first entries of each head turn by position * frequency; entry i is paired with
    entry i + dims/2 ("half") or entry 2i with entry 2i + 1 ("pairs"); the rest pass."""
    dims, freqs, factor = turn
    if not dims:
        return x
    a = (torch.as_tensor(positions, dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :]).to(x.dtype)
    c, s = (factor * torch.cos(a))[:, None, :], (factor * torch.sin(a))[:, None, :]
    out = x.clone()
    first, second = (slice(0, dims // 2), slice(dims // 2, dims)) if layout == "half" else (slice(0, dims, 2), slice(1, dims, 2))
    u, v = x[..., first], x[..., second]
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------------------ attention

def in_window(t, window):
    """The first position that position t sees (window 0: all)."""
    return max(0, t - window + 1) if window else 0


def in_chunk(t, chunk):
    return t // chunk * chunk if chunk else 0


def attention(q, k, v, scale, first_seen, cap=None, extra_one=False):
    """q [T, H, d], k [T, G, d], v [T, G, e], token t at position t.  One token and one head at a time.  ``cap``: scores pass
    cap tanh(./cap).  ``extra_one``: the softmax's denominator also holds a one, a score of zero that has no value."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        lo = first_seen(t)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:t + 1, g] @ q[t, h]) * scale
            if cap:
                s = capped(s, cap)
            top = max(float(s.max()), 0.0) if extra_one else float(s.max())
            e = torch.exp(s - top)
            out[t, h] = (e / (e.sum() + (math.exp(-top) if extra_one else 0.0))) @ v[lo:t + 1, g]
    return out


def window_keys_values(h, w, p, m, eps):
    """Keys (normed over the whole projection, then rotated) and values of a windowed attention layer."""
    T, G = h.shape[0], m["kv_heads"]
    k = unit_rms(h @ w[f"{p}.k"].T + w[f"{p}.k.b"], eps) * w[f"{p}.k.norm"]
    v = h @ w[f"{p}.v"].T + w[f"{p}.v.b"]
    return rotate(k.view(T, G, m["dim"]), range(T), rotation(m.get("rot")), "half"), v.view(T, G, m["vdim"])


def window_mixer(h, w, p, m, eps, lent=None):
    """Attention inside a sliding window with capped scores and a gate a head; ``lent``: another layer's keys and values.
    Returns (output, the keys and values it attends over)."""
    T, H = h.shape[0], m["heads"]
    q = unit_rms(h @ w[f"{p}.q"].T + w[f"{p}.q.b"], eps) * w[f"{p}.q.norm"]
    q = rotate(q.view(T, H, m["dim"]), range(T), rotation(m.get("rot")), "half")
    k, v = lent if lent is not None else window_keys_values(h, w, p, m, eps)
    window = (m.get("mask") or {}).get("size", 0)
    o = attention(q, k, v, m["scale"], lambda t: in_window(t, window), cap=m.get("softcap"))
    o = o * torch.sigmoid(h @ w[f"{p}.g"].T)[..., None]
    return o.reshape(T, H * m["vdim"]) @ w[f"{p}.o"].T, (k, v)


def chunk_mixer(h, w, p, m, eps):
    """The left half of a parallel mixer: q and k turned in neighbouring pairs and THEN normed a head, softmax within the chunk
    with one more in its denominator."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    turn = rotation(m.get("rot"))
    q = unit_rms(rotate((h @ w[f"{p}.q"].T).view(T, H, m["dim"]), range(T), turn, "pairs"), eps)
    k = unit_rms(rotate((h @ w[f"{p}.k"].T).view(T, G, m["dim"]), range(T), turn, "pairs"), eps)
    v = (h @ w[f"{p}.v"].T).view(T, G, m["vdim"])
    chunk = (m.get("mask") or {}).get("size", 0)
    o = attention(q, k, v, m["scale"], lambda t: in_chunk(t, chunk), extra_one=True)
    return o.reshape(T, H * m["vdim"]) @ w[f"{p}.o"].T


# ------------------------------------------------------------------------------------------ recurrence

def causal_conv_silu(u, taps_w):
    """u [T, C], taps_w [C, taps] (the last column meets the current token), zeros before the start, no bias."""
    T, C = u.shape
    taps = taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], 0)
    return silu(sum(padded[j:j + T] * taps_w[:, j] for j in range(taps)))


def delta_rule(q, k, v, beta, g):
    """q, k [T, G, d], v [T, H, e], beta [T, H], g [T, H, d].  Per head: the rows of S times the decays of their key entries;
    u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, e = v.shape
    G, d = q.shape[1], q.shape[2]
    out = torch.zeros(T, H, e, dtype=q.dtype)
    for h in range(H):
        kh = h // (H // G)
        S = torch.zeros(d, e, dtype=q.dtype)
        for t in range(T):
            S = g[t, h][:, None] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, kh])
            S = S + torch.outer(k[t, kh], u)
            out[t, h] = S.T @ q[t, kh]
    return out


def channel_decay(z, a_log, dt_bias, heads):
    """z [T, heads d]: exp(-exp(A_log of the head) softplus(z + dt_bias)), laid out [T, heads, d]."""
    rate = softplus(z + dt_bias).view(z.shape[0], heads, -1)
    return torch.exp(-torch.exp(a_log)[None, :, None] * rate)


def delta_mixer(h, w, p, m, eps):
    """The right half of a parallel mixer: the gated delta rule with a decay a key entry."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_conv_silu(h @ w[f"{p}.q"].T, w[f"{p}.q.conv"]).view(T, G, d)
    k = causal_conv_silu(h @ w[f"{p}.k"].T, w[f"{p}.k.conv"]).view(T, G, d)
    v = causal_conv_silu(h @ w[f"{p}.v"].T, w[f"{p}.v.conv"]).view(T, H, e)
    beta = torch.sigmoid(h @ w[f"{p}.b"].T)
    g = channel_decay((h @ w[f"{p}.a1"].T) @ w[f"{p}.a2"].T, w[f"{p}.A_log"], w[f"{p}.dt_bias"], H)
    o = delta_rule(unit_vector(q) * d ** -0.5, unit_vector(k), v, beta, g)
    o = (unit_rms(o, eps) * w[f"{p}.norm"]).reshape(T, H * e)
    return (o * torch.sigmoid((h @ w[f"{p}.g1"].T) @ w[f"{p}.g2"].T)) @ w[f"{p}.o"].T


def parallel_mixer(h, w, p, m, eps):
    return m["left_scale"] * chunk_mixer(h, w, f"{p}.left", m["left"], eps) \
        + m["right_scale"] * delta_mixer(h, w, f"{p}.right", m["right"], eps)


# ------------------------------------------------------------------------------------------ feed-forward, model

def clamped_ff(h, w, p, limit):
    g = torch.clamp(h @ w[f"{p}.gate"].T, max=limit)
    u = torch.clamp(h @ w[f"{p}.up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[f"{p}.down"].T


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence; with ``want_layers`` also the stream after every layer."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    norm = lambda x, name: layer_norm(x, w[name], w[f"{name}.b"], eps)
    x = norm(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], "embed.norm")
    streams, kept = [], {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}", L["mixer"]
        h = norm(x, f"{p}.norm1")
        if L["type"] == "attention":
            a, kept[i] = window_mixer(h, w, f"{p}.mix", m, eps, kept[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            a = parallel_mixer(h, w, f"{p}.mix", m, eps)
        if L.get("mlp") is not None:
            a = a + clamped_ff(h, w, f"{p}.mlp", L["mlp"]["limit"])
        x = x + mult * a
        streams.append(x)
    logits = norm(x, "final.norm") @ w["head"].T
    if cfg.get("logit_softcap"):
        logits = capped(logits, cfg["logit_softcap"])
    return (logits, streams) if want_layers else logits


def greedy(logits):
    return int(torch.argmax(logits))
