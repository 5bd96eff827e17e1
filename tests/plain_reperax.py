"""Reperax in plain PyTorch on the CPU, float64, one function per mechanism, one token sequence at a time and nothing kept
between calls: what the engine's kernels, caches and state slots are compared with.

Notation: x is the residual stream [T, width]; positions count from 0; weights are stored [out, in]; w maps tensor names to
float64 tensors; p is a prefix of tensor names ("l3", "l3.mix").
"""

import math

import torch

F64 = torch.float64


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_plus(x, weight, eps):
    """The layer norms and the last norm: the file holds gain - 1."""
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z * torch.sigmoid(z)


def token_shift(h, mix):
    """h_t + (h_(t-1) - h_t) * mix, entry by entry; the first token's predecessor is zero."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)
    return h + (before - h) * mix


# ------------------------------------------------------------------------------------------ attention

def visible_keys(t, chunk):
    """Positions that position t sees: those of its own chunk of the sequence, up to itself (chunk 0: all up to itself)."""
    return range(t - t % chunk if chunk else 0, t + 1)


def chunked_attention(q, k, v, scale, chunk):
    """q [T, H, d], k [T, G, d], v [T, G, e], token t at position t.  One token and one head at a time."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        seen = visible_keys(t, chunk)
        lo = seen[0]
        for h in range(H):
            g = h // (H // G)
            out[t, h] = torch.softmax((k[lo:t + 1, g] @ q[t, h]) * scale, 0) @ v[lo:t + 1, g]
    return out


def attention_mixer(h, w, p, m, eps):
    """The left half of a parallel mixer: q and k normed over the whole projection, no rotation, softmax within the chunk."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (unit_rms(h @ w[f"{p}.q"].T, eps) * w[f"{p}.q.norm"]).view(T, H, d)
    k = (unit_rms(h @ w[f"{p}.k"].T, eps) * w[f"{p}.k.norm"]).view(T, G, d)
    v = (h @ w[f"{p}.v"].T).view(T, G, e)
    chunk = (m.get("mask") or {}).get("size", 0)
    return chunked_attention(q, k, v, m["scale"], chunk).reshape(T, H * e) @ w[f"{p}.o"].T


# ------------------------------------------------------------------------------------------ recurrences

def linear_recurrence(q, k, v, alpha):
    """q, k [T, H, d], v [T, H, e], alpha [T, H, d].  Per head: S <- diag(alpha_t) S + k_t v_t^T;  o_t = S^T q_t."""
    T, H, e = v.shape
    out = torch.zeros(T, H, e, dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(q.shape[2], e, dtype=q.dtype)
        for t in range(T):
            S = alpha[t, h][:, None] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def channel_decay(h, w, p, tau):
    """A decay per key channel: sigmoid(z)^(1 / tau) with z = W_a2 (W_a1 h) + b."""
    z = (h @ w[f"{p}.a1"].T) @ w[f"{p}.a2"].T + w[f"{p}.a2.b"]
    return torch.sigmoid(z) ** (1.0 / tau)


def gla_mixer(h, w, p, m, eps):
    """The right half of a parallel mixer: gated linear attention."""
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[f"{p}.q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[f"{p}.k"].T).view(T, H, d)
    v = (h @ w[f"{p}.v"].T).view(T, H, e)
    o = linear_recurrence(q, k, v, channel_decay(h, w, p, m["tau"]).view(T, H, d))
    o = (unit_rms(o, eps) * w[f"{p}.norm"]).reshape(T, H * e)
    return (o * silu(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


def parallel_mixer(h, w, p, m, eps):
    return m["left_scale"] * attention_mixer(h, w, f"{p}.left", m["left"], eps) \
        + m["right_scale"] * gla_mixer(h, w, f"{p}.right", m["right"], eps)


def rotate_half(x, positions, dims, base):
    """x [T, heads, dim]: the first ``dims`` entries of each head turn by position * base^(-2i/dims), entry i
    paired with entry i + dims/2; the rest pass."""
    if not dims:
        return x
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    a = (torch.as_tensor(positions, dtype=F64)[:, None] * f[None, :]).to(x.dtype)
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def retention_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {}
    turn = lambda z: rotate_half(z, list(range(T)), rot.get("dims", 0), rot.get("base", 1.0))
    q = turn((h @ w[f"{p}.q"].T).view(T, H, d))
    k = turn((h @ w[f"{p}.k"].T).view(T, H, d)) * d ** -0.5
    v = (h @ w[f"{p}.v"].T).view(T, H, e)
    alpha = torch.tensor(m["decay"], dtype=q.dtype)[None, :, None].expand(T, H, d)
    o = unit_rms(linear_recurrence(q, k, v, alpha), eps).reshape(T, H * e)
    return (o * silu(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


# ------------------------------------------------------------------------------------------ feed-forward, model

def poly_norm(u, abce, eps):
    """a N(u) + b N(u^2) + c N(u^3) + e, N dividing a token's vector by its root mean square."""
    a, b, c, e = (abce[i] for i in range(4))
    return a * unit_rms(u, eps) + b * unit_rms(u ** 2, eps) + c * unit_rms(u ** 3, eps) + e


def dense_ff(h, w, p, eps):
    return poly_norm(h @ w[f"{p}.up"].T, w[f"{p}.act"], eps) @ w[f"{p}.down"].T


MIXERS = {"parallel": parallel_mixer, "retention": retention_mixer}


def layer(x, w, p, L, eps):
    """Both sublayers read the same x, each through a norm of its own, and each result is multiplied by a gate of its normed
    input; the mixer alone reads that input shifted by a token."""
    h = norm_one_plus(x, w[f"{p}.norm1"], eps)
    a = MIXERS[L["type"]](token_shift(h, w[f"{p}.shift"]), w, f"{p}.mix", L["mixer"], eps)
    out = a * torch.sigmoid(h @ w[f"{p}.rg1"].T + w[f"{p}.rg1.b"])
    if L.get("mlp") is not None:
        h2 = norm_one_plus(x, w[f"{p}.norm2"], eps)
        out = out + dense_ff(h2, w, f"{p}.mlp", eps) * torch.sigmoid(h2 @ w[f"{p}.rg2"].T + w[f"{p}.rg2.b"])
    return x + out


def runs(cfg):
    """(layer, pass that begins ahead of it or None) in the order layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(loop["times"]) for i in range(a, b)] \
        + [(i, None) for i in range(b, n)]


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one sequence; with ``want_layers`` also the stream after every layer run."""
    w = {k: v.to(F64) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    embedded = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x, streams = embedded, []
    for i, t in runs(cfg):
        if t is not None:
            x = x + (embedded if t > 0 else 0.0) + w["loop.step"][t]
        x = layer(x, w, f"l{i}", cfg["layers"][i], eps)
        streams.append(x)
    logits = norm_one_plus(x, w["final.norm"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, streams) if want_layers else logits


def greedy(logits):
    return int(torch.argmax(logits))
