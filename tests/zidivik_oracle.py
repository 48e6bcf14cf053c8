"""Slow, plain statement of the Zidivik decoder, one function per mechanism: what the tests compare the framework with.

Everything runs token by token or as a full matrix in one floating type (double by default) on the CPU.  Nothing is
cached, batched or fused, and nothing of the package is used.  A checkpoint is a dict `name -> tensor`, a configuration
the dict read from `config.json`."""

import math

import torch

from zozopel_oracle import causal_conv, gelu_tanh, rms, silu, softplus, unit


def position_vectors(positions, width, dtype=torch.float64):
    """`[T, width]`: sine and cosine of `p / 10000^(2i / width)` at entries 2i and 2i + 1."""
    p = positions.to(torch.float64)
    out = torch.empty(len(p), width, dtype=torch.float64)
    for c in range(width):
        a = p * 10000.0 ** (-2 * (c // 2) / width)
        out[:, c] = torch.sin(a) if c % 2 == 0 else torch.cos(a)
    return out.to(dtype)


def visible(T, window, first):
    """`[T, T]`: whether query i sees key j: causal, and near enough or among the first keys."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if window is None else (i - j < window)
    return (j <= i) & (near | (j < first))


def masked_attention(q, k, v, scale, mask):
    """Softmax attention, `q [T, H, D]`, `k [T, G, D]`, `v [T, G, V]`; query head h belongs to key head h // (H / G)."""
    share = q.shape[1] // k.shape[1]
    owner = [h // share for h in range(q.shape[1])]
    s = torch.einsum("ihd,jhd->hij", q, k[:, owner]) * scale
    s = s.masked_fill(~mask, -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v[:, owner])


def attention_mixer(h, w, p, m, eps, shared):
    """`shared`: keys and values of every earlier attention layer by number (this layer's own are added under its
    prefix's number)."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    me = int(p.split(".")[0][1:])
    q = rms((h @ w[p + "q"].T).view(T, H, D), eps)
    if m.get("kv_from") is None:
        k = rms((h @ w[p + "k"].T).view(T, G, D), eps)
        v = (h @ w[p + "v"].T).view(T, G, V)
        shared[me] = (k, v)
    else:
        k, v = shared[m["kv_from"]]
    mask = m.get("mask") or {}
    o = masked_attention(q, k, v, m["scale"], visible(T, mask.get("size"), mask.get("keep_first", 0)))
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w[p + "o"].T


def channel_delta_recurrence(q, k, v, decay, beta):
    """`q, k, decay [T, H, D]`, `v [T, H, V]`, `beta [T, H]` -> read-outs `[T, H, V]`; state zero at the start."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def channel_decay(a, a_log, dt_bias, H, D):
    """Decay per head and key channel from the low-rank projection `a [T, H * D]`."""
    rate = torch.exp(a_log)[None, :, None]
    return torch.exp(-rate * softplus(a + dt_bias).view(-1, H, D))


def channel_delta_mixer(h, w, p, m, eps):
    T, H, Hk, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def part(name, heads, d):
        return silu(causal_conv(h @ w[p + name].T, w[p + name + ".conv"])).view(T, heads, d)

    owner = [i // (H // Hk) for i in range(H)]
    q = unit(part("q", Hk, D))[:, owner] * D ** -0.5
    k = unit(part("k", Hk, D))[:, owner]
    v = part("v", H, V)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    decay = channel_decay((h @ w[p + "a1"].T) @ w[p + "a2"].T, w[p + "A_log"], w[p + "dt_bias"], H, D)
    o = rms(channel_delta_recurrence(q, k, v, decay, beta), eps) * w[p + "norm"]
    o = o * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, V)
    return o.reshape(T, H * V) @ w[p + "o"].T


def clipped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, w, p, top):
    """Experts of every token and their weights, `[T, top]` each."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best = torch.topk(z, top, dim=-1)
    return best.indices, torch.softmax(best.values, -1)


def sparse_ff(h, w, p, m):
    ids, weights = route(h, w, p, m["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(ids[t].tolist(), weights[t]):
            x = f"{p}e{e}."
            out[t] += c * clipped_expert(h[t], w[x + "gate"], w[x + "up"], w[x + "down"], m["expert"]["limit"])
    return out


def token_side(x, tokens, w, i, dim, eps):
    e = w["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ w[f"l{i}.side.gate"].T) * e) @ w[f"l{i}.side.proj"].T
    return rms(y, eps) * w[f"l{i}.side.norm"]


def layer(x, tokens, w, i, entry, cfg, shared):
    eps, p = cfg["norm"]["eps"], f"l{i}."
    h = rms(x, eps) * w[p + "norm1"]
    if entry["type"] == "attention":
        y = attention_mixer(h, w, p + "mix.", entry["mixer"], eps, shared)
    else:
        y = channel_delta_mixer(h, w, p + "mix.", entry["mixer"], eps)
    if entry["mlp"] is not None:
        y = y + sparse_ff(h, w, p + "mlp.", entry["mlp"])
    x = x + y
    return x + token_side(x, tokens, w, i, cfg["token_side"]["dim"], eps)


def forward(tokens, weights, cfg, dtype=torch.float64, trace=None):
    """Logits `[T, vocab]` of one sequence.  `trace`, a list, receives the residual stream after every layer."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in weights.items()}
    tokens = torch.as_tensor(tokens)
    x = w["embed"][tokens] + position_vectors(torch.arange(len(tokens)), cfg["width"], dtype)
    shared = {}
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, tokens, w, i, entry, cfg, shared)
        if trace is not None:
            trace.append(x)
    return (rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T


def greedy(tokens, weights, cfg, n, dtype=torch.float64):
    """`n` greedy tokens after the prompt, the whole sequence computed anew for each."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(forward(seq, weights, cfg, dtype)[-1].argmax()))
    return seq[len(tokens):]
