"""Slow, plain statement of the Kunudra decoder, one function per mechanism: what the tests compare the framework with.

Everything runs as full matrices over one sequence in one floating type (double by default) on the CPU.  Nothing is cached,
batched or fused, and nothing of the package is used.  A checkpoint is a dict `name -> tensor`, a configuration the dict
read from `config.json`."""

import math

import torch

from zozopel_oracle import rms, rotate, silu


def norm_sum(x, y, scale, alpha, weight, eps):
    """Residual step with the norm behind the sum; the norm's weight is stored around zero."""
    return rms(alpha * x + y * scale, eps) * (1 + weight)


def pair_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token: its predecessor and itself, hashed; the last row for the first token."""
    rows, prev = [], None
    for t in tokens:
        rows.append(buckets if prev is None else (prev * mul_prev + t * mul_cur) % buckets)
        prev = t
    return rows


def embedding(tokens, w, cfg):
    c = cfg["embedding"]["bigram"]
    toks = [int(t) for t in tokens]
    return w["embed"][toks] + w["bigram"][pair_rows(toks, c["buckets"], c["mul_prev"], c["mul_cur"])]


def visible(T, size):
    """`[T, T]`: whether query i sees key j: itself and the `size - 1` before it (None: all before it)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else torch.ones(T, T, dtype=torch.bool))


def slopes(H):
    return torch.tensor([2.0 ** (-8 * (h + 1) / H) for h in range(H)], dtype=torch.float64)


def distance_bias(T, H):
    """`[H, T, T]`: slope of the head times how far back the key is."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return slopes(H)[:, None, None] * (i - j)


def cap(score, limit):
    return limit * torch.tanh(score / limit) if limit else score


def sink_softmax(score, mask, sink):
    """Softmax of `score [H, T, S]` over the visible keys and one more entry per head that has no value."""
    s = score.masked_fill(~mask, -math.inf)
    return torch.softmax(torch.cat([s, sink[:, None, None].expand(-1, s.shape[1], 1)], -1), -1)[..., :-1]


def mix_values(v, first, share):
    return (1 - share) * v + share * first


def attention_mixer(h, w, p, m, eps, first):
    """`first`: a list, empty until the first layer that mixes values has put its own values there."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, D)
    k = (rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, D)
    v = h @ w[p + "v"].T
    if m.get("v_mix"):
        if first:
            v = mix_values(v, first[0], w[p + "vmix"])
        else:
            first.append(v)
    v = v.view(T, G, V)
    owner = [i // (H // G) for i in range(H)]
    s = cap(torch.einsum("ihd,jhd->hij", q, k[:, owner]) * m["scale"], m.get("softcap"))
    s = s - distance_bias(T, H).to(s.dtype)
    a = sink_softmax(s, visible(T, (m.get("mask") or {}).get("size")), w[p + "sink"])
    return torch.einsum("hij,jhd->ihd", a, v[:, owner]).reshape(T, H * V) @ w[p + "o"].T


def latent_mixer(h, w, p, m, eps):
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos, base = torch.arange(T), m["rot"]["base"]
    c_q = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (c_q @ w[p + "uq"].T).view(T, H, D + R)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :C], eps) * w[p + "dkv.norm"]
    k_rot = rotate(down[:, C:], pos, base)
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    s = torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihd,jd->hij", rotate(q[..., D:], pos, base), k_rot)
    a = sink_softmax(s * m["scale"], visible(T, (m.get("mask") or {}).get("size")), w[p + "sink"])
    return torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * V) @ w[p + "o"].T


def gated(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, w, p, top, scale):
    """Outputs chosen by every token and their weights, `[T, top]` each: the choice sees the correction, the weight does not."""
    s = torch.softmax(h @ w[p + "router"].T, -1)
    ids = torch.topk(s + w[p + "correction"], top, dim=-1).indices
    return ids, s.gather(1, ids) * scale


def shared_ff(h, w, p):
    return torch.sigmoid(h @ w[p + "shared.sg"].T) * gated(h, w, p + "shared.")


def sparse_ff(h, w, p, m):
    """Outputs from number `experts` on hand the input back."""
    r = m["router"]
    ids, weights = route(h, w, p, r["top"], r["scale"])
    out = shared_ff(h, w, p) if m.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(ids[t].tolist(), weights[t]):
            out[t] += c * (gated(h[t], w, f"{p}e{e}.") if e < r["experts"] else h[t])
    return out


def layer(x, w, i, entry, cfg, first):
    eps, alpha, p = cfg["norm"]["eps"], cfg["postln_alpha"], f"l{i}."
    if entry["type"] == "attention":
        y = attention_mixer(x, w, p + "mix.", entry["mixer"], eps, first)
    else:
        y = latent_mixer(x, w, p + "mix.", entry["mixer"], eps)
    x = norm_sum(x, y, w[p + "ls1"], alpha, w[p + "norm1"], eps)
    if entry.get("mlp") is None:
        return x
    y = gated(x, w, p + "mlp.") if entry["mlp"]["kind"] == "dense" else sparse_ff(x, w, p + "mlp.", entry["mlp"])
    return norm_sum(x, y, w[p + "ls2"], alpha, w[p + "norm2"], eps)


def forward(tokens, weights, cfg, dtype=torch.float64, trace=None):
    """Logits `[T, vocab]` of one sequence.  `trace`, a list, receives the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    x, first = embedding(tokens, w, cfg), []
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, w, i, entry, cfg, first)
        if trace is not None:
            trace.append(x)
    return (rms(x, cfg["norm"]["eps"]) * (1 + w["final.norm"])) @ w["embed"].T


def greedy(tokens, weights, cfg, n, dtype=torch.float64):
    """`n` greedy tokens after the prompt, the whole sequence computed anew for each."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(forward(seq, weights, cfg, dtype)[-1].argmax()))
    return seq[len(tokens):]
