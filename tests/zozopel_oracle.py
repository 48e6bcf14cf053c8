"""Slow, plain statement of the Zozopel decoder, one function per mechanism: what the tests compare the framework with.

Everything runs token by token or as a full matrix in one floating type (double by default) on the CPU.  Nothing is
cached, batched or fused, and nothing of the package is used.  A checkpoint is a dict `name -> tensor`, a configuration
the dict read from `config.json`."""

import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x, eps=1e-6):
    """x divided by its Euclidean length over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate(x, positions, base):
    """Interleaved rotary embedding of the whole last axis; `x [T, ..., d]`, `positions [T]`."""
    d = x.shape[-1]
    out = torch.empty_like(x)
    for i in range(d // 2):
        a = positions.to(x.dtype) * base ** (-2 * i / d)
        a = a.view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def causal_conv(x, w):
    """Depth-wise convolution over time, `x [T, C]`, `w [C, K]` (last tap = the current token), zeros before the start."""
    T, K = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y


def delta_recurrence(q, k, v, decay, beta):
    """`q, k [T, H, D]`, `v [T, H, V]`, `decay, beta [T, H]` -> read-outs `[T, H, V]`; state zero at the start."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def delta_mixer(h, w, p, m, eps):
    """`p` is the tensors' prefix, `m` the mixer's sizes."""
    T, H, Hk, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def part(name, heads, d):
        return silu(causal_conv(h @ w[p + name].T, w[p + name + ".conv"])).view(T, heads, d)

    owner = [i // (H // Hk) for i in range(H)]
    q = unit(part("q", Hk, D))[:, owner] * D ** -0.5
    k = unit(part("k", Hk, D))[:, owner]
    v = part("v", H, V)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = delta_recurrence(q, k, v, decay, beta)
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ w[p + "o"].T


def softmax_attention(q, k, v, scale):
    """Causal softmax attention; `q, k [T, H, D]`, `v [T, H, V]`."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), 1), -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def latent_mixer(h, w, p, m, eps):
    T, H, D, R, V, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    q = torch.cat([q[..., :D], rotate(q[..., D:], pos, m["rot"]["base"])], -1)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :C], eps) * w[p + "dkv.norm"]
    shared = rotate(down[:, C:], pos, m["rot"]["base"])
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, D), shared[:, None].expand(T, H, R)], -1)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    o = softmax_attention(q, k, v, m["scale"]).reshape(T, H * V)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def dense_ff(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer(x, w, i, entry, cfg):
    eps, m, p = cfg["norm"]["eps"], cfg["residual_mult"], f"l{i}."
    mix = {"delta": delta_mixer, "latent_attention": latent_mixer}[entry["type"]]
    x = x + m * rms(mix(x, w, p + "mix.", entry["mixer"], eps), eps) * w[p + "norm1"] * w[p + "ls1"]
    if entry["mlp"] is not None:
        x = x + m * rms(dense_ff(x, w, p + "mlp."), eps) * w[p + "norm2"] * w[p + "ls2"]
    return x


def forward(tokens, weights, cfg, dtype=torch.float64, trace=None):
    """Logits `[T, vocab]` of one sequence.  `trace`, a list, receives the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, w, i, entry, cfg)
        if trace is not None:
            trace.append(x)
    return (rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]


def greedy(tokens, weights, cfg, n, dtype=torch.float64):
    """`n` greedy tokens after the prompt, the whole sequence computed anew for each."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(forward(seq, weights, cfg, dtype)[-1].argmax()))
    return seq[len(tokens):]
