"""Small Zidivik configurations and random checkpoints, and the comparison of a replayed schedule with the oracle."""

import torch

import zidivik_oracle as oracle
from zozopel_cases import cut, error, interleave, replay, tokens, write_checkpoint  # noqa: F401


def moe(ff, experts, top, limit=1.0):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def attention(heads, kv_heads, dim, vdim, size, keep_first=0, kv_from=None, scale=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5,
         "mask": {"size": size, "keep_first": keep_first}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, ranks=(8, 8), mlp=None):
    """`ranks` (decay, gate) go into the tensors only."""
    return {"type": "channel_delta", "mlp": mlp, "ranks": ranks,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(layers, width, vocab, side, eps=1e-6):
    return {"architecture": "Zidivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side},
            "layers": layers}


CONFIGS = {
    # sizes that the tensor-core kernels take; two readers of one layer's keys, with masks of their own
    "plain": config([attention(4, 2, 32, 32, 24, 3, mlp=moe(48, 6, 2)), delta(4, 2, 32, 32, 4, mlp=moe(48, 6, 2)),
                     attention(4, 2, 32, 32, 50, 1, kv_from=0, mlp=moe(48, 6, 2)), delta(4, 2, 32, 32, 4, mlp=moe(48, 6, 2)),
                     attention(4, 2, 32, 32, 9, 0, kv_from=0, mlp=moe(48, 6, 2))], 128, 200, 8),
    # every size another one, values wider or narrower than keys, no feed-forward in places, one expert of one, all of all
    "mixed": config([delta(6, 3, 24, 40, 3, (5, 17), mlp=moe(40, 5, 3, 0.7)), attention(6, 3, 24, 40, 17, 5, mlp=moe(24, 1, 1)),
                     delta(2, 1, 40, 16, 2, (16, 3)), attention(5, 1, 40, 24, 70, 2, scale=0.31, mlp=moe(32, 4, 4, 2.5)),
                     attention(10, 1, 40, 24, 1, 1, kv_from=3)], 120, 333, 12, eps=1e-5),
    # sizes without any alignment, one tap
    "odd": config([attention(3, 3, 10, 7, 11, 2, mlp=moe(37, 3, 2)), delta(3, 1, 13, 9, 1, (3, 2), mlp=moe(21, 7, 5)),
                   attention(3, 3, 10, 7, 30, 0, kv_from=0)], 51, 77, 5),
    "delta_only": config([delta(4, 4, 16, 16, 4, mlp=moe(32, 4, 2)), delta(2, 1, 16, 32, 6)], 64, 96, 4),
    # query groups of more than 16 heads, head widths beyond 64 and 128
    "attention_only": config([attention(17, 1, 72, 136, 40, 70, mlp=moe(64, 8, 2)), attention(2, 2, 136, 64, 33, 1),
                              attention(4, 1, 200, 96, 1000, 0)], 64, 96, 8),
}


def checkpoint_config(cfg):
    """The file's form: what only the tensors tell is left out."""
    return dict(cfg, layers=[{k: v for k, v in e.items() if k != "ranks"} for e in cfg["layers"]])


def random_weights(cfg, seed=0):
    """Checkpoint tensors in bf16, sized so that every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    w, n, side = cfg["width"], len(cfg["layers"]), cfg["token_side"]["dim"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    def vec(n, mean=1.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    sd = {"embed": torch.randn(cfg["vocab"], w, generator=g), "side.embed": torch.randn(cfg["vocab"], n * side, generator=g),
          "final.norm": vec(w), "head": mat(cfg["vocab"], w)}
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}.mix."
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        sd[f"l{i}.norm1"] = vec(w)
        if e["type"] == "channel_delta":
            ra, rg = e["ranks"]
            for name, rows in (("q", G * D), ("k", G * D), ("v", H * V), ("b", H)):
                sd[p + name] = mat(rows, w, 1.5)
            for name, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                sd[p + name + ".conv"] = torch.randn(rows, m["conv"], generator=g) * 0.6
            sd[p + "a1"], sd[p + "a2"] = mat(ra, w), mat(H * D, ra, 2.0)
            sd[p + "g1"], sd[p + "g2"] = mat(rg, w), mat(H * V, rg, 1.5)
            sd[p + "A_log"], sd[p + "dt_bias"] = vec(H, -1.5, 1.0), vec(H * D, -1.0, 1.0)
            sd[p + "norm"], sd[p + "o"] = vec(V), mat(w, H * V)
        else:
            sd[p + "q"] = mat(H * D, w)
            if m.get("kv_from") is None:
                sd[p + "k"], sd[p + "v"] = mat(G * D, w), mat(G * V, w)
            sd[p + "g"], sd[p + "o"] = mat(H, w, 2.0), mat(w, H * V, 2.0)
        if e["mlp"] is not None:
            f, r, q = e["mlp"]["expert"]["ff"], e["mlp"]["router"]["experts"], f"l{i}.mlp."
            sd[q + "router"], sd[q + "router.b"] = mat(r, w, 1.5), vec(r, 0.0, 0.5)
            for x in range(r):
                sd[f"{q}e{x}.gate"], sd[f"{q}e{x}.up"], sd[f"{q}e{x}.down"] = mat(f, w), mat(f, w), mat(w, f, 2.0)
        sd[f"l{i}.side.gate"], sd[f"l{i}.side.proj"], sd[f"l{i}.side.norm"] = mat(side, w), mat(w, side), vec(w, 0.5)
    return {n: t.to(torch.bfloat16).contiguous() for n, t in sd.items()}


def write(path, cfg, weights) -> str:
    return write_checkpoint(path, checkpoint_config(cfg), weights)


def sensitivity(ids, weights, cfg, want, draws=3):
    """Per position: how far the logits move when every weight moves by one part in 2^9 (a bf16 rounding)."""
    worst = torch.zeros(len(ids), dtype=torch.float64)
    for seed in range(draws):
        g = torch.Generator().manual_seed(seed)
        moved = {n: t.double() * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=g, dtype=torch.float64))
                 for n, t in weights.items()}
        worst = torch.maximum(worst, error(oracle.forward(ids, moved, cfg), want))
    return worst


def close_calls(ids, weights, cfg, gap):
    """Positions from which on a router's choice is open: the last chosen and the first left out are nearer than `gap`."""
    seen, route = [], oracle.route

    def watch(h, w, p, top):
        z = torch.sort(h @ w[p + "router"].T + w[p + "router.b"], -1, descending=True).values
        if top < z.shape[1]:
            seen.append(z[:, top - 1] - z[:, top] < gap)
        return route(h, w, p, top)

    oracle.route = watch
    try:
        oracle.forward(ids, weights, cfg)
    finally:
        oracle.route = route
    return torch.stack(seen).any(0) if seen else torch.zeros(len(ids), dtype=torch.bool)


# a router that is this undecided may choose another expert after rounding
ROUTER_GAP = {"float32": 1e-4, "bfloat16": 0.06}
LIMIT = {"float32": 5e-5, "bfloat16": 4e-2}
PER_SENSITIVITY = {"float32": 2.0 ** -11, "bfloat16": 4.0}


def expectation(ids, weights, cfg):
    """`(logits, sensitivity, open router choices by precision)` of one request."""
    want = oracle.forward(ids, weights, cfg)
    return want, sensitivity(ids, weights, cfg, want), {d: close_calls(ids, weights, cfg, g) for d, g in ROUTER_GAP.items()}


def check(path, cfg, weights, dtype, device, requests, schedule, max_tokens, want=None, **kw):
    """Positions whose own experts hang on a rounding are left out; those behind them, whose keys and states may carry another
    expert's output, get three times the limit."""
    want = want or {n: expectation(t, weights, cfg) for n, t in requests.items()}
    got = replay(path, dtype, device, requests, schedule, max_tokens, **kw)
    for n, g in got.items():
        logits, moves, undecided = want[n]
        over = error(g, logits) / torch.clamp(PER_SENSITIVITY[dtype] * moves, min=LIMIT[dtype])
        over = torch.where(undecided[dtype], 0.0, over / (1 + 2 * (torch.cumsum(undecided[dtype], 0) > 0)))
        assert torch.isfinite(g).all() and float(over.max()) < 1, (n, int(over.argmax()), float(over.max()))
    return want
