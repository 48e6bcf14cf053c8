"""Small Kunudra configurations and random checkpoints, and the comparison of a replayed schedule with the oracle."""

import itertools

import torch

import kunudra_oracle as oracle
from zozopel_cases import cut, error, interleave, replay, tokens, write_checkpoint  # noqa: F401


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, identity=0, scale=1.0, shared=None):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": shared and {"ff": shared},
            "router": {"experts": experts, "top": top, "identity": identity, "scale": scale}}


def attention(heads, kv_heads, dim, vdim, size, softcap=None, v_mix=False, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or 1.3 * dim ** -0.5,
                      "softcap": softcap, "v_mix": v_mix, "mask": size and {"size": size}}}


def latent(heads, dim, rot, vdim, rank, q_rank, size, base=10000.0, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                      "scale": scale or 1.3 * (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot},
                      "mask": size and {"size": size}}}


def config(layers, width, vocab, buckets=97, mul_prev=13, mul_cur=5, eps=1e-6, alpha=1.7):
    return {"architecture": "Kunudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": layers}


CONFIGS = {
    # sizes that the tensor-core kernels take; two readers of the first values; identity choices and a shared expert
    "plain": config([attention(4, 2, 32, 32, 24, 9.0, True, mlp=moe(48, 6, 2, 2, 1.3, 40)),
                     latent(4, 40, 16, 48, 72, 56, 24, mlp=dense(160)),
                     attention(4, 2, 32, 32, 50, 4.0, True, mlp=moe(48, 6, 3, 3, 0.8, 40)),
                     latent(4, 40, 24, 32, 80, 48, 9, 500.0, mlp=moe(48, 6, 2, 2, 2.0, 24)),
                     attention(4, 2, 32, 32, 9, 30.0, True)], 128, 200),
    # no routers, whose choices may hang on a rounding
    "dense": config([attention(6, 2, 64, 64, 70, 5.0, True, mlp=dense(200)), latent(6, 48, 32, 64, 96, 80, 40, 1000.0, mlp=dense(144)),
                     attention(2, 2, 64, 64, 20, 2.0, True), latent(3, 32, 24, 40, 64, 48, 100, mlp=dense(96))], 192, 150, alpha=2.2),
    # every size another one, values wider or narrower than keys, a layer that keeps its values to itself, no cap, no window, no
    # feed-forward in places, no identity choice, no shared expert, one expert of one, all of all, other hash and constants
    "mixed": config([latent(6, 24, 8, 40, 56, 40, 17, 300.0, mlp=moe(40, 5, 3, 1, 0.7, 32)),
                     attention(6, 3, 24, 40, 33, None, False, mlp=moe(24, 1, 1, 0, 1.0)), latent(2, 40, 24, 16, 32, 96, 70),
                     attention(5, 1, 40, 24, 70, 2.5, True, scale=0.31, mlp=moe(32, 4, 4, 0, 2.5, 8)),
                     attention(6, 3, 16, 8, None, 12.0, True, mlp=dense(72)), latent(3, 16, 8, 24, 40, 24, None, mlp=moe(24, 2, 3, 4, 1.1)),
                     attention(4, 2, 40, 24, 1, 1.0, False)], 120, 333, 211, 7, 31, eps=1e-5, alpha=0.6),
    # sizes without any alignment
    "odd": config([attention(3, 3, 10, 7, 11, 3.0, True, mlp=moe(37, 3, 2, 2, 1.5, 13)),
                   latent(3, 10, 6, 11, 21, 19, 30, mlp=dense(37)), attention(3, 3, 13, 7, 30, 20.0, True),
                   latent(2, 7, 2, 5, 9, 5, 6, mlp=moe(21, 7, 5, 1, 1.0, 11))], 51, 77, 1, 3, 2),
    "latent_only": config([latent(2, 64, 48, 56, 112, 64, 40, 50.0, mlp=dense(64)), latent(17, 8, 8, 8, 32, 72, 100)], 64, 96, 1009,
                          1_000_003, 999_983),
    # query groups of more than 16 heads, head widths beyond 64 and 128
    "attention_only": config([attention(17, 1, 72, 136, 40, 5.0, True, mlp=moe(64, 8, 2, 1, 1.0, 64)),
                              attention(2, 2, 136, 64, 33, None, True), attention(4, 1, 200, 136, 1000, 50.0, True)], 64, 96),
}
# (layers that mix values hold equally many)
CONFIGS["mixed"]["layers"][4]["mixer"].update(kv_heads=1, heads=6, vdim=24)
CONFIGS["attention_only"]["layers"][1]["mixer"]["vdim"] = 68


def random_weights(cfg, seed=0):
    """Checkpoint tensors in bf16, sized so that every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    def vec(n, mean=1.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    def three(p, ff):
        sd[p + "gate"], sd[p + "up"], sd[p + "down"] = mat(ff, w, 1.5), mat(ff, w, 1.5), mat(w, ff, 1.5)

    sd = {"embed": torch.randn(cfg["vocab"], w, generator=g),
          "bigram": torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, w, generator=g), "final.norm": vec(w, 0.0)}
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}.mix."
        H, D, V = m["heads"], m["dim"], m["vdim"]
        sd[f"l{i}.norm1"], sd[f"l{i}.ls1"] = vec(w, 0.0), vec(w)
        sd[p + "sink"], sd[p + "o"] = vec(H, 0.5, 1.0), mat(w, H * V, 2.0)
        if e["type"] == "attention":
            G = m["kv_heads"]
            sd[p + "q"], sd[p + "k"], sd[p + "v"] = mat(H * D, w), mat(G * D, w), mat(G * V, w)
            sd[p + "q.norm"], sd[p + "k.norm"] = vec(H * D), vec(G * D)
            if m["v_mix"]:
                sd[p + "vmix"] = vec(1, 0.4, 0.1)[0]
        else:
            R, C = m["rot_dim"], m["kv_rank"]
            sd[p + "dq"], sd[p + "dq.norm"], sd[p + "uq"] = mat(m["q_rank"], w), vec(m["q_rank"]), mat(H * (D + R), m["q_rank"])
            sd[p + "dkv"], sd[p + "dkv.norm"] = mat(C + R, w), vec(C)
            sd[p + "uk"], sd[p + "uv"] = mat(H * D, C), mat(H * V, C)
        if e["mlp"] is None:
            continue
        f, q = e["mlp"], f"l{i}.mlp."
        sd[f"l{i}.norm2"], sd[f"l{i}.ls2"] = vec(w, 0.0), vec(w)
        if f["kind"] == "dense":
            three(q, f["ff"])
            continue
        n = f["router"]["experts"]
        sd[q + "router"] = mat(n + f["router"]["identity"], w, 2.5)
        sd[q + "correction"] = vec(n + f["router"]["identity"], 0.0, 0.15)
        for x in range(n):
            three(f"{q}e{x}.", f["expert"]["ff"])
        if f["shared"]:
            three(q + "shared.", f["shared"]["ff"])
            sd[q + "shared.sg"] = mat(1, w, 2.0)
    return {n: t.to(torch.bfloat16).contiguous() for n, t in sd.items()}


def write(path, cfg, weights) -> str:
    return write_checkpoint(path, cfg, weights)


def sensitivity(ids, weights, cfg, want, draws=3):
    """Per position: how far the logits move when every weight moves by one part in 2^9 (a bf16 rounding) while the routers'
    choices stay."""
    choices, route = [], oracle.route

    def keep(*a):
        choices.append(route(*a)[0])
        return route(*a)

    def again(h, w, p, top, scale):
        chosen = choices[next(turn)]
        return chosen, torch.softmax(h @ w[p + "router"].T, -1).gather(1, chosen) * scale

    worst = torch.zeros(len(ids), dtype=torch.float64)
    try:
        oracle.route = keep
        oracle.forward(ids, weights, cfg)
        oracle.route = again
        for seed in range(draws):
            g, turn = torch.Generator().manual_seed(seed), itertools.count()
            moved = {n: t.double() * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=g, dtype=torch.float64))
                     for n, t in weights.items()}
            worst = torch.maximum(worst, error(oracle.forward(ids, moved, cfg), want))
    finally:
        oracle.route = route
    return worst


def close_calls(ids, weights, cfg, gap):
    """Positions at which a router's choice is open: the last chosen and the first left out are nearer than `gap`."""
    seen, route = [], oracle.route

    def watch(h, w, p, top, scale):
        s = torch.softmax(h @ w[p + "router"].T, -1) + w[p + "correction"]
        s = torch.sort(s, -1, descending=True).values
        if top < s.shape[1]:
            seen.append(s[:, top - 1] - s[:, top] < gap)
        return route(h, w, p, top, scale)

    oracle.route = watch
    try:
        oracle.forward(ids, weights, cfg)
    finally:
        oracle.route = route
    return torch.stack(seen).any(0) if seen else torch.zeros(len(ids), dtype=torch.bool)


# a router that is this undecided may choose another expert after rounding
ROUTER_GAP = {"float32": 1e-5, "bfloat16": 0.015}
LIMIT = {"float32": 5e-5, "bfloat16": 4e-2}
PER_SENSITIVITY = {"float32": 2.0 ** -11, "bfloat16": 4.0}


def expectation(ids, weights, cfg):
    """`(logits, sensitivity, open router choices by precision)` of one request."""
    want = oracle.forward(ids, weights, cfg)
    return want, sensitivity(ids, weights, cfg, want), {d: close_calls(ids, weights, cfg, g) for d, g in ROUTER_GAP.items()}


def check(path, cfg, weights, dtype, device, requests, schedule, max_tokens, want=None, **kw):
    """Positions whose own experts plainly hang on a rounding are left out; those behind them, whose keys may carry another
    expert's output, get five times the limit.  In bf16 one position in twenty may be over its limit all the same where there
    are routers: roundings add up over the layers, and a choice that is less close may turn, too."""
    want = want or {n: expectation(t, weights, cfg) for n, t in requests.items()}
    got = replay(path, dtype, device, requests, schedule, max_tokens, **kw)
    for n, g in got.items():
        logits, moves, undecided = want[n]
        over = error(g, logits) / torch.clamp(PER_SENSITIVITY[dtype] * moves, min=LIMIT[dtype])
        over = torch.where(undecided[dtype], 0.0, over / (1 + 4 * (torch.cumsum(undecided[dtype], 0) > 0)))
        allowed = max(1, len(over) // 20) if dtype == "bfloat16" and undecided[dtype].any() else 0
        assert torch.isfinite(g).all() and int((over >= 1).sum()) <= allowed, (n, int(over.argmax()), float(over.max()))
    return want
