"""Small Zozopel configurations and random checkpoints, and the comparison of a replayed schedule with the oracle."""

import json
import os

import numpy as np
import torch

import zozopel_oracle as oracle


def latent(heads, dim, rot, vdim, rank, base=10000.0, scale=None, ff=None):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank,
                      "scale": scale or (dim + rot) ** -0.5, "rot": {"base": base, "dims": rot}}}


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(layers, width, vocab, eps=1e-6, mult=0.4, embed=0.7, logit=1.5):
    return {"architecture": "Zozopel", "vocab": vocab, "width": width, "embedding": {"scale": embed},
            "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit, "layers": layers}


CONFIGS = {
    # latent first, sizes that the tensor-core kernels take, grouped delta heads
    "plain": config([latent(4, 32, 16, 32, 64, ff=160), delta(4, 2, 32, 32, 4, ff=160), latent(4, 32, 16, 32, 64, ff=160),
                     delta(4, 2, 32, 32, 4, ff=160)], 128, 200),
    # delta first and last, every size another one, no feed-forward in places, 1 and 3 taps' neighbours, one key head
    "mixed": config([delta(6, 3, 24, 40, 3, ff=96), latent(3, 24, 8, 40, 48, base=500.0, ff=72), delta(2, 1, 40, 16, 2),
                     latent(5, 16, 24, 8, 72, scale=0.31), delta(3, 3, 16, 48, 5, ff=56)], 120, 333, eps=1e-5, mult=1.0,
                    embed=1.3, logit=0.5),
    # sizes without any alignment
    "odd": config([latent(3, 10, 6, 11, 21, ff=37), delta(3, 1, 13, 9, 4, ff=37)], 51, 77),
    "delta_only": config([delta(4, 4, 16, 16, 4, ff=64), delta(2, 1, 16, 32, 4)], 64, 96),
    "latent_only": config([latent(2, 64, 48, 56, 112, base=50.0, ff=64), latent(17, 8, 8, 8, 32)], 64, 96),
}


def random_weights(cfg, seed=0):
    """Checkpoint tensors in bf16, sized so that every mechanism moves the logits."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain * cols ** -0.5

    def vec(n, mean=1.0, std=0.2):
        return mean + std * torch.randn(n, generator=g)

    sd = {"embed": torch.randn(cfg["vocab"], w, generator=g), "final.norm": vec(w), "head": mat(cfg["vocab"], w)}
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}.mix."
        if e["type"] == "delta":
            qk, v, h = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"]
            for n, rows in (("q", qk), ("k", qk), ("v", v), ("g", v), ("b", h), ("a", h)):
                sd[p + n] = mat(rows, w, 1.5)
            for n, rows in (("q", qk), ("k", qk), ("v", v)):
                sd[p + n + ".conv"] = torch.randn(rows, m["conv"], generator=g) * 0.6
            sd[p + "A_log"], sd[p + "dt_bias"] = vec(h, -2.5, 1.0), vec(h, 0.0, 0.5)
            sd[p + "norm"], sd[p + "o"] = vec(m["vdim"]), mat(w, v)
        else:
            h = m["heads"]
            sd[p + "q"] = mat(h * (m["dim"] + m["rot_dim"]), w)
            sd[p + "dkv"] = mat(m["kv_rank"] + m["rot_dim"], w)
            sd[p + "dkv.norm"] = vec(m["kv_rank"])
            sd[p + "uk"] = mat(h * m["dim"], m["kv_rank"])
            sd[p + "uv"] = mat(h * m["vdim"], m["kv_rank"])
            sd[p + "g"], sd[p + "o"] = mat(h * m["vdim"], w), mat(w, h * m["vdim"])
        sd[f"l{i}.norm1"], sd[f"l{i}.ls1"] = vec(w), vec(w)
        if e["mlp"] is not None:
            ff = e["mlp"]["ff"]
            sd[f"l{i}.mlp.gate"], sd[f"l{i}.mlp.up"], sd[f"l{i}.mlp.down"] = mat(ff, w), mat(ff, w), mat(w, ff)
            sd[f"l{i}.norm2"], sd[f"l{i}.ls2"] = vec(w), vec(w)
    return {n: t.to(torch.bfloat16).contiguous() for n, t in sd.items()}


def write_checkpoint(path, cfg, weights) -> str:
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(weights, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens(n, vocab, seed):
    return np.random.RandomState(seed).randint(0, vocab, n).tolist()


def replay(path, dtype, device, requests, schedule, max_tokens, page_size=64, max_requests=4):
    """Run `schedule` (steps of `(request, number of tokens)`) and return every request's logits, `[tokens, vocab]`."""
    from sglang_jax_b200.parallel import state as ps
    from sglang_jax_b200.trace_replay import TraceReplayer
    ps.reset_state()
    r = TraceReplayer(path, dtype, max_tokens, max_requests=max_requests, page_size=page_size, device=device)
    at, out = {}, {n: [] for n in requests}
    for step in schedule:
        entries = []
        for name, n in step:
            lo = at.get(name, 0)
            ids = requests[name][lo:lo + n]
            assert len(ids) == n
            entries.append({"id": name, "tokens": ids, "want": list(range(n))})
            at[name] = lo + n
        logits, o = r.step(entries), 0
        for name, n in step:
            out[name].append(logits[o:o + n])
            o += n
        for name, _ in step:
            if at[name] == len(requests[name]):
                r.finish(name)
    assert r.allocator.available_size() == r.worker.max_total_num_tokens and r.pool.available_size() == max_requests
    if device == "cuda":
        from sglang_jax_b200.ops import native
        native.check_status()
        assert native.LOADED
    return {n: torch.from_numpy(np.concatenate(v)).double() for n, v in out.items() if v}


def error(got, want):
    """Per position: root mean square of the difference over the vocabulary, mean taken off, over the logits' own."""
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / s.pow(2).mean().sqrt())


def sensitivity(ids, weights, cfg, want, draws=3):
    """Per position: how far the logits move when every weight moves by one part in 2^9 (a bf16 rounding).  The design has
    places where that is a lot, for instance a first token whose key and query are almost orthogonal: its read-out is
    nearly zero and normalised all the same."""
    worst = torch.zeros(len(ids), dtype=torch.float64)
    for seed in range(draws):
        g = torch.Generator().manual_seed(seed)
        moved = {n: t.double() * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=g, dtype=torch.float64))
                 for n, t in weights.items()}
        worst = torch.maximum(worst, error(oracle.forward(ids, moved, cfg), want))
    return worst


LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}
PER_SENSITIVITY = {"float32": 2.0 ** -12, "bfloat16": 4.0}


def expectation(ids, weights, cfg):
    """`(logits, sensitivity)` of one request."""
    want = oracle.forward(ids, weights, cfg)
    return want, sensitivity(ids, weights, cfg, want)


def check(path, cfg, weights, dtype, device, requests, schedule, max_tokens, want=None, **kw):
    want = want or {n: expectation(t, weights, cfg) for n, t in requests.items()}
    got = replay(path, dtype, device, requests, schedule, max_tokens, **kw)
    for n, g in got.items():
        logits, moves = want[n]
        over = error(g, logits) / torch.clamp(PER_SENSITIVITY[dtype] * moves, min=LIMIT[dtype])
        assert torch.isfinite(g).all() and float(over.max()) < 1, (n, int(over.argmax()), float(over.max()))
    return want


def cut(total, sizes):
    """Portions of the given sizes, repeated, that add up to `total`."""
    out, i = [], 0
    while total:
        n = min(sizes[i % len(sizes)], total)
        out.append(n)
        total -= n
        i += 1
    return out


def interleave(requests, portions, live=4):
    """A schedule in which up to `live` requests advance together, each by its own list of portions."""
    waiting, running, steps = list(requests), [], []
    left = {n: list(portions[n]) for n in requests}
    while waiting or running:
        while waiting and len(running) < live:
            running.append(waiting.pop(0))
        steps.append([(n, left[n].pop(0)) for n in running])
        running = [n for n in running if left[n]]
    return steps
