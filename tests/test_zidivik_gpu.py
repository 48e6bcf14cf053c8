"""Zidivik on the GPU: its kernels against plain double-precision statements, and schedules, caches and generation of
whole models against the oracle, in bf16 and in fp32."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import zidivik_cases as cases
import zidivik_oracle as oracle
from test_zidivik_cpu import first_token_model, needle_model, needle_prompt

pytestmark = pytest.mark.gpu
DTYPES = ["bfloat16", "float32"]
TORCH = {"bfloat16": torch.bfloat16, "float32": torch.float32}


@pytest.fixture(scope="module")
def native():
    from sglang_jax_b200.ops import native as n
    n.lib()
    yield n
    torch.cuda.synchronize()
    n.check_status()


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in cases.CONFIGS.items():
        w = cases.random_weights(cfg, seed=len(name))
        out[name] = (cases.write(str(tmp_path_factory.mktemp(name)), cfg, w), cfg, w)
    return out


def _i32(x):
    return torch.tensor(np.asarray(x), dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------ stream kernels
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("W", [24, 51, 1000, 4096])
def test_stream_kernels(native, dtype, W):
    g = torch.Generator().manual_seed(W)
    T, eps = 7, 1e-5
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    table, ids = rnd(9, W).to(dtype), torch.tensor([3, 0, 8, 3, 7, 1, 2], dtype=torch.int32)
    pos = torch.tensor([0, 1, 2, 63, 1000, 131071, 1048575], dtype=torch.int32)
    turns = 10000.0 ** (-2.0 * torch.arange((W + 1) // 2, dtype=torch.float64) / W) / (2 * np.pi)
    x, h = native.embed_scaled(ids.cuda(), table.cuda(), 1.0, pos.cuda(), turns.cuda())
    want = table[ids.long()].double() + oracle.position_vectors(pos, W)
    assert torch.allclose(x.cpu().double(), want, atol=1e-6) and torch.equal(h, x.to(dtype))
    y, s, s2 = (rnd(T, W) * 3).to(dtype), rnd(W), rnd(W)
    base = x.cpu().double()
    want = base + oracle.rms(y.double(), eps) * s.double()
    h = native.postnorm_add_norm(y.cuda(), x, s.cuda(), eps, s2.cuda(), 1e-3)
    assert torch.allclose(x.cpu().double(), want, atol=2e-6, rtol=2e-6)
    assert torch.allclose(h.cpu().double(), oracle.rms(want, 1e-3) * s2.double(), atol=tol, rtol=tol)
    expert, weights = rnd(20, W).to(dtype), torch.rand(T, 3, generator=g)
    rows = torch.randint(-1, 20, (T, 3), generator=g, dtype=torch.int32)
    for k in (0, 3):
        want = x.cpu().double() + y.double()
        if k:
            want += ((weights * (rows >= 0)).unsqueeze(-1).double() * expert[rows.clamp_min(0).long()].double()).sum(1)
        h = native.stream_add(y.cuda(), x, *((expert.cuda(), weights.cuda(), rows.cuda()) if k else ()))
        assert torch.allclose(x.cpu().double(), want, atol=5e-6, rtol=5e-6) and torch.equal(h, x.to(dtype))


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("F", [16, 37, 96, 1000])
def test_gates_of_the_feed_forward_and_the_token_input(native, dtype, F):
    g = torch.Generator().manual_seed(F)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    x = (torch.randn(5, 2 * F, generator=g) * 3).to(dtype)
    for limit in (0.5, 7.0):
        eye = torch.eye(F, dtype=torch.float64)
        want = oracle.clipped_expert(x.double(), eye.repeat(1, 2)[:, :2 * F] * torch.tensor([1.0] * F + [0.0] * F),
                                     eye.repeat(1, 2) * torch.tensor([0.0] * F + [1.0] * F), eye, limit)
        assert torch.allclose(native.clipped_swiglu(x.cuda(), limit).cpu().double(), want, atol=tol, rtol=tol)
    table, ids = torch.randn(11, 3 * F + 5, generator=g).to(dtype), torch.tensor([0, 10, 4, 4, 9], dtype=torch.int32)
    z = (torch.randn(5, F, generator=g) * 3).to(dtype)
    for off in (0, F, 2 * F + 5):
        want = oracle.gelu_tanh(z.double()) * table[ids.long(), off:off + F].double()
        got = native.token_side_gate(z.cuda(), table.cuda(), ids.cuda(), off)
        assert torch.allclose(got.cpu().double(), want, atol=tol, rtol=tol)


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("T", [1, 5, 300])
@pytest.mark.parametrize("E,k,K", [(1, 1, 64), (10, 4, 192), (64, 8, 129), (500, 16, 40)])
def test_routing_by_logit(native, dtype, T, E, k, K):
    from sglang_jax_b200.ops import moe_native
    g = torch.Generator().manual_seed(E + T)
    x, w = torch.randn(T, K, generator=g).to(dtype), (torch.randn(E, K, generator=g) * K ** -0.5).to(dtype)
    b = torch.randn(E, generator=g).to(dtype)
    z = x.double() @ w.double().T + b.double()
    best = torch.topk(z, k, -1)
    weights, ids = moe_native.route_by_logit(x.cuda(), w.cuda(), b.cuda(), k)
    assert torch.allclose(weights.cpu().double(), torch.softmax(best.values, -1), atol=2e-6)
    chosen = torch.gather(z, 1, ids.cpu().long())
    assert torch.allclose(chosen, best.values, atol=1e-5)
    assert all(len(set(r)) == k for r in ids.tolist())


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("T", [1, 9, 70, 400])
@pytest.mark.parametrize("W,I,E,k", [(64, 48, 6, 2), (51, 37, 3, 3), (192, 72, 10, 4), (128, 40, 1, 1)])
def test_experts_on_the_stream(native, dtype, T, W, I, E, k):
    """Few and many tokens (one expert may get none, or all of them)."""
    from sglang_jax_b200.layers.moe import FusedMoE
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    g = torch.Generator().manual_seed(T + W)
    with torch.device("cuda"):
        m = FusedMoE(E, W, I, dtype, activation="clipped_swiglu", act_limit=0.8)
    w13, w2 = (torch.randn(E, 2 * I, W, generator=g) * W ** -0.5).to(dtype), (torch.randn(E, W, I, generator=g) * I ** -0.5).to(dtype)
    m.w13_weight.data.copy_(w13)
    m.w2_weight.data.copy_(w2)
    x, mixed = torch.randn(T, W, generator=g).to(dtype), torch.randn(T, W, generator=g).to(dtype)
    stream = torch.randn(T, W, generator=g)
    ids = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).int()
    weights = torch.softmax(torch.randn(T, k, generator=g), -1)
    want = stream.double() + mixed.double()
    for e in range(E):
        y = oracle.clipped_expert(x.double(), w13[e, :I].double(), w13[e, I:].double(), w2[e].double(), 0.8)
        want += (weights.double() * (ids == e)).sum(1, keepdim=True) * y
    s = stream.cuda()
    h = m.forward_stream(x.cuda(), weights.cuda(), ids.cuda(), mixed.cuda(), s)
    tol = 1e-5 if dtype == torch.float32 else 3e-2
    assert torch.allclose(s.cpu().double(), want, atol=tol, rtol=tol) and torch.equal(h, s.to(dtype))


# ------------------------------------------------------------------ delta rule with decays per channel
def _delta_case(H, Hk, D, V, K, lens, dtype, strong, seed=0):
    """Inputs of `delta_scan`, the oracle's read-outs, and freshly dirtied pools."""
    g = torch.Generator().manual_seed(seed)
    B, T, ch = len(lens), sum(lens), 2 * Hk * D + H * V
    bo = -(-ch // 8) * 8
    proj = torch.randn(T, bo + 8 * -(-H // 8), generator=g).to(dtype)
    a = (torch.randn(T, H * D, generator=g) * 2).to(dtype)
    conv = (torch.randn(ch, K, generator=g) * 0.5).to(dtype)
    # decays near one, and decays that forget a channel within a token (their logarithms add up to hundreds)
    a_log, dt = torch.randn(H, generator=g) * 0.5 + (2.5 if strong else -2), torch.randn(H * D, generator=g)
    cu = np.concatenate([[0], np.cumsum(lens)])
    want = []
    for b in range(B):
        x = proj[cu[b]:cu[b + 1]].double()
        y = oracle.silu(oracle.causal_conv(x[:, :ch], conv.double()))
        own = [i // (H // Hk) for i in range(H)]
        q = oracle.unit(y[:, :Hk * D].view(-1, Hk, D))[:, own] * D ** -0.5
        k = oracle.unit(y[:, Hk * D:2 * Hk * D].view(-1, Hk, D))[:, own]
        decay = oracle.channel_decay(a[cu[b]:cu[b + 1]].double(), a_log.double(), dt.double(), H, D)
        want.append(oracle.channel_delta_recurrence(q, k, y[:, 2 * Hk * D:].view(-1, H, V), decay, torch.sigmoid(x[:, bo:bo + H])))
    pools = lambda: (torch.randn(B + 3, ch, K - 1, generator=g).to(dtype).cuda(), torch.randn(B + 3, H, D, V, generator=g).cuda())
    args = (-1, bo, -1, conv.cuda(), a_log.cuda(), dt.cuda())
    slots = torch.tensor([B + 2 - b for b in range(B)], device="cuda")
    return proj.cuda(), a.cuda(), args, torch.cat(want), pools, slots, cu


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("H,Hk,D,V,K,lens", [
    (6, 2, 64, 48, 4, [70, 1, 33]), (6, 3, 24, 40, 3, [50, 9, 4]), (2, 1, 128, 128, 4, [130]), (3, 3, 100, 36, 2, [41, 2]),
    (2, 1, 16, 200, 6, [23]), (2, 2, 256, 64, 1, [40]), (3, 1, 13, 9, 4, [18, 5]), (16, 16, 128, 128, 4, [9] * 40),
    (16, 4, 32, 32, 4, [6] * 150)])
def test_channel_delta_scan_whole_in_portions_and_token_by_token(native, H, Hk, D, V, K, lens, strong, dtype):
    proj, a, args, want, pools, slots, cu = _delta_case(H, Hk, D, V, K, lens, dtype, strong)
    B, dims = len(lens), (H, Hk, D, V)
    tol = dict(atol=4e-6 * float(want.abs().max()) + 1e-7, rtol=0)
    conv, state = pools()
    track = lens[0] // 2 + 1                                             # a checkpoint inside the first sequence
    o = native.delta_scan(proj, *args, conv, state, slots, *dims, cu=_i32(cu), prefix=_i32([0] * B),
                          track_len=_i32([track] + [0] * (B - 1)), track_slot=_i32([1] + [0] * (B - 1)), channel_a=a)
    assert torch.allclose(o.cpu().double(), want, **tol)
    # the same in portions, decode steps among them; first and last states and windows agree
    conv2, state2 = pools()
    at, got, step, sizes = [0] * B, torch.empty_like(o), 0, [2, 1, 3, 5, 17, 1, 1, 31]
    while any(at[b] < lens[b] for b in range(B)):
        m = [min(sizes[(step + b) % len(sizes)], lens[b] - at[b]) for b in range(B)]
        rows = torch.tensor(np.concatenate([np.arange(cu[b] + at[b], cu[b] + at[b] + m[b]) for b in range(B)]).astype(int),
                            device="cuda")
        ragged = {} if all(x == 1 for x in m) and all(at) else dict(
            cu=_i32(np.concatenate([[0], np.cumsum(m)])), prefix=_i32(at), lens=np.asarray(m) if step % 2 else None)
        got[rows] = native.delta_scan(proj[rows], *args, conv2, state2, slots, *dims, channel_a=a[rows], **ragged)
        at, step = [x + y for x, y in zip(at, m)], step + 1
        if at[0] == track:
            assert torch.allclose(state[1], state2[slots[0]], atol=1e-5) and torch.equal(conv[1], conv2[slots[0]])
    assert torch.allclose(got.cpu().double(), want, **tol)
    assert torch.allclose(state[slots], state2[slots], atol=1e-5) and torch.equal(conv[slots], conv2[slots])
    # decode, all requests one token at a time (equal lengths), over slots that held other states
    conv3, state3 = pools()
    first = torch.tensor(cu[:-1], device="cuda")
    for t in range(min(lens)):
        ragged = dict(cu=_i32(range(B + 1)), prefix=_i32([0] * B)) if t == 0 else {}
        r = native.delta_scan(proj[first + t], *args, conv3, state3, slots, *dims, channel_a=a[first + t], **ragged)
        assert torch.allclose(r.cpu().double(), want[cu[:-1] + t], **tol)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,V", [(3, 128), (2, 200), (5, 9)])
def test_sigmoid_gate_of_the_read_out(native, H, V, dtype):
    g = torch.Generator().manual_seed(V)
    o, w = torch.randn(6, H, V, generator=g), torch.randn(V, generator=g)
    wide = (torch.randn(6, H * V + 8, generator=g) * 3).to(dtype)
    want = oracle.rms(o.double(), 1e-4) * w.double() * torch.sigmoid(wide[:, :H * V].double()).view(6, H, V)
    got = native.delta_gate(o.cuda(), wide.cuda()[:, :H * V], w.cuda(), 1e-4, "sigmoid").cpu().double()
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(got, want.reshape(6, -1), atol=tol, rtol=tol)


# ------------------------------------------------------------------ windowed attention
def _pages(lens, P, seed):
    """Pages in shuffled order and the page table (row b + 1 belongs to request b)."""
    g = torch.Generator().manual_seed(seed)
    n = [-(-x // P) for x in lens]
    order = torch.randperm(sum(n), generator=g) + 1
    table, o = torch.zeros(len(lens) + 1, max(n) + 1, dtype=torch.int32), 0
    for b, m in enumerate(n):
        table[b + 1, :m] = order[o:o + m]
        o += m
    return table, sum(n) + 1


def _slots(table, b, n, P):
    t = np.arange(n)
    return table[b + 1].numpy()[t // P] * P + t % P


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("D,V,H,G", [(64, 64, 4, 2), (48, 40, 6, 1), (10, 7, 3, 3), (136, 72, 2, 1)])
def test_queries_and_cache_rows(native, D, V, H, G, dtype):
    g = torch.Generator().manual_seed(D)
    T, P, up = 9, 16, lambda n: -(-n // 8) * 8
    q0, k0, v0 = 8, 8 + up(H * D), 8 + up(H * D) + up(G * D)
    proj = (torch.randn(T, v0 + up(G * V), generator=g) * 3).to(dtype)
    loc = torch.randperm(4 * P, generator=g)[:T].int()
    cache = torch.full((4, G, P, up(D) + up(V)), 7.0, dtype=dtype)
    got = cache.cuda()
    q = native.attn_prep(proj.cuda(), q0, k0, v0, H, G, D, V, 1e-4, True, loc.cuda(), got)
    part = lambda o, n, d: proj[:, o:o + n * d].double().view(T, n, d)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(q[..., :D].cpu().double(), oracle.rms(part(q0, H, D), 1e-4), atol=tol, rtol=tol)
    assert (q[..., D:] == 0).all()
    page, off = (loc // P).long(), (loc % P).long()
    rows = got.cpu()[page, :, off]
    assert torch.allclose(rows[..., :D].double(), oracle.rms(part(k0, G, D), 1e-4), atol=tol, rtol=tol)
    assert torch.equal(rows[..., up(D):up(D) + V], part(v0, G, V).to(dtype))
    assert (rows[..., D:up(D)] == 0).all() and (rows[..., up(D) + V:] == 0).all()
    untouched = torch.ones(4, P, dtype=torch.bool)
    untouched[page, off] = False
    assert (got.cpu().transpose(1, 2)[untouched] == 7).all()
    before = got.clone()                                 # a reader of another layer's keys writes nothing
    native.attn_prep(proj.cuda(), q0, -1, -1, H, G, D, V, 1e-4, False, loc.cuda(), got)
    assert torch.equal(before, got)


WINDOWS = [(0, 0), (1, 0), (1, 1), (17, 0), (63, 3), (64, 64), (65, 70), (100, 1), (128, 130), (1000, 5)]
SIZES = [(64, 64, 4, 2), (48, 40, 6, 1), (10, 7, 3, 3), (136, 72, 2, 1), (200, 200, 17, 1), (96, 128, 8, 2), (24, 256, 33, 1)]


def _window_case(D, V, H, G, lens, P, dtype, seed, gain=1.5):
    g = torch.Generator().manual_seed(seed)
    up = lambda n: -(-n // 8) * 8
    table, pages = _pages(lens, P, seed)
    cache = torch.zeros(pages, G, P, up(D) + up(V))
    cache[..., :D] = torch.randn(pages, G, P, D, generator=g)
    cache[..., up(D):up(D) + V] = torch.randn(pages, G, P, V, generator=g)
    cache = cache.to(dtype)

    def rows(b):
        kv = cache[table[b + 1, :-(-lens[b] // P)].long()].transpose(1, 2).flatten(0, 1)[:lens[b]].double()
        return kv[..., :D], kv[..., up(D):up(D) + V]

    def queries(n):
        q = torch.zeros(n, H, up(D))
        q[..., :D] = torch.randn(n, H, D, generator=g) * gain
        return q.to(dtype), (torch.randn(n, H + 8, generator=g) * 2).to(dtype)[:, 3:3 + H]
    return table, cache, rows, queries


def _attend(q, gate, k, v, pos, scale, window, keep):
    """Queries `[n, H, D]` at positions `pos`."""
    own = [h // (q.shape[1] // k.shape[1]) for h in range(q.shape[1])]
    see = oracle.visible(k.shape[0], window or None, keep)[pos]
    s = torch.einsum("nhd,shd->hns", q, k[:, own]) * scale
    w = torch.softmax(s.masked_fill(~see, -torch.inf), -1)
    return torch.einsum("hns,shd->nhd", w, v[:, own]) * torch.sigmoid(gate)[..., None]


@pytest.mark.parametrize("P", [16, 64, 128])
@pytest.mark.parametrize("D,V,H,G", SIZES)
def test_single_queries_of_any_size_and_window(native, D, V, H, G, P):
    """bf16 on the tensor cores and fp32 on the CUDA cores, one split of the keys and several."""
    lens = [1, 2, P - 1, P, P + 1, 3 * P + 5, 300]
    for dtype in (torch.bfloat16, torch.float32):
        table, cache, rows, queries = _window_case(D, V, H, G, lens, P, dtype, D + P)
        q, gate = queries(len(lens))
        for window, keep in WINDOWS[P // 64::2]:
            want = torch.cat([_attend(q[b:b + 1, :, :D].double(), gate[b:b + 1].double(), *rows(b), [n - 1], 0.11, window, keep)
                              for b, n in enumerate(lens)])
            args = (q.cuda(), gate.cuda(), cache.cuda(), table.cuda(), _i32(range(1, len(lens) + 1)), _i32(lens), D, V, P,
                    0.11, window, keep)
            got = [native.window_attn_any(*args)]
            tol = 1e-5
            if dtype == torch.bfloat16:
                assert native.window_decode_supported(args[0], args[2], D, V, P)
                got += [native.window_decode(*args, num_splits=n) for n in (None, 1, 3)]
                tol = 2.0 ** -8                                          # half a step of the bf16 result
            for o in got:
                assert ((o.cpu().double() - want).abs() <= tol * want.abs() + 2e-5 * want.abs().max()).all(), (window, keep)


@pytest.mark.parametrize("D,V,H,G,P,lens,pres,gain", [
    (64, 64, 2, 1, 64, [256], [0], 1), (64, 40, 2, 2, 16, [32], [0], 1), (40, 72, 3, 1, 64, [300, 77, 600], [0, 5, 500], 1),
    (128, 128, 2, 1, 128, [513, 33], [64, 0], 1), (96, 80, 2, 1, 64, [129], [1], 6), (192, 128, 4, 2, 64, [700], [0], 4),
    (10, 7, 3, 3, 32, [400], [13], 1), (256, 64, 2, 1, 64, [300], [130], 2), (128, 128, 8, 2, 64, [90, 256, 257], [37, 63, 64], 3)])
def test_prefill_tiles_of_any_window(native, D, V, H, G, P, lens, pres, gain):
    ctx = [a + b for a, b in zip(lens, pres)]
    table, cache, rows, queries = _window_case(D, V, H, G, ctx, P, torch.bfloat16, D + V, gain)
    q, gate = queries(sum(lens))
    qs = np.concatenate([[0], np.cumsum(lens)])
    plan = SimpleNamespace(q_start=_i32(qs[:-1]), q_len=_i32(lens), prefix=_i32(pres), rows=_i32(range(1, len(lens) + 1)),
                           long=len(lens), num_tiles=sum((n + 255) // 256 for n in lens))
    qc, gc, cc, tc = q.cuda(), gate.cuda(), cache.cuda(), table.cuda()
    assert native.window_extend_supported(qc, cc, D, V)
    for window, keep in WINDOWS + [(300, 200), (7, 300)]:
        out = torch.full((sum(lens), H, V), torch.nan, device="cuda", dtype=torch.bfloat16)
        native.window_extend(qc, gc, cc, tc, plan, out, D, V, D ** -0.5, window, keep)
        for b in range(len(lens)):
            s = slice(qs[b], qs[b + 1])
            want = _attend(q[s, :, :D].double(), gate[s].double(), *rows(b), np.arange(pres[b], ctx[b]), D ** -0.5, window, keep)
            diff = (out[s].cpu().double() - want).abs()
            assert (diff <= 2.0 ** -8 * want.abs() + 3e-5 * want.abs().max()).all(), (b, window, keep)


# ------------------------------------------------------------------ models and schedules
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_whole_prompts(models, name, dtype):
    path, cfg, w = models[name]
    reqs = {n: cases.tokens(n, cfg["vocab"], n) for n in (1, 2, 31, 33, 150)}
    cases.check(path, cfg, w, dtype, "cuda", reqs, [[(n, n)] for n in reqs], 192)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["plain", "mixed", "odd"])
def test_portions_token_by_token_and_long_decoding(models, name, dtype):
    path, cfg, w = models[name]
    ids = cases.tokens(200, cfg["vocab"], 1)
    want = {"a": cases.expectation(ids, w, cfg)}
    for sizes in ([1], [2], [40, 1, 1, 2, 33], [128, 1], [63, 1, 1, 100]):
        cases.check(path, cfg, w, dtype, "cuda", {"a": ids}, [[("a", n)] for n in cases.cut(200, sizes)], 256, want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype):
    path, cfg, w = models[name]
    lens = [140, 3, 165, 17, 70, 64, 1, 90]
    reqs = {i: cases.tokens(n, cfg["vocab"], 50 + i) for i, n in enumerate(lens)}
    sizes = [[37, 1, 1, 2], [1], [132, 1], [2], [16, 1, 50], [63, 1], [1], [3, 34, 1]]
    steps = cases.interleave(reqs, {i: cases.cut(n, sizes[i]) for i, n in enumerate(lens)})
    cases.check(path, cfg, w, dtype, "cuda", reqs, steps, 512)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("distance", [0, 1, 63, 64, 65, 98, 99, 100, 101, 128, 290, 295, 296, 297])
def test_one_key_decides_inside_the_window_and_among_the_first(tmp_path, distance, dtype):
    cfg, w = needle_model(100, 4)
    ids = needle_prompt(distance, 300)
    want = {"a": cases.expectation(ids, w, cfg)}
    path = cases.write(str(tmp_path), cfg, w)
    for steps in ([[("a", 300)]], [[("a", 299)], [("a", 1)]], [[("a", n)] for n in cases.cut(300, [60, 2, 131, 1])]):
        cases.check(path, cfg, w, dtype, "cuda", {"a": ids}, steps, 320, want)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_past_the_window(tmp_path, dtype):
    cfg, w = first_token_model()
    ids = cases.tokens(180, cfg["vocab"], 2)
    path = cases.write(str(tmp_path), cfg, w)
    want = {"a": cases.expectation(ids, w, cfg)}
    for first in (2, 70):
        steps = [[("a", first)]] + [[("a", 1)]] * (180 - first)
        cases.check(path, cfg, w, dtype, "cuda", {"a": ids}, steps, 192, want)


# ------------------------------------------------------------------ engine
def _engine(path, dtype, **kw):
    from sglang_jax_b200 import Engine
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    return Engine(model_path=path, device="cuda", dtype=dtype, skip_tokenizer_init=True, enable_single_process=True,
                  **{"page_size": 64, "max_total_tokens": 4096, "max_running_requests": 8, "cuda_graph_max_bs": 8, **kw})


def _near_greedy(ids, w, cfg, slack):
    """Every generated token is the oracle's best one, or as good within `slack` of the logits' spread."""
    prompt, out = ids
    logits = oracle.forward(prompt + out, w, cfg)[len(prompt) - 1:-1]
    best = logits.max(-1).values - logits[torch.arange(len(out)), torch.tensor(out)]
    return bool((best <= slack * logits.std()).all())


@pytest.mark.parametrize("kw", [dict(), dict(disable_cuda_graph=True), dict(chunked_prefill_size=64, enable_mixed_chunk=True)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_engine(models, dtype, kw):
    path, cfg, w = models["plain"]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (29, 7, 170, 64, 65)]
    eng = _engine(path, dtype, **kw)
    try:
        got = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 12, "temperature": 0, "ignore_eos": True})
        for p, o in zip(prompts, got):
            assert len(o["output_ids"]) == 12
            assert _near_greedy((p, o["output_ids"]), w, cfg, 1e-4 if dtype == "float32" else 0.3)
        info = eng.get_server_info()["internal_states"][0]
        assert (info["cuda_graph_replays"] > 5) != bool(kw.get("disable_cuda_graph")) and info["cuda_graph_recaptures"] == 0
        eng.scheduler.check_memory()
    finally:
        eng.shutdown()


def test_shared_prefixes_restart_from_state_checkpoints(models):
    path, cfg, w = models["mixed"]
    base = cases.tokens(150, cfg["vocab"], 1)
    eng = _engine(path, "float32", recurrent_snapshot_slots=16)
    try:
        sp = {"max_new_tokens": 4, "temperature": 0, "ignore_eos": True}
        eng.generate(input_ids=base, sampling_params=sp)
        again = base[:140] + cases.tokens(20, cfg["vocab"], 2)
        out = eng.generate(input_ids=again, sampling_params=sp)
        assert out["meta_info"]["cached_tokens"] == 128
        assert _near_greedy((again, out["output_ids"]), w, cfg, 1e-4)
    finally:
        eng.shutdown()
