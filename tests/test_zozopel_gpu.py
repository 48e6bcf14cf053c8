"""Zozopel on the GPU: its kernels against plain double-precision statements, and schedules, caches and generation of
whole models against the oracle, in bf16 and in fp32."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import zozopel_cases as cases
import zozopel_oracle as oracle
from test_zozopel_cpu import needle_model, needle_prompt

pytestmark = pytest.mark.gpu
DTYPES = ["bfloat16", "float32"]


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
        out[name] = (cases.write_checkpoint(str(tmp_path_factory.mktemp(name)), cfg, w), cfg, w)
    return out


def _i32(x):
    return torch.tensor(np.asarray(x), dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------ kernels
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("W", [24, 51, 1000, 4096])
def test_stream_kernels(native, dtype, W):
    g = torch.Generator().manual_seed(W)
    T, eps = 7, 1e-5
    rnd = lambda *s: torch.randn(*s, generator=g)
    table, ids = rnd(9, W).to(dtype), torch.tensor([3, 0, 8, 3, 7, 1, 2], dtype=torch.int32)
    x, h = native.embed_scaled(ids.cuda(), table.cuda(), 0.37)
    assert torch.allclose(x.cpu(), table[ids.long()].float() * 0.37, rtol=1e-6) and h.dtype == dtype
    y, s = (rnd(T, W) * 3).to(dtype), rnd(W)
    want = x.cpu().double() + oracle.rms(y.double(), eps) * s.double()
    h = native.postnorm_add(y.cuda(), x, s.cuda(), eps)
    assert torch.allclose(x.cpu().double(), want, atol=2e-6, rtol=2e-6)
    assert torch.equal(h.cpu(), x.cpu().to(dtype))
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    n = native.rmsnorm_stream(x, s.cuda(), eps, dtype).cpu()
    assert torch.allclose(n.double(), oracle.rms(want, eps) * s.double(), atol=tol, rtol=tol)
    ab = (rnd(T, 2 * W) * 4).to(dtype)
    a, b = ab.double().split(W, -1)
    assert torch.allclose(native.gelu_tanh_and_mul(ab.cuda()).cpu().double(), oracle.gelu_tanh(a) * b, atol=tol, rtol=tol)
    gate = ab[:, 3:3 + W]
    got = native.sigmoid_gate(y.cuda(), ab.cuda()[:, 3:3 + W]).cpu().double()
    assert torch.allclose(got, y.double() * torch.sigmoid(gate.double()), atol=tol, rtol=tol)


def _delta_case(H, Hk, D, V, K, lens, dtype, seed=0):
    """Inputs of `delta_scan`, the oracle's read-outs, and freshly dirtied pools."""
    g = torch.Generator().manual_seed(seed)
    B, T, ch, pad = len(lens), sum(lens), 2 * Hk * D + H * V, (H + 7) // 8 * 8
    go, bo, ao = ch, ch + H * V, ch + H * V + pad
    proj = torch.randn(T, ao + pad, generator=g).to(dtype)
    conv = (torch.randn(ch, K, generator=g) * 0.5).to(dtype)
    a_log, dt = torch.randn(H, generator=g) * 0.5 - 2, torch.randn(H, generator=g) * 0.3
    cu = np.concatenate([[0], np.cumsum(lens)])
    want = []
    for b in range(B):
        x = proj[cu[b]:cu[b + 1]].double()
        y = oracle.silu(oracle.causal_conv(x[:, :ch], conv.double()))
        own = [i // (H // Hk) for i in range(H)]
        q = oracle.unit(y[:, :Hk * D].view(-1, Hk, D))[:, own] * D ** -0.5
        k = oracle.unit(y[:, Hk * D:2 * Hk * D].view(-1, Hk, D))[:, own]
        decay = torch.exp(-torch.exp(a_log.double()) * oracle.softplus(x[:, ao:ao + H] + dt.double()))
        want.append(oracle.delta_recurrence(q, k, y[:, 2 * Hk * D:].view(-1, H, V), decay, torch.sigmoid(x[:, bo:bo + H])))
    pools = lambda: (torch.randn(B + 3, ch, K - 1, generator=g).to(dtype).cuda(), torch.randn(B + 3, H, D, V, generator=g).cuda())
    args = (go, bo, ao, conv.cuda(), a_log.cuda(), dt.cuda())
    slots = torch.tensor([B + 2 - b for b in range(B)], device="cuda")
    return proj.cuda(), args, torch.cat(want), pools, slots, cu


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,Hk,D,V,K,lens", [
    (6, 2, 64, 48, 4, [70, 1, 33]), (6, 3, 24, 40, 3, [50, 9, 4]), (2, 1, 128, 128, 4, [130]), (3, 3, 100, 36, 2, [41, 2]),
    (2, 1, 16, 200, 6, [23]), (2, 2, 256, 64, 1, [20]), (3, 1, 13, 9, 4, [18, 5]), (32, 16, 128, 128, 4, [9] * 40),
    (16, 4, 32, 32, 4, [6] * 150)])
def test_delta_scan_whole_in_portions_and_token_by_token(native, H, Hk, D, V, K, lens, dtype):
    proj, args, want, pools, slots, cu = _delta_case(H, Hk, D, V, K, lens, dtype)
    B, dims = len(lens), (H, Hk, D, V)
    tol = dict(atol=2e-6 * float(want.abs().max()) + 1e-7, rtol=0)
    conv, state = pools()
    track = lens[0] // 2 + 1                                             # a checkpoint inside the first sequence
    o = native.delta_scan(proj, *args, conv, state, slots, *dims, cu=_i32(cu), prefix=_i32([0] * B),
                          track_len=_i32([track] + [0] * (B - 1)), track_slot=_i32([1] + [0] * (B - 1)))
    assert torch.allclose(o.cpu().double(), want, **tol)
    # the same in portions, decode steps among them; first and last states and windows agree
    conv2, state2 = pools()
    at, got, step, sizes = [0] * B, torch.empty_like(o), 0, [2, 1, 3, 5, 17, 1, 1, 31]
    while any(at[b] < lens[b] for b in range(B)):
        m = [min(sizes[(step + b) % len(sizes)], lens[b] - at[b]) for b in range(B)]
        rows = torch.tensor(np.concatenate([np.arange(cu[b] + at[b], cu[b] + at[b] + m[b]) for b in range(B)]).astype(int),
                            device="cuda")
        ragged = {} if all(x == 1 for x in m) and all(at) else dict(cu=_i32(np.concatenate([[0], np.cumsum(m)])), prefix=_i32(at))
        got[rows] = native.delta_scan(proj[rows], *args, conv2, state2, slots, *dims, **ragged)
        at, step = [a + x for a, x in zip(at, m)], step + 1
        if at[0] == track:
            assert torch.allclose(state[1], state2[slots[0]], atol=1e-5) and torch.equal(conv[1], conv2[slots[0]])
    assert torch.allclose(got.cpu().double(), want, **tol)
    assert torch.allclose(state[slots], state2[slots], atol=1e-5) and torch.equal(conv[slots], conv2[slots])
    # decode, all requests one token at a time (equal lengths), over slots that held other states
    n = min(lens)
    conv3, state3 = pools()
    first = torch.tensor(cu[:-1], device="cuda")
    for t in range(n):
        ragged = dict(cu=_i32(range(B + 1)), prefix=_i32([0] * B)) if t == 0 else {}
        r = native.delta_scan(proj[first + t], *args, conv3, state3, slots, *dims, **ragged)
        assert torch.allclose(r.cpu().double(), want[cu[:-1] + t], **tol)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,V", [(3, 128), (2, 200), (5, 9)])
def test_delta_gate(native, H, V, dtype):
    g = torch.Generator().manual_seed(V)
    o, w = torch.randn(6, H, V, generator=g), torch.randn(V, generator=g)
    wide = (torch.randn(6, H * V + 8, generator=g) * 3).to(dtype)
    want = oracle.rms(o.double(), 1e-4) * w.double() * oracle.silu(wide[:, :H * V].double()).view(6, H, V)
    got = native.delta_gate(o.cuda(), wide.cuda()[:, :H * V], w.cuda(), 1e-4).cpu().double()
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert got.shape == (6, H * V) and torch.allclose(got, want.reshape(6, -1), atol=tol, rtol=tol)


def _latent_cache(lens, R, rot, P, dtype, seed):
    """Cache pages in shuffled order, the page table (row b + 1 belongs to request b), and each request's rows."""
    g = torch.Generator().manual_seed(seed)
    width = -(-(R + rot) // 8) * 8
    pages = [-(-n // P) for n in lens]
    order = torch.randperm(sum(pages), generator=g) + 1
    cache = torch.randn(sum(pages) + 1, P, width, generator=g).to(dtype)
    table = torch.zeros(len(lens) + 1, max(pages) + 1, dtype=torch.int32)
    rows, o = [], 0
    for b, n in enumerate(pages):
        table[b + 1, :n] = order[o:o + n]
        rows.append(cache[order[o:o + n]].reshape(-1, width)[:lens[b], :R + rot].double())
        o += n
    return cache.cuda(), table.cuda(), rows


@pytest.mark.parametrize("P", [16, 64, 128])
@pytest.mark.parametrize("R,rot,H", [(512, 64, 16), (64, 32, 6), (128, 24, 17), (48, 8, 3), (320, 64, 4), (21, 6, 3),
                                     (256, 16, 33)])
def test_absorbed_latent_attention_of_any_size(native, R, rot, H, P):
    """bf16 on the tensor cores and fp32 on the CUDA cores; in fp32, and with `exact` weights, far beyond bf16 steps."""
    lens = [1, P - 1, P, P + 1, 3 * P + 5, 500]
    g = torch.Generator().manual_seed(R + P)
    q = torch.randn(len(lens), H, R + rot + 2, generator=g) * 1.5
    for dtype in (torch.bfloat16, torch.float32):
        cache, table, rows = _latent_cache(lens, R, rot, P, dtype, R)
        qd = q.to(dtype)
        ql, qp = qd[..., :R].contiguous().cuda(), qd.cuda()[..., R:R + rot]          # the rotary part is a strided view
        want = []
        for b, k in enumerate(rows):
            s = (qd[b, :, :R].double() @ k[:, :R].T + qd[b, :, R:R + rot].double() @ k[:, R:].T) * 0.11
            want.append(torch.softmax(s, -1) @ k[:, :R])
        want = torch.stack(want)
        args = (table, _i32(range(1, len(lens) + 1)), _i32(lens))
        if dtype == torch.float32:
            got = [native.latent_attn_any(ql, qp, cache, *args, P, 0.11)]
            tol = 1e-5
        else:
            assert native.mla_decode_supported(ql, qp, cache, R, P)
            got = [native.mla_decode(ql, qp, cache, *args, P, 0.11, max_seq_len=500, num_splits=n, exact=True) for n in (1, 3)]
            got.append(native.latent_attn_any(ql, qp, cache, *args, P, 0.11))
            tol = 2.0 ** -8                                                          # half a step of the bf16 result
        for o in got:
            assert ((o.cpu().double() - want).abs() <= tol * want.abs() + 2e-5 * want.abs().max()).all()


@pytest.mark.parametrize("H,dim,rot,v,lens,pres,gain", [
    (2, 64, 40, 72, [256], [0], 1), (2, 64, 40, 72, [32], [0], 1), (3, 64, 40, 72, [300, 77, 1000], [0, 5, 900], 1),
    (2, 128, 64, 128, [513, 33], [64, 0], 1), (2, 96, 16, 80, [129], [1], 6), (4, 128, 64, 128, [1024], [0], 8),
    (1, 40, 8, 24, [700], [13], 1), (2, 192, 64, 128, [300], [10], 3)])
def test_expanded_latent_prefill(native, H, dim, rot, v, lens, pres, gain):
    g = torch.Generator(device="cuda").manual_seed(dim + v)
    rnd = lambda *s: torch.randn(*s, generator=g, device="cuda").bfloat16()
    T, ctx = sum(lens), [a + b for a, b in zip(lens, pres)]
    q = (rnd(T, H * (dim + rot) + 24) * gain)[:, :H * (dim + rot)].unflatten(-1, (H, dim + rot))
    kv, pe = rnd(sum(ctx), H * (dim + v)), rnd(sum(ctx), rot)
    out = torch.zeros(T, H, v, device="cuda", dtype=torch.bfloat16)
    qs, cs = np.concatenate([[0], np.cumsum(lens)]), np.concatenate([[0], np.cumsum(ctx)])
    plan = SimpleNamespace(q_start=_i32(qs[:-1]), q_len=_i32(lens), prefix=_i32(pres), long=len(lens),
                           context=lambda window: SimpleNamespace(start=_i32(cs), skip=None),
                           num_tiles=sum((n + 255) // 256 for n in lens))
    assert native.latent_extend_supported(q, dim, rot, v, 64)
    native.latent_extend(q, kv, pe, out, plan, dim, v, (dim + rot) ** -0.5)
    for b in range(len(lens)):
        k = kv[cs[b]:cs[b + 1]].view(-1, H, dim + v).double()
        kk = torch.cat([k[..., :dim], pe[cs[b]:cs[b + 1], None].double().expand(-1, H, rot)], -1)
        s = torch.einsum("ihd,jhd->hij", q[qs[b]:qs[b + 1]].double(), kk) * (dim + rot) ** -0.5
        i = torch.arange(lens[b], device="cuda")[:, None] + pres[b]
        w = torch.softmax(s.masked_fill(torch.arange(ctx[b], device="cuda")[None] > i, -torch.inf), -1)
        want = torch.einsum("hij,jhd->ihd", w, k[..., dim:])
        diff = (out[qs[b]:qs[b + 1]].double() - want).abs()
        assert (diff <= 2.0 ** -8 * want.abs() + 2e-5 * want.abs().max()).all()      # weights keep more than bf16's bits


def test_gather_of_contexts(native):
    lens = [5, 64, 130]
    cache, table, rows = _latent_cache(lens, 40, 8, 64, torch.bfloat16, 1)
    start = np.concatenate([[0], np.cumsum(lens)])
    lat, pe = native.latent_gather(cache, table, _i32([1, 2, 3]), _i32(start), sum(lens), 40, 8, 64)
    assert torch.equal(torch.cat([lat, pe], -1).cpu().double(), torch.cat(rows))


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
@pytest.mark.parametrize("distance", [1, 63, 64, 65, 127, 128, 255, 256, 299])
def test_one_far_key_decides(tmp_path, distance, dtype):
    cfg, w = needle_model()
    ids = needle_prompt(distance, 300)
    want = {"a": cases.expectation(ids, w, cfg)}
    path = cases.write_checkpoint(str(tmp_path), cfg, w)
    for steps in ([[("a", 300)]], [[("a", 299)], [("a", 1)]], [[("a", n)] for n in cases.cut(300, [60, 2, 131, 1])]):
        cases.check(path, cfg, w, dtype, "cuda", {"a": ids}, steps, 320, want)


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
            assert _near_greedy((p, o["output_ids"]), w, cfg, 1e-4 if dtype == "float32" else 0.15)
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


def test_trace_runner_as_a_program(models, tmp_path):
    import json
    import os
    import subprocess
    path, cfg, w = models["plain"]
    ids = cases.tokens(40, cfg["vocab"], 8)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[33:34], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": ids, "want": [39]}, {"id": "x", "tokens": ids[34:35], "want": [0]}],
              "end": ["x", "y"]}]
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([exe, "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert sorted(f for f in os.listdir(tmp_path)) == ["0.f32", "2.f32"]
    want = oracle.forward(ids, w, cfg)
    for f, rows in (("0.f32", [0, 32]), ("2.f32", [39, 34])):
        got = torch.from_numpy(np.fromfile(tmp_path / f, "<f4").reshape(2, -1)).double()
        assert float(cases.error(got, want[rows]).max()) < cases.LIMIT["float32"]
