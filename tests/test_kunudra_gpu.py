"""Kunudra on the GPU: its kernels against plain double-precision statements, and schedules, caches and generation of whole
models against the oracle, in bf16 and in fp32."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import kunudra_cases as cases
import kunudra_oracle as oracle
from test_kunudra_cpu import needle_model, needle_prompt, sink_model

pytestmark = pytest.mark.gpu
DTYPES = ["bfloat16", "float32"]
BOTH = [torch.bfloat16, torch.float32]


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


up8 = lambda n: -(-n // 8) * 8


# ------------------------------------------------------------------ stream kernels
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("W", [24, 51, 1000, 4096])
def test_norm_behind_the_sum(native, dtype, W):
    g = torch.Generator().manual_seed(W)
    T, E, k, eps = 7, 5, 3, 1e-5
    rnd = lambda *s: torch.randn(*s, generator=g)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    y, s, w, nw = (rnd(T, W) * 3).to(dtype), rnd(W), rnd(W), rnd(W)
    e, weights, gate = rnd(20, W).to(dtype), torch.rand(T, k, generator=g), torch.rand(T, generator=g)
    ids = torch.randint(0, E + 3, (T, k), generator=g, dtype=torch.int32)
    rows = torch.where(ids < E, torch.randint(0, 20, (T, k), generator=g), -1).int()
    own = (weights.double() * (ids >= E)).sum(1, keepdim=True)
    routed = ((weights * (ids < E)).unsqueeze(-1).double() * e[rows.clamp_min(0).long()].double()).sum(1)
    for with_experts in (False, True):
        for then in (False, True):
            x = rnd(T, W)
            add = y.double()
            kw = dict(next_weight=nw.cuda(), next_eps=1e-3) if then else {}
            if with_experts:
                add = add * gate.double()[:, None] + routed + own * x.double()
                kw.update(y_gate=gate.cuda(), expert_out=e.cuda(), weights=weights.cuda(), pair_row=rows.cuda(), ids=ids.cuda(),
                          experts=E)
            want = oracle.norm_sum(x.double(), add, s.double(), 0.8, w.double() - 1, eps)
            xc = x.cuda()
            h = native.sum_norm(y.cuda(), xc, 0.8, s.cuda(), w.cuda(), eps, **kw)
            assert torch.allclose(xc.cpu().double(), want, atol=3e-6, rtol=3e-6)
            if then:
                want = oracle.rms(want, 1e-3) * nw.double()
                assert torch.allclose(h.cpu().double(), want, atol=tol, rtol=tol) and h.dtype == dtype
            else:
                assert torch.equal(h, xc.to(dtype))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("W,buckets,mp,mc", [(24, 11, 5, 3), (51, 1, 1, 1), (1000, 30011, 1_000_003, 999_983)])
def test_token_pairs(native, dtype, W, buckets, mp, mc):
    """Portions of unequal requests, single tokens among them, then decode steps; predecessors come from the step or the slot."""
    g = torch.Generator().manual_seed(W)
    V, P, lens = 90, 16, [40, 1, 23, 70]
    table, pairs = torch.randn(V, W, generator=g).to(dtype), torch.randn(buckets + 1, W, generator=g).to(dtype)
    seqs = [cases.tokens(n, V, n) for n in lens]
    pt = torch.zeros(6, 5, dtype=torch.int32)
    pt[1:5] = torch.randperm(20, generator=g).view(4, 5) + 1
    slots = torch.full((21 * P,), V - 1, dtype=torch.int32, device="cuda")
    at, step = [0] * 4, 0
    sizes = [[13, 1, 2], [1], [20, 1, 1, 1], [1, 30, 5, 2]]
    while any(a < n for a, n in zip(at, lens)):
        m = [min(sizes[b][step % len(sizes[b])], lens[b] - at[b]) for b in range(4)]
        live = [b for b in range(4) if m[b]]
        pos = np.concatenate([np.arange(at[b], at[b] + m[b]) for b in live])
        row = np.concatenate([np.full(m[b], b + 1) for b in live])
        ids = [t for b in live for t in seqs[b][at[b]:at[b] + m[b]]]
        loc = pt[row, pos // P].numpy() * P + pos % P
        decode = all(at[b] and m[b] == 1 for b in live)
        cu = None if decode else _i32(np.concatenate([[0], np.cumsum([m[b] for b in live])]))
        x, h = native.embed_pair(_i32(ids), table.cuda(), pairs.cuda(), mp, mc, slots, _i32(pos), _i32(loc), cu,
                                 _i32([b + 1 for b in live]), pt.cuda(), P)
        rows = [oracle.pair_rows(seqs[b], buckets, mp, mc)[i] for b, i in zip(row - 1, pos)]
        assert torch.equal(x.cpu(), table[ids].float() + pairs[rows].float()) and torch.equal(h, x.to(dtype))
        at, step = [a + n for a, n in zip(at, m)], step + 1


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("F", [16, 37, 96, 1000])
def test_gated_activation(native, dtype, F):
    from sglang_jax_b200 import ops
    x = (torch.randn(5, 2 * F, generator=torch.Generator().manual_seed(F)) * 4).to(dtype)
    want = oracle.silu(x[:, :F].double()) * x[:, F:].double()
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(ops.swiglu(x.cuda()).cpu().double(), want, atol=tol, rtol=tol)


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T", [1, 5, 300])
@pytest.mark.parametrize("E,k,K", [(1, 1, 64), (12, 4, 192), (65, 8, 129), (500, 16, 40)])
def test_routing_by_score(native, dtype, T, E, k, K):
    from sglang_jax_b200.ops import moe_native
    g = torch.Generator().manual_seed(E + T)
    x, w = torch.randn(T, K, generator=g).to(dtype), (torch.randn(E + 4, K, generator=g) * 2 * K ** -0.5).to(dtype)
    c = torch.randn(E, generator=g) * 0.05
    for gated in (False, True):
        s = torch.softmax(x.double() @ w[:E].double().T, -1)
        best = torch.topk(s + c.double(), k, -1)
        weights, ids, gate = moe_native.route_by_score(x.cuda(), (w if gated else w[:E]).cuda(), c.cuda(), k, 1.6, E, gated)
        chosen = ids.cpu().long()
        assert torch.allclose((s + c.double()).gather(1, chosen), best.values, atol=2e-6)
        assert torch.allclose(weights.cpu().double(), 1.6 * s.gather(1, chosen), atol=2e-6)
        assert all(len(set(r)) == k for r in ids.tolist())
        assert (gate is not None) == gated
        if gated:
            assert torch.allclose(gate.cpu().double(), torch.sigmoid(x.double() @ w[E].double()), atol=2e-6)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T", [1, 9, 400])
@pytest.mark.parametrize("W,E,identity,k,ff,shared", [(64, 6, 3, 2, 48, 24), (51, 3, 2, 4, 37, 0), (128, 1, 0, 1, 40, 16)])
def test_feed_forward_on_the_stream(native, dtype, T, W, E, identity, k, ff, shared):
    from sglang_jax_b200.layers.layernorm import SumNorm
    from sglang_jax_b200.layers.moe import ScoredFeedForward
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    cfg = cases.config([cases.attention(1, 1, 8, 8, 4, mlp=cases.moe(ff, E, k, identity, 1.3, shared))], W, 20)
    w = cases.random_weights(cfg, T)
    with torch.device("cuda"):
        m, norm = ScoredFeedForward(W, E, identity, k, ff, 1.3, shared, dtype), SumNorm(W, 1e-6, 0.9, dtype)
    for n, t in w.items():
        if n.startswith("l0.mlp."):
            m.load(n[7:], t)
    norm.fold()
    x = torch.randn(T, W, generator=torch.Generator().manual_seed(W)).to(dtype)
    wd = {n: t.double() for n, t in w.items()}
    want = oracle.norm_sum(x.double(), oracle.sparse_ff(x.double(), wd, "l0.mlp.", cfg["layers"][0]["mlp"]), 1.0, 0.9, torch.zeros(W), 1e-6)
    s = x.float().cuda()
    m(x.cuda(), s, norm)
    s = torch.sort(torch.softmax(x.double() @ wd["l0.mlp.router"].T, -1) + wd["l0.mlp.correction"], -1, descending=True).values, s
    clear = torch.ones(T, dtype=torch.bool) if k == E + identity else s[0][:, k - 1] - s[0][:, k] > 1e-5
    tol = 2e-5 if dtype == torch.float32 else 3e-2
    assert torch.allclose(s[1].cpu().double()[clear], want[clear], atol=tol, rtol=tol)


# ------------------------------------------------------------------ caches and queries
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("D,V,H,G", [(64, 64, 4, 2), (48, 40, 6, 1), (10, 7, 3, 3), (136, 72, 2, 1), (128, 128, 32, 8)])
def test_norms_over_whole_projections_and_mixed_values(native, D, V, H, G, dtype):
    g = torch.Generator().manual_seed(D)
    T, P = 9, 16
    q0, k0, v0 = 8, 8 + up8(H * D), 8 + up8(H * D) + up8(G * D)
    proj = (torch.randn(T, v0 + up8(G * V), generator=g) * 3).to(dtype)
    other = (torch.randn(T, 16 + G * V, generator=g) * 3).to(dtype)[:, 8:8 + G * V]
    qw, kw, share = torch.randn(H * D, generator=g), torch.randn(G * D, generator=g), torch.tensor([0.3])
    loc = torch.randperm(4 * P, generator=g)[:T].int()
    part = lambda o, n: proj[:, o:o + n].double()
    tol = 1e-5 if dtype == torch.float32 else 1.2e-2
    page, off = (loc // P).long(), (loc % P).long()
    untouched = torch.ones(4, P, dtype=torch.bool)
    untouched[page, off] = False
    for mixed in (False, True):
        for given in (False, True):                            # sums of squares of projections twice as wide
            got = torch.full((4, G, P, up8(D) + up8(V)), 7.0, dtype=dtype).cuda()
            kwargs = dict(mix=other.cuda(), share=share.cuda()) if mixed else {}
            qn, kn = (oracle.rms(part(o, n), 1e-4) for o, n in ((q0, H * D), (k0, G * D)))
            if given:
                sq = torch.stack([part(q0, H * D).pow(2).sum(-1) + 50, part(k0, G * D).pow(2).sum(-1) + 70], -1)
                kwargs.update(squares=sq.float().cuda(), totals=(2 * H * D, 2 * G * D))
                qn = part(q0, H * D) / torch.sqrt(sq[:, :1] / (2 * H * D) + 1e-4)
                kn = part(k0, G * D) / torch.sqrt(sq[:, 1:] / (2 * G * D) + 1e-4)
            q = native.attn_prep_rows(proj.cuda(), q0, k0, v0, H, G, D, V, 1e-4, qw.cuda(), kw.cuda(), loc.cuda(), got, **kwargs)
            assert torch.allclose(q[..., :D].cpu().double(), (qn * qw.double()).view(T, H, D), atol=tol, rtol=tol)
            rows = got.cpu()[page, :, off]
            assert torch.allclose(rows[..., :D].double(), (kn * kw.double()).view(T, G, D), atol=tol, rtol=tol)
            v = part(v0, G * V)
            if mixed:
                v = oracle.mix_values(v, other.double(), share.double())
            assert torch.allclose(rows[..., up8(D):up8(D) + V].double(), v.view(T, G, V), atol=tol, rtol=tol)
            assert (q[..., D:] == 0).all() and (rows[..., D:up8(D)] == 0).all() and (rows[..., up8(D) + V:] == 0).all()
            assert (got.cpu().transpose(1, 2)[untouched] == 7).all()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,dim,rot,R,Rq", [(4, 40, 16, 72, 56), (3, 10, 6, 21, 19), (2, 7, 2, 9, 5), (16, 128, 64, 512, 768)])
def test_latent_rows_and_queries_from_their_latent(native, H, dim, rot, R, Rq, dtype):
    from sglang_jax_b200.layers.embeddings import get_rope
    g = torch.Generator().manual_seed(R)
    T, P, base, at = 9, 16, 300.0, up8(Rq)
    proj = (torch.randn(T, at + up8(R + rot), generator=g) * 3).to(dtype)
    qw, cw, pos = torch.randn(Rq, generator=g), torch.randn(R, generator=g), torch.randint(0, 500, (T,), generator=g).int()
    loc = torch.randperm(4 * P, generator=g)[:T].int()
    cs = get_rope(rot, rot, 500, base, False, {"rope_type": "exact"}, dtype).cos_sin_cache.cuda()
    cache = torch.zeros(4, P, up8(R + rot), dtype=dtype, device="cuda")
    c_q = native.latent_prep(proj.cuda(), 0, at, H, dim, rot, R, cw.cuda(), 1e-4, cs, pos.cuda(), loc.cuda(), cache, qw.cuda())
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    assert torch.allclose(c_q.cpu().double(), oracle.rms(proj[:, :Rq].double(), 1e-4) * qw.double(), atol=tol, rtol=tol)
    rows = cache.cpu().flatten(0, 1)[loc.long()].double()
    assert torch.allclose(rows[:, :R], oracle.rms(proj[:, at:at + R].double(), 1e-4) * cw.double(), atol=tol, rtol=tol)
    want, turned = oracle.rotate(proj[:, at + R:at + R + rot].double(), pos, base), max(tol, 5e-4)      # (fp32 angles)
    assert torch.allclose(rows[:, R:R + rot], want, atol=turned, rtol=tol)
    q = (torch.randn(T, H * (dim + rot) + 4, generator=g) * 2).to(dtype)
    qc = q.cuda()[:, :H * (dim + rot)].unflatten(-1, (H, dim + rot))
    native.latent_rotate(qc, dim, cs, pos.cuda())
    q = q[:, :H * (dim + rot)].double().unflatten(-1, (H, dim + rot))
    want = torch.cat([q[..., :dim], oracle.rotate(q[..., dim:], pos, base)], -1)
    assert torch.allclose(qc.cpu().double(), want, atol=turned, rtol=tol)


# ------------------------------------------------------------------ attention
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


def _window_case(D, V, H, G, lens, P, dtype, seed, gain=1.5):
    g = torch.Generator().manual_seed(seed)
    table, pages = _pages(lens, P, seed)
    cache = torch.zeros(pages, G, P, up8(D) + up8(V))
    cache[..., :D] = torch.randn(pages, G, P, D, generator=g)
    cache[..., up8(D):up8(D) + V] = torch.randn(pages, G, P, V, generator=g)
    cache = cache.to(dtype)

    def rows(b):
        kv = cache[table[b + 1, :-(-lens[b] // P)].long()].transpose(1, 2).flatten(0, 1)[:lens[b]].double()
        return kv[..., :D], kv[..., up8(D):up8(D) + V]

    def queries(n):
        q = torch.zeros(n, H, up8(D))
        q[..., :D] = torch.randn(n, H, D, generator=g) * gain
        return q.to(dtype)
    return table, cache, rows, queries


def _attend(q, k, v, pos, scale, window, softcap, slope, sink):
    """Queries `[n, H, D]` at positions `pos`; also the denominators."""
    own = [h // (q.shape[1] // k.shape[1]) for h in range(q.shape[1])]
    S = k.shape[0]
    s = oracle.cap(torch.einsum("nhd,shd->hns", q, k[:, own]) * scale, softcap)
    if slope is not None:
        s = s - slope.double()[:, None, None] * (torch.as_tensor(pos)[:, None] - torch.arange(S)[None])
    see = oracle.visible(S, window or None)[pos]
    none = torch.full((q.shape[1],), -torch.inf, dtype=torch.float64)
    return torch.einsum("hns,shd->nhd", oracle.sink_softmax(s, see, none if sink is None else sink.double()), v[:, own])


# softcap, slopes?, sinks?
TERMS = [(0.0, True, True), (3.0, False, False), (1.0, True, True), (0.0, False, True), (30.0, True, False)]


def _terms(H, t, seed):
    g = torch.Generator().manual_seed(seed)
    slope = oracle.slopes(H).float() if t[1] else None
    sink = torch.randn(H, generator=g) * 2 + 1 if t[2] else None
    put = lambda x: None if x is None else x.cuda()
    return (t[0], slope, sink), dict(softcap=t[0], slope=put(slope), sink=put(sink))


@pytest.mark.parametrize("P", [16, 64])
@pytest.mark.parametrize("D,V,H,G", [(64, 64, 4, 2), (48, 40, 6, 1), (10, 7, 3, 3), (200, 200, 17, 1), (128, 128, 32, 8), (24, 256, 33, 1)])
def test_single_queries_with_shaped_scores_and_sinks(native, D, V, H, G, P):
    """bf16 on the tensor cores and fp32 on the CUDA cores, one split of the keys and several."""
    lens = [1, 2, P - 1, P, P + 1, 3 * P + 5, 300]
    for dtype in BOTH:
        table, cache, rows, queries = _window_case(D, V, H, G, lens, P, dtype, D + P)
        q = queries(len(lens))
        for i, t in enumerate(TERMS):
            window = (0, 1, 63, 64, 65)[i]
            plain, kw = _terms(H, t, i)
            want = torch.cat([_attend(q[b:b + 1, :, :D].double(), *rows(b), [n - 1], 0.11, window, *plain)
                              for b, n in enumerate(lens)])
            args = (q.cuda(), None, cache.cuda(), table.cuda(), _i32(range(1, len(lens) + 1)), _i32(lens), D, V, P, 0.11, window, 0)
            got = [native.window_attn_any(*args, **kw)]
            tol = 1e-5
            if dtype == torch.bfloat16:
                got += [native.window_decode(*args, num_splits=n, **kw) for n in (None, 1, 3)]
                tol = 2.0 ** -8                                          # half a step of the bf16 result
            for o in got:
                assert ((o.cpu().double() - want).abs() <= tol * want.abs() + 3e-5 * want.abs().max()).all(), (t, window)


@pytest.mark.parametrize("D,V,H,G,P,lens,pres,gain", [
    (64, 64, 2, 1, 64, [256], [0], 1), (40, 72, 3, 1, 64, [300, 77, 600], [0, 5, 500], 1), (128, 128, 8, 2, 128, [513, 33], [64, 0], 2),
    (192, 128, 4, 2, 64, [700], [0], 4), (10, 7, 3, 3, 32, [400], [13], 1), (64, 64, 16, 2, 64, [90, 256, 257], [37, 63, 64], 8)])
def test_prefill_tiles_with_shaped_scores_and_sinks(native, D, V, H, G, P, lens, pres, gain):
    ctx = [a + b for a, b in zip(lens, pres)]
    table, cache, rows, queries = _window_case(D, V, H, G, ctx, P, torch.bfloat16, D + V, gain)
    q = queries(sum(lens))
    qs = np.concatenate([[0], np.cumsum(lens)])
    plan = SimpleNamespace(q_start=_i32(qs[:-1]), q_len=_i32(lens), prefix=_i32(pres), rows=_i32(range(1, len(lens) + 1)),
                           long=len(lens), num_tiles=sum((n + 255) // 256 for n in lens))
    qc, cc, tc = q.cuda(), cache.cuda(), table.cuda()
    assert native.window_extend_supported(qc, cc, D, V)
    for i, t in enumerate(TERMS):
        for window in ((0, 1, 100), (64, 300), (65, 128), (17, 0), (200, 63))[i]:
            plain, kw = _terms(H, t, i)
            out = torch.full((sum(lens), H, V), torch.nan, device="cuda", dtype=torch.bfloat16)
            native.window_extend(qc, None, cc, tc, plan, out, D, V, D ** -0.5, window, 0, **kw)
            for b in range(len(lens)):
                s = slice(qs[b], qs[b + 1])
                want = _attend(q[s, :, :D].double(), *rows(b), np.arange(pres[b], ctx[b]), D ** -0.5, window, *plain)
                diff = (out[s].cpu().double() - want).abs()
                assert (diff <= 2.0 ** -8 * want.abs() + 5e-5 * want.abs().max()).all(), (b, t, window)


def _latent_case(R, rot, lens, P, dtype, seed):
    g = torch.Generator().manual_seed(seed)
    table, pages = _pages(lens, P, seed)
    cache = torch.randn(pages, P, up8(R + rot), generator=g).to(dtype)
    rows = [cache[table[b + 1, :-(-n // P)].long()].flatten(0, 1)[:n, :R + rot].double() for b, n in enumerate(lens)]
    return table, cache, rows


@pytest.mark.parametrize("P", [16, 64, 128])
@pytest.mark.parametrize("R,rot,H", [(512, 64, 16), (64, 16, 6), (128, 24, 17), (21, 6, 3)])
def test_absorbed_latent_attention_with_windows_and_sinks(native, R, rot, H, P):
    lens = [1, P - 1, P, P + 1, 3 * P + 5, 500]
    g = torch.Generator().manual_seed(R + P)
    q, sink = torch.randn(len(lens), H, R + rot, generator=g) * 1.5, torch.randn(H, generator=g) * 3
    for dtype in BOTH:
        table, cache, rows = _latent_case(R, rot, lens, P, dtype, R)
        qd = q.to(dtype)
        ql, qp = qd[..., :R].contiguous().cuda(), qd.cuda()[..., R:]
        args = (ql, qp, cache.cuda(), table.cuda(), _i32(range(1, len(lens) + 1)), _i32(lens), P, 0.11)
        for window, k in ((0, sink), (1, sink), (63, None), (64, sink), (65, sink), (130, None)):
            want = []
            for b, c in enumerate(rows):
                s = (qd[b].double() @ c.T)[:, None] * 0.11
                see = oracle.visible(len(c), window or None)[-1:]
                none = torch.full((H,), -torch.inf, dtype=torch.float64)
                want.append(oracle.sink_softmax(s, see, none if k is None else k.double())[:, 0] @ c[:, :R])
            want = torch.stack(want)
            kw = dict(window=window, sink=None if k is None else k.cuda())
            got, tol = [native.latent_attn_any(*args, **kw)], 1e-5
            if dtype == torch.bfloat16:
                got += [native.mla_decode(*args, max_seq_len=500, num_splits=n, exact=True, **kw) for n in (None, 1, 3)]
                tol = 2.0 ** -8
            for o in got:
                assert ((o.cpu().double() - want).abs() <= tol * want.abs() + 2e-5 * want.abs().max()).all(), window


@pytest.mark.parametrize("H,dim,rot,v,lens,pres,gain", [
    (2, 64, 40, 72, [256], [0], 1), (3, 64, 40, 72, [300, 77, 700], [0, 5, 900], 1), (2, 128, 64, 128, [513, 33], [64, 0], 4),
    (1, 40, 8, 24, [700], [130], 1)])
def test_expanded_latent_prefill_with_windows_and_sinks(native, H, dim, rot, v, lens, pres, gain):
    """Only the context that a window reaches is laid out."""
    from sglang_jax_b200.layers.extend_plan import ExtendPlan
    g = torch.Generator(device="cuda").manual_seed(dim + v)
    rnd = lambda *s: torch.randn(*s, generator=g, device="cuda").bfloat16()
    T, ctx = sum(lens), [a + b for a, b in zip(lens, pres)]
    q = (rnd(T, H * (dim + rot) + 24) * gain)[:, :H * (dim + rot)].unflatten(-1, (H, dim + rot))
    kv, pe = [rnd(n, H, dim + v) for n in ctx], [rnd(n, rot) for n in ctx]
    sink = torch.randn(H, generator=g, device="cuda") * 3
    fb = SimpleNamespace(extend_seq_lens_cpu=lens, extend_prefix_lens_cpu=pres, num_tokens=T, positions=torch.zeros(T, device="cuda"),
                         req_pool_indices=_i32(range(1, len(lens) + 1)), extend_seq_lens=_i32(lens))
    plan = ExtendPlan(fb, True)
    qs = np.concatenate([[0], np.cumsum(lens)])
    for window in (0, 1, 63, 64, 65, 128, 300, 1000):
        c = plan.context(window)
        skip = [0] * len(lens) if c.skip is None else c.skip.tolist()
        rows = lambda x: torch.cat([t[s:] for t, s in zip(x, skip)]).contiguous()
        assert c.total == rows(pe).shape[0]
        out = torch.full((T, H, v), torch.nan, device="cuda", dtype=torch.bfloat16)
        native.latent_extend(q, rows(kv).flatten(1), rows(pe), out, plan, dim, v, (dim + rot) ** -0.5, window, sink)
        for b in range(len(lens)):
            k = torch.cat([kv[b][..., :dim], pe[b][:, None].expand(-1, H, rot)], -1).double().cpu()
            s = torch.einsum("ihd,jhd->hij", q[qs[b]:qs[b + 1]].double().cpu(), k) * (dim + rot) ** -0.5
            a = oracle.sink_softmax(s, oracle.visible(ctx[b], window or None)[pres[b]:], sink.double().cpu())
            want = torch.einsum("hij,jhd->ihd", a, kv[b][..., dim:].double().cpu())
            diff = (out[qs[b]:qs[b + 1]].double().cpu() - want).abs()
            assert (diff <= 2.0 ** -8 * want.abs() + 3e-5 * want.abs().max()).all(), (b, window)


def test_gather_from_a_token_on(native):
    lens, skip = [70, 64, 200], [64, 0, 128]
    table, cache, rows = _latent_case(40, 8, lens, 16, torch.bfloat16, 1)
    start = np.concatenate([[0], np.cumsum([n - s for n, s in zip(lens, skip)])])
    lat, pe = native.latent_gather(cache.cuda(), table.cuda(), _i32([1, 2, 3]), _i32(start), int(start[-1]), 40, 8, 16, _i32(skip))
    assert torch.equal(torch.cat([lat, pe], -1).cpu().double(), torch.cat([r[s:] for r, s in zip(rows, skip)]))


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
def test_mixed_batches_with_pages_used_again(models, name, dtype):
    path, cfg, w = models[name]
    lens = [140, 3, 165, 17, 70, 64, 1, 90]
    reqs = {i: cases.tokens(n, cfg["vocab"], 50 + i) for i, n in enumerate(lens)}
    sizes = [[37, 1, 1, 2], [1], [132, 1], [2], [16, 1, 50], [63, 1], [1], [3, 34, 1]]
    steps = cases.interleave(reqs, {i: cases.cut(n, sizes[i]) for i, n in enumerate(lens)})
    cases.check(path, cfg, w, dtype, "cuda", reqs, steps, 512)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_one_key_decides_inside_the_window(tmp_path, kind, dtype):
    cfg, w = needle_model(kind, 100)
    path = cases.write(str(tmp_path), cfg, w)
    for distance in (0, 1, 63, 64, 65, 98, 99, 100, 101, 290):
        ids = needle_prompt(distance, 300)
        want = {"a": cases.expectation(ids, w, cfg)}
        for steps in ([[("a", 300)]], [[("a", 299)], [("a", 1)]], [[("a", n)] for n in cases.cut(300, [60, 2, 131, 1])]):
            cases.check(path, cfg, w, dtype, "cuda", {"a": ids}, steps, 320, want)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_with_heavy_sinks(tmp_path, dtype):
    cfg, w = sink_model()
    ids = cases.tokens(180, cfg["vocab"], 2)
    path, want = cases.write(str(tmp_path), cfg, w), {"a": cases.expectation(ids, w, cfg)}
    for first in (2, 70):
        cases.check(path, cfg, w, dtype, "cuda", {"a": ids}, [[("a", first)]] + [[("a", 1)]] * (180 - first), 192, want)


# ------------------------------------------------------------------ engine
def _engine(path, dtype, **kw):
    from sglang_jax_b200 import Engine
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    return Engine(model_path=path, device="cuda", dtype=dtype, skip_tokenizer_init=True, enable_single_process=True,
                  **{"page_size": 64, "max_total_tokens": 4096, "max_running_requests": 8, "cuda_graph_max_bs": 8, **kw})


def _near_greedy(prompt, out, w, cfg, dtype):
    """Every generated token is the oracle's best one, or nearly as good."""
    logits = oracle.forward(prompt + out, w, cfg)[len(prompt) - 1:-1]
    best = logits.max(-1).values - logits[torch.arange(len(out)), torch.tensor(out)]
    return bool((best <= (1e-4 if dtype == "float32" else 0.2) * logits.std()).all())


@pytest.mark.parametrize("kw", [dict(), dict(disable_cuda_graph=True), dict(chunked_prefill_size=64, enable_mixed_chunk=True)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_engine(models, dtype, kw):
    path, cfg, w = models["plain" if dtype == "float32" else "dense"]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (29, 7, 170, 64, 65)]
    eng = _engine(path, dtype, **kw)
    try:
        got = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 12, "temperature": 0, "ignore_eos": True})
        for p, o in zip(prompts, got):
            assert len(o["output_ids"]) == 12
            assert _near_greedy(p, o["output_ids"], w, cfg, dtype)
        info = eng.get_server_info()["internal_states"][0]
        assert (info["cuda_graph_replays"] > 5) != bool(kw.get("disable_cuda_graph")) and info["cuda_graph_recaptures"] == 0
        eng.scheduler.check_memory()
    finally:
        eng.shutdown()


def test_shared_prefixes(models):
    path, cfg, w = models["mixed"]
    base = cases.tokens(150, cfg["vocab"], 1)
    eng = _engine(path, "float32")
    try:
        sp = {"max_new_tokens": 4, "temperature": 0, "ignore_eos": True}
        eng.generate(input_ids=base, sampling_params=sp)
        again = base[:128] + cases.tokens(20, cfg["vocab"], 2)
        out = eng.generate(input_ids=again, sampling_params=sp)
        assert out["meta_info"]["cached_tokens"] == 128
        assert _near_greedy(again, out["output_ids"], w, cfg, "float32")
    finally:
        eng.shutdown()
