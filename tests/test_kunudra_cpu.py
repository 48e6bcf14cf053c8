"""Kunudra on the CPU: every mechanism against the oracle, schedules, caches, loading and generation through the engine."""

import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import kunudra_cases as cases
import kunudra_oracle as oracle


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in cases.CONFIGS.items():
        w = cases.random_weights(cfg, seed=len(name))
        out[name] = (cases.write(str(tmp_path_factory.mktemp(name)), cfg, w), cfg, w)
    return out


# ------------------------------------------------------------------ mechanisms alone
def test_pairs_are_hashed_and_the_predecessor_comes_from_the_step_or_the_slot():
    from sglang_jax_b200 import ops
    g = torch.Generator().manual_seed(0)
    buckets, mp, mc, P = 11, 1_000_003, 7, 4
    table, pairs = torch.randn(50, 6, generator=g), torch.randn(buckets + 1, 6, generator=g)
    seqs = [cases.tokens(n, 50, n) for n in (9, 1, 6)]
    page_table = torch.tensor([[0, 0, 0], [5, 2, 7], [1, 0, 0], [3, 4, 0]], dtype=torch.int32)
    slots = torch.full((32,), 49, dtype=torch.int32)
    mode = lambda decode: SimpleNamespace(is_decode=lambda: decode)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32)

    def step(parts, decode=False):
        """`parts`: (sequence, from, to)."""
        ids = [t for s, a, b in parts for t in seqs[s][a:b]]
        pos = [i for _, a, b in parts for i in range(a, b)]
        loc = [int(page_table[s + 1, i // P]) * P + i % P for s, a, b in parts for i in range(a, b)]
        fb = SimpleNamespace(positions=i32(pos), out_cache_loc=i32(loc), forward_mode=mode(decode), page_table=page_table,
                             page_size=P, req_pool_indices=i32([s + 1 for s, _, _ in parts]),
                             cu_q_lens=i32(np.concatenate([[0], np.cumsum([b - a for _, a, b in parts])])))
        x, _ = ops.embed_pair(i32(ids), table, pairs, mp, mc, slots, fb)
        rows = [oracle.pair_rows(seqs[s], buckets, mp, mc)[i] for s, a, b in parts for i in range(a, b)]
        assert torch.equal(x, table[ids] + pairs[rows])

    step([(0, 0, 4), (1, 0, 1), (2, 0, 2)])
    step([(2, 2, 5), (0, 4, 7)])
    step([(0, 7, 8), (2, 5, 6)], decode=True)
    step([(0, 8, 9)], decode=True)
    assert oracle.pair_rows([3, 3], 11, 2, 5) == [11, 21 % 11]


def test_norm_behind_the_sum_takes_experts_the_input_itself_and_a_gate():
    from sglang_jax_b200 import ops
    g = torch.Generator().manual_seed(1)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, y, s, w, nw = rnd(5, 24), rnd(5, 24), rnd(24), rnd(24), rnd(24)
    e, weights, gate = rnd(9, 24), torch.rand(5, 2, generator=g), torch.rand(5, generator=g)
    ids = torch.tensor([[0, 3], [4, 1], [3, 4], [2, 0], [1, 2]], dtype=torch.int32)                  # experts 0 .. 2
    rows = torch.where(ids < 3, torch.arange(10).view(5, 2) % 9, -1).int()
    add = torch.stack([sum((weights[t, j] * (e[rows[t, j]] if ids[t, j] < 3 else x[t]) for j in range(2)), gate[t] * y[t])
                       for t in range(5)])
    want = oracle.norm_sum(x, add, s, 0.7, w - 1, 1e-3)
    got = x.clone()
    h = ops.sum_norm(y, got, 0.7, s, w, 1e-3, y_gate=gate, expert_out=e, weights=weights, pair_row=rows.flatten(), ids=ids,
                     experts=3)
    assert torch.allclose(got, want, atol=1e-5) and torch.equal(h, got)
    got = x.clone()
    h = ops.sum_norm(y, got, 0.7, s, w, 1e-3, next_weight=nw, next_eps=1e-2)
    want = oracle.norm_sum(x, y, s, 0.7, w - 1, 1e-3)
    assert torch.allclose(got, want, atol=1e-5) and torch.allclose(h, oracle.rms(want, 1e-2) * nw, atol=1e-5)


def test_norm_weights_around_zero():
    from sglang_jax_b200.layers.layernorm import StreamRMSNorm, SumNorm
    a, b = SumNorm(8, 1e-6, 2.0, torch.float32), StreamRMSNorm(8, 1e-6, dtype=torch.float32, one_plus=True)
    for m in (a, b):
        assert torch.equal(m.weight.data, torch.zeros(8))
        m.weight.data.fill_(0.25)
        m.fold()
    assert torch.equal(a.norm_scale, torch.full((8,), 1.25)) and torch.equal(b.channel_scale, torch.full((8,), 1.25))


def test_router_chooses_by_corrected_score_and_weighs_by_the_score():
    from sglang_jax_b200.layers.gate import GateLogit
    gate = GateLogit(8, 6, torch.float32, correction_bias=True, token_gate=True)
    g = torch.Generator().manual_seed(0)
    gate.weight.data[:7] = torch.randn(7, 8, generator=g)
    gate.e_score_correction_bias.data.copy_(torch.randn(6, generator=g) * 0.3)
    x = torch.randn(20, 8, generator=g)
    w = {"router": gate.weight[:6], "correction": gate.e_score_correction_bias}
    for top in (1, 3, 6):
        got, ids, own = gate.route_by_score(x, top, 1.7)
        want_ids, want_w = oracle.route(x, w, "", top, 1.7)
        assert torch.equal(ids.long(), want_ids) and torch.allclose(got, want_w, atol=1e-6)
        assert torch.allclose(own, torch.sigmoid(x @ gate.weight[6]), atol=1e-6)
    plain = torch.topk(torch.softmax(x @ w["router"].T, -1), 3).indices
    assert gate.weight.shape[0] == 8 and not gate.weight[7].any()
    assert not torch.equal(plain, gate.route_by_score(x, 3, 1.0)[1].long())               # the correction matters here


def test_identity_choices_and_the_shared_expert():
    from sglang_jax_b200.layers.layernorm import SumNorm
    from sglang_jax_b200.layers.moe import ScoredFeedForward
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    cfg = cases.config([cases.attention(2, 1, 8, 8, 4, mlp=cases.moe(12, 2, 3, 3, 1.4, 10))], 16, 20)
    w = {n: t.float() for n, t in cases.random_weights(cfg, 1).items()}
    ff, norm = ScoredFeedForward(16, 2, 3, 3, 12, 1.4, 10, torch.float32), SumNorm(16, 1e-6, 1.0, torch.float32)
    for n, t in w.items():
        if n.startswith("l0.mlp."):
            ff.load(n[7:], t)
    x = torch.randn(40, 16, generator=torch.Generator().manual_seed(2))
    ids = oracle.route(x, w, "l0.mlp.", 3, 1.4)[0]
    assert (ids >= 2).all(1).any() and (ids < 2).any()
    want = oracle.norm_sum(x, oracle.sparse_ff(x, w, "l0.mlp.", cfg["layers"][0]["mlp"]), torch.ones(16), 1.0, torch.zeros(16), 1e-6)
    got = x.clone()
    ff(x.clone(), got, norm)
    assert torch.allclose(got, want, atol=1e-5)


def test_listeners_hear_of_experts_only():
    from sglang_jax_b200.eplb.expert_location import ExpertDistributionRecorder, ExpertLocation
    from sglang_jax_b200.layers.moe import FusedMoE
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    m = FusedMoE(3, 8, 8, torch.float32, activation="swiglu")
    m.extra_choices = 2
    m.recorder, m.expert_location = ExpertDistributionRecorder(1, 3), ExpertLocation(3, 1, 1)
    m.expert_location.dispatch_algorithm = "static"
    ids = torch.tensor([[0, 4], [3, 2], [2, 1]], dtype=torch.int32)
    assert m._observe(ids).tolist() == [[0, -1], [-1, 2], [2, 1]]
    assert m.recorder.counts.tolist() == [[1, 1, 2]]


def test_score_terms_of_the_oracle():
    assert torch.allclose(oracle.slopes(8), torch.tensor([2.0 ** -(h + 1) for h in range(8)], dtype=torch.float64))
    assert torch.allclose(oracle.slopes(6)[[0, 5]], torch.tensor([2 ** (-8 / 6), 2.0 ** -8], dtype=torch.float64))
    assert oracle.distance_bias(5, 2)[0, 4, 1] == 3 * oracle.slopes(2)[0]
    assert oracle.visible(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 1, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 1, 1]]
    s = torch.zeros(1, 1, 2)
    assert torch.allclose(oracle.sink_softmax(s, torch.ones(1, 2, dtype=torch.bool), torch.tensor([math.log(2.0)])),
                          torch.full((1, 1, 2), 0.25))


@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_whole_prompts_match_the_oracle(models, name):
    path, cfg, w = models[name]
    reqs = {n: cases.tokens(n, cfg["vocab"], n) for n in (1, 2, 95)}
    cases.check(path, cfg, w, "float32", "cpu", reqs, [[(n, n)] for n in reqs], 128)


# ------------------------------------------------------------------ schedules
@pytest.mark.parametrize("name", ["plain", "mixed"])
@pytest.mark.parametrize("sizes", [[1], [2], [5, 1, 1, 2], [16, 15, 17], [64, 1]])
def test_portions_and_token_by_token(models, name, sizes):
    path, cfg, w = models[name]
    reqs = {"a": cases.tokens(81, cfg["vocab"], 1)}
    cases.check(path, cfg, w, "float32", "cpu", reqs, [[("a", n)] for n in cases.cut(81, sizes)], 96, page_size=16)


@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_unequal_requests_in_mixed_batches_with_pages_used_again(models, name):
    path, cfg, w = models[name]
    lens = [40, 3, 65, 17, 33, 64, 1, 20]
    reqs = {i: cases.tokens(n, cfg["vocab"], 50 + i) for i, n in enumerate(lens)}
    sizes = [[7, 1, 1, 2], [1], [32, 1, 1, 1], [2], [16], [63, 1], [1], [3, 1]]
    portions = {i: cases.cut(n, sizes[i]) for i, n in enumerate(lens)}
    cases.check(path, cfg, w, "float32", "cpu", reqs, cases.interleave(reqs, portions), 240, page_size=16)


def test_a_request_may_pause_between_its_steps(models):
    path, cfg, w = models["plain"]
    reqs = {"a": cases.tokens(20, cfg["vocab"], 1), "b": cases.tokens(30, cfg["vocab"], 2)}
    steps = [[("a", 9)], [("b", 10)], [("b", 1)], [("a", 1), ("b", 5)], [("b", 14)], [("a", 10)]]
    cases.check(path, cfg, w, "float32", "cpu", reqs, steps, 128)


# ------------------------------------------------------------------ what random weights would hide
def needle_model(kind, window, seed=3):
    """One layer whose last token (48) asks for the marker token (49): keys are the first half of a token's embedding, queries the
    second half, and the two agree for that pair only, so that its score stands far above all others (also above the bias of
    a distance as long as the window and above the sink) and whether that key is seen decides the logits."""
    W, D = 64, 16
    if kind == "attention":
        layers = [cases.attention(2, 2, D, D, window, 60.0, scale=6.0)]
    else:
        layers = [cases.latent(2, D, 2, D, 64, 64, window, scale=3.0)]
    cfg = cases.config(layers, W, 50, alpha=1.0)
    w = cases.random_weights(cfg, seed)
    w["bigram"] = torch.zeros_like(w["bigram"])
    p = "l0.mix."
    pick = torch.zeros(2, D, W)
    for h in range(2):
        pick[h, torch.arange(D), torch.arange(D) + D * h] = 1.0
    if kind == "attention":
        w[p + "k"], w[p + "q"] = pick.reshape(2 * D, W), pick.roll(W // 2, 2).reshape(2 * D, W)
        w[p + "q.norm"], w[p + "k.norm"] = torch.ones(2 * D), torch.ones(2 * D)
    else:
        w[p + "dkv"] = torch.cat([torch.eye(W), torch.zeros(2, W)])
        w[p + "dq"], w[p + "dkv.norm"], w[p + "dq.norm"] = torch.eye(W), torch.ones(W), torch.ones(W)
        w[p + "uk"] = pick.reshape(2 * D, W)
        up = torch.zeros(2, D + 2, W)
        up[:, :D] = pick.roll(W // 2, 2)
        w[p + "uq"] = up.reshape(-1, W)
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    w["embed"][48, 32:] = w["embed"][49, :32]
    w[p + "sink"] = torch.full((2,), -2.0).bfloat16()
    return cfg, w


def needle_prompt(distance, length):
    """The asking token at the end, the marker `distance` tokens before it (0: no marker)."""
    ids = cases.tokens(length, 40, distance)
    ids[-1] = 48
    if distance:
        ids[-1 - distance] = 49
    return ids


@pytest.mark.parametrize("kind", ["attention", "latent"])
@pytest.mark.parametrize("distance", [1, 15, 16, 17, 38, 39, 40, 41, 100])
def test_one_key_decides_inside_the_window(tmp_path, kind, distance):
    """Window 40: seen or not, the key shows."""
    cfg, w = needle_model(kind, 40)
    ids = needle_prompt(distance, 110)
    without = list(ids)
    without[-1 - distance] = 7
    moved = float(cases.error(oracle.forward(ids, w, cfg)[-1:], oracle.forward(without, w, cfg)[-1:]))
    # (token 49 in front of the last one also moves the pair's row, which is zero here)
    assert (moved > 0.05) == (distance < 40), moved
    path = cases.write(str(tmp_path), cfg, w)
    want = {"a": cases.expectation(ids, w, cfg)}
    for steps in ([[("a", 110)]], [[("a", 109)], [("a", 1)]], [[("a", n)] for n in cases.cut(110, [60, 2, 31])]):
        cases.check(path, cfg, w, "float32", "cpu", {"a": ids}, steps, 128, want, page_size=16)


def sink_model(seed=4):
    """Sinks as heavy as the keys, slopes that matter within the window and a cap that bites."""
    cfg = cases.config([cases.attention(4, 2, 32, 24, 30, 2.0, True, scale=1.5), cases.latent(4, 24, 8, 24, 40, 32, 30, scale=1.0),
                        cases.attention(4, 2, 32, 24, 12, 1.0, True, scale=1.5)], 96, 64)
    w = cases.random_weights(cfg, seed)
    for i in range(3):
        w[f"l{i}.mix.sink"] = torch.tensor([-1.0, 1.0, 2.5, 4.0]).bfloat16()
    return cfg, w


MISTAKES = ["bias_absolute", "bias_before_cap", "no_cap", "no_bias", "sink_left_out", "sink_capped", "window_short", "window_long",
            "shared_head", "own_key", "norm_per_head", "value_mix", "value_mix_first_own", "rotation_halves", "alpha", "norm_before",
            "one_plus", "pair_first", "pair_swapped", "pair_lost", "correction_in_weights", "renormalised", "identity", "shared_gate",
            "slopes"]


@pytest.mark.parametrize("wrong", MISTAKES)
def test_the_oracle_tells_planted_mistakes_apart(models, wrong, monkeypatch):
    """A mistake planted in the oracle moves the logits by far more than the tests' limits."""
    _, cfg, w = models["plain"]
    if wrong in ("sink_left_out", "sink_capped", "bias_before_cap", "bias_absolute"):
        cfg, w = sink_model()
    ids = cases.tokens(40, cfg["vocab"], 9)
    good = oracle.forward(ids, w, cfg)
    names = ("cap", "distance_bias", "sink_softmax", "visible", "mix_values", "rms", "rotate", "norm_sum", "pair_rows", "route",
             "shared_ff", "sparse_ff", "slopes", "attention_mixer")
    was = {n: getattr(oracle, n) for n in names}
    put = lambda n, f: monkeypatch.setattr(oracle, n, f)
    if wrong == "bias_absolute":          # slope * j, as if the softmax had no other entries
        put("distance_bias", lambda T, H: -oracle.slopes(H)[:, None, None] * torch.arange(T)[None, :].expand(T, T))
    elif wrong == "bias_before_cap":
        put("cap", lambda s, c: was["cap"](s - was["distance_bias"](s.shape[-1], s.shape[0]), c))
        put("distance_bias", lambda T, H: torch.zeros(H, T, T))
    elif wrong == "no_cap":
        put("cap", lambda s, c: s)
    elif wrong == "no_bias":
        put("distance_bias", lambda T, H: torch.zeros(H, T, T))
    elif wrong == "slopes":
        put("slopes", lambda H: was["slopes"](H).flip(0))
    elif wrong == "sink_left_out":
        put("sink_softmax", lambda s, m, k: was["sink_softmax"](s, m, torch.full_like(k, -math.inf)))
    elif wrong == "sink_capped":
        put("sink_softmax", lambda s, m, k: was["sink_softmax"](s, m, 2 * torch.tanh(k / 2)))
    elif wrong in ("window_short", "window_long"):
        put("visible", lambda T, n: was["visible"](T, n + (1 if wrong == "window_long" else -1)))
    elif wrong == "shared_head":
        w = {**w, "l0.mix.k": w["l0.mix.k"].view(2, 32, -1).flip(0).reshape(64, -1)}
    elif wrong == "own_key":              # every token sees its predecessor's key in the place of its own
        put("sink_softmax", lambda s, m, k: was["sink_softmax"](s.roll(1, -1), m, k))
    elif wrong == "norm_per_head":
        put("rms", lambda x, eps: was["rms"](x.view(-1, x.shape[-1] // 32, 32), eps).view(x.shape) if x.shape[-1] in (64, 128) else
            was["rms"](x, eps))
    elif wrong == "value_mix":
        put("mix_values", lambda v, f, s: s * v + (1 - s) * f)
    elif wrong == "value_mix_first_own":  # no mixing at all
        put("mix_values", lambda v, f, s: v)
    elif wrong == "rotation_halves":      # pairs (i, i + d / 2)
        def halves(x, p, base):
            d = x.shape[-1]
            order = torch.arange(d).view(2, d // 2).T.flatten()
            return was["rotate"](x[..., order], p, base)[..., torch.argsort(order)]
        put("rotate", halves)
    elif wrong == "alpha":
        put("norm_sum", lambda x, y, s, a, wt, e: was["norm_sum"](x, y, s, 1.0, wt, e))
    elif wrong == "norm_before":
        put("norm_sum", lambda x, y, s, a, wt, e: a * x + oracle.rms(y * s, e) * (1 + wt))
    elif wrong == "one_plus":
        put("norm_sum", lambda x, y, s, a, wt, e: oracle.rms(a * x + y * s, e) * wt)
    elif wrong == "pair_first":
        put("pair_rows", lambda t, b, p, c: [t[0] * c % b] + was["pair_rows"](t, b, p, c)[1:])
    elif wrong == "pair_swapped":
        put("pair_rows", lambda t, b, p, c: was["pair_rows"](t, b, c, p))
    elif wrong == "pair_lost":            # the portion from token 20 on has no predecessor
        put("pair_rows", lambda t, b, p, c: was["pair_rows"](t[:20], b, p, c) + was["pair_rows"](t[20:], b, p, c))
    elif wrong == "correction_in_weights":
        def corrected(h, w, p, top, scale):
            chosen, _ = was["route"](h, w, p, top, scale)
            return chosen, (torch.softmax(h @ w[p + "router"].T, -1) + w[p + "correction"]).gather(1, chosen) * scale
        put("route", corrected)
    elif wrong == "renormalised":
        def whole(h, w, p, top, scale):
            chosen, c = was["route"](h, w, p, top, scale)
            return chosen, c / c.sum(-1, keepdim=True) * scale
        put("route", whole)
    elif wrong == "identity":             # identity choices give nothing
        def nothing(h, w, p, m):
            chosen, c = oracle.route(h, w, p, m["router"]["top"], m["router"]["scale"])
            return was["sparse_ff"](h, w, p, m) - (c * (chosen >= m["router"]["experts"])).sum(-1, keepdim=True) * h
        put("sparse_ff", nothing)
    elif wrong == "shared_gate":
        put("shared_ff", lambda h, w, p: oracle.gated(h, w, p + "shared."))
    assert float(cases.error(oracle.forward(ids, w, cfg), good).max()) > 1e-2


def test_sinks_caps_and_slopes_in_portions(tmp_path):
    cfg, w = sink_model()
    ids = cases.tokens(70, cfg["vocab"], 2)
    path, want = cases.write(str(tmp_path), cfg, w), {"a": cases.expectation(ids, w, cfg)}
    for sizes in ([70], [1], [33, 2]):
        cases.check(path, cfg, w, "float32", "cpu", {"a": ids}, [[("a", n)] for n in cases.cut(70, sizes)], 96, want, page_size=16)


# ------------------------------------------------------------------ engine
def _engine(path, **kw):
    from sglang_jax_b200 import Engine
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    return Engine(model_path=path, skip_tokenizer_init=True, enable_single_process=True,
                  **{"device": "cpu", "dtype": "float32", "page_size": 16, "max_total_tokens": 2048, **kw})


PROMPTS = [29, 7, 70, 33]
GREEDY = {"temperature": 0, "ignore_eos": True}


@pytest.mark.parametrize("kw", [dict(), dict(chunked_prefill_size=16), dict(disable_overlap_schedule=True),
                                dict(chunked_prefill_size=32, enable_mixed_chunk=True),
                                dict(max_total_tokens=176, disable_overlap_schedule=True)])
def test_greedy_generation_through_the_engine(models, kw):
    """The last one runs out of pages: requests are retracted and start again."""
    path, cfg, w = models["plain"]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in PROMPTS]
    want = [oracle.greedy(p, w, cfg, 8) for p in prompts]
    eng = _engine(path, **kw)
    try:
        got = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 8, **GREEDY})
        assert [o["output_ids"] for o in got] == want
        eng.scheduler.check_memory()
    finally:
        eng.shutdown()


@pytest.mark.parametrize("name", ["mixed", "odd", "latent_only", "attention_only"])
def test_greedy_generation_of_every_layout(models, name):
    path, cfg, w = models[name]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (20, 5)]
    eng = _engine(path)
    try:
        got = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 5, **GREEDY})
        assert [o["output_ids"] for o in got] == [oracle.greedy(p, w, cfg, 5) for p in prompts]
    finally:
        eng.shutdown()


@pytest.mark.parametrize("kw", [dict(), dict(hicache_storage="file", hicache_ratio=2.0)])
def test_shared_prefixes(models, kw):
    """A request that starts inside another's pages takes its first token's predecessor from there."""
    path, cfg, w = models["plain"]
    base = cases.tokens(70, cfg["vocab"], 1)
    sp = {"max_new_tokens": 4, **GREEDY}
    eng = _engine(path, **kw)
    try:
        eng.generate(input_ids=base, sampling_params=sp)
        again = base[:64] + cases.tokens(20, cfg["vocab"], 2)
        out = eng.generate(input_ids=again, sampling_params=sp)
        assert out["meta_info"]["cached_tokens"] == 64
        assert out["output_ids"] == oracle.greedy(again, w, cfg, 4)
        eng.scheduler.check_memory()
    finally:
        eng.shutdown()


def test_sampling_and_input_logprobs(models):
    path, cfg, w = models["plain"]
    ids = cases.tokens(30, cfg["vocab"], 4)
    eng = _engine(path)
    try:
        out = eng.generate(input_ids=ids, sampling_params={"max_new_tokens": 2, "temperature": 0.8, "top_k": 5,
                                                           "ignore_eos": True}, return_logprob=True, logprob_start_len=0)
        logits = oracle.forward(ids, w, cfg)
        assert out["output_ids"][0] in torch.topk(logits[-1], 5).indices.tolist()
        lp = torch.log_softmax(logits, -1)
        want = [float(lp[i, ids[i + 1]]) for i in range(29)]
        got = [x[0] for x in out["meta_info"]["input_token_logprobs"] if x[0] is not None]
        assert np.allclose(got, want, atol=1e-3)
    finally:
        eng.shutdown()


# ------------------------------------------------------------------ configuration, loading, pools
def test_unknown_parts_of_a_configuration_are_refused(tmp_path):
    from sglang_jax_b200.configs.model_config import ModelConfig
    good = cases.CONFIGS["plain"]
    attn, lat = good["layers"][:2]
    other = dict(attn, mixer=dict(attn["mixer"], vdim=48))
    for change in ([dict(attn, type="window")], [dict(attn, mlp={"kind": "conv"})], [attn, other],
                   [dict(lat, mixer=dict(lat["mixer"], rot={"base": 1e4, "dims": 8}))]):
        (tmp_path / "config.json").write_text(json.dumps({**good, "layers": change}))
        with pytest.raises(ValueError):
            ModelConfig(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps(good))
    mc = ModelConfig(str(tmp_path), context_length=100_000)           # positions have no limit of their own
    assert mc.architectures == ["KunudraForCausalLM"] and mc.context_len == 100_000 and mc.num_experts == 6


@pytest.mark.parametrize("change", ["missing", "unexpected", "expert"])
def test_checkpoints_must_be_complete(tmp_path, change):
    cfg = cases.CONFIGS["plain"]
    w = cases.random_weights(cfg)
    if change == "missing":
        w.pop("l1.mix.sink")
    else:
        w["l1.mix.bias" if change == "unexpected" else "l0.mlp.e6.up"] = torch.zeros(4)
    path = cases.write(str(tmp_path), cfg, w)
    with pytest.raises(RuntimeError, match="missing|unexpected"):
        cases.replay(path, "float32", "cpu", {}, [], 64)


def test_tensors_that_nothing_reads_may_be_there(tmp_path):
    """The second norm of a layer without a feed-forward, the share of a layer that mixes no values."""
    cfg = cases.CONFIGS["mixed"]
    w = cases.random_weights(cfg, 5)
    extra = {"l2.norm2": torch.zeros(120), "l2.ls2": torch.ones(120), "l1.mix.vmix": torch.tensor(0.5)}
    path = cases.write(str(tmp_path), cfg, {**w, **{n: t.bfloat16() for n, t in extra.items()}})
    cases.check(path, cfg, w, "float32", "cpu", {"a": cases.tokens(9, cfg["vocab"], 1)}, [[("a", 9)]], 64)


def test_pool_of_latent_and_packed_rows_with_token_ids():
    from sglang_jax_b200.mem_cache.memory_pool import PackedKVPool
    shapes = [(1, 27, 0), (2, 10, 16)]
    kv = PackedKVPool(64, 16, torch.float32, shapes, "cpu", token_ids=True)
    assert [tuple(b.shape) for b in kv.kv_buffer] == [(5, 1, 16, 32), (5, 2, 16, 32), (5, 16)]
    assert kv.get_latent_buffer(0).shape == (5, 16, 32) and kv.get_latent_buffer(0).data_ptr() == kv.kv_buffer[0].data_ptr()
    assert kv.get_kv_size_bytes() == 5 * 16 * PackedKVPool.cell_size(shapes, torch.float32, True)
    src, dst = torch.tensor([17, 63, 5]), torch.tensor([2, 70, 33])
    want = [(torch.randn(3, h, k), torch.randn(3, h, v)) for h, k, v in shapes]
    for i, (k, v) in enumerate(want):
        kv.set_kv_buffer(i, src, k, v)
    kv.token_ids[src] = torch.tensor([7, 8, 9], dtype=torch.int32)
    kv.move_kv(src, dst)
    for i in range(2):
        for loc in (src, dst):
            assert all(torch.equal(a, b) for a, b in zip(kv.gather(i, loc), want[i]))
    assert kv.token_ids[dst].tolist() == [7, 8, 9]


def test_host_tier_moves_token_ids_with_the_pages():
    from sglang_jax_b200.mem_cache.host_kv_pool import HostKVPool
    from sglang_jax_b200.mem_cache.memory_pool import PackedKVPool
    kv = PackedKVPool(64, 16, torch.float32, [(1, 8, 0)], "cpu", token_ids=True)
    kv.token_ids[32:48] = torch.arange(16, dtype=torch.int32)
    host = HostKVPool(kv, 4)
    host.backup_from_device(np.array([2]), np.array([1]))
    host.load_to_device(np.array([1]), np.array([4]))
    assert torch.equal(kv.token_ids[64:80], torch.arange(16, dtype=torch.int32))


def test_context_of_a_window():
    from sglang_jax_b200.layers.extend_plan import ExtendPlan
    fb = SimpleNamespace(extend_seq_lens_cpu=[100, 5, 40], extend_prefix_lens_cpu=[300, 0, 64], num_tokens=145,
                         positions=torch.zeros(145, dtype=torch.int32), req_pool_indices=torch.tensor([3, 1, 2], dtype=torch.int32),
                         extend_seq_lens=torch.tensor([100, 5, 40], dtype=torch.int32))
    plan = ExtendPlan(fb, True)
    every = plan.context()
    assert every.start.tolist() == [0, 400, 504] and every.skip is None and every.total == 504
    some = plan.context(65)                                   # token 300 sees from 236 on: rows from 192 on
    assert some.skip.tolist() == [192, 0] and some.start.tolist() == [0, 208, 312] and some.total == 312
    assert plan.context(65) is some and plan.context(500).skip is None


# ------------------------------------------------------------------ tensor parallel
def _tp_rank(rank, world, port, path, prompts, kw, q):
    from sglang_jax_b200.parallel import state as ps
    from sglang_jax_b200.server_args import ServerArgs
    torch.set_num_threads(2)
    ps.init_distributed(rank, world, "cpu", init_method=f"tcp://127.0.0.1:{port}", timeout_s=120)
    sa = ServerArgs(model_path=path, device="cpu", dtype="float32", page_size=16, skip_tokenizer_init=True,
                    max_total_tokens=1024, enable_single_process=True, max_running_requests=8, tp_size=world,
                    log_level="error", watchdog_timeout=0, **kw)
    if rank:
        from sglang_jax_b200.managers.tp_worker import run_tp_follower
        run_tp_follower(sa)
    else:
        from sglang_jax_b200 import Engine
        eng = Engine(server_args=sa)
        outs = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 8, **GREEDY})
        q.put([o["output_ids"] for o in outs])
        eng.shutdown()
    ps.destroy()


@pytest.mark.parametrize("kv_heads,kw", [(2, {}), (1, {}), (2, {"ep_size": 2})])
def test_two_tensor_ranks_generate_what_one_does(models, tmp_path, kv_heads, kw):
    """Key heads split over the ranks, one key head that both hold, and experts split over the ranks."""
    import torch.multiprocessing as mp
    from sglang_jax_b200.utils.common import get_free_port
    path, cfg, w = models["plain"]
    if kv_heads == 1:
        cfg = cases.config([cases.attention(4, 1, 32, 24, 24, 3.0, True, mlp=cases.moe(48, 6, 2, 2, 1.2, 16)),
                            cases.attention(2, 1, 32, 24, 50, None, True, mlp=cases.dense(64))], 128, 200)
        w = cases.random_weights(cfg, 3)
        path = cases.write(str(tmp_path), cfg, w)
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (21, 40)]
    ctx = mp.get_context("spawn")
    q, port = ctx.Queue(), get_free_port()
    procs = [ctx.Process(target=_tp_rank, args=(r, 2, port, path, prompts, kw, q)) for r in range(2)]
    for p in procs:
        p.start()
    try:
        outs = q.get(timeout=240)
    finally:
        for p in procs:
            p.join(timeout=60)
            if p.is_alive():
                p.kill()
    assert outs == [oracle.greedy(p, w, cfg, 8) for p in prompts]
