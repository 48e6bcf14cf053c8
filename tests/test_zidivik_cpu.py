"""Zidivik on the CPU: every mechanism against the oracle, schedules, caches, loading and generation through the engine."""

import json
import math

import numpy as np
import pytest
import torch

import zidivik_cases as cases
import zidivik_oracle as oracle


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in cases.CONFIGS.items():
        w = cases.random_weights(cfg, seed=len(name))
        out[name] = (cases.write(str(tmp_path_factory.mktemp(name)), cfg, w), cfg, w)
    return out


# ------------------------------------------------------------------ mechanisms alone
def test_positions_are_added_to_the_embedding():
    from sglang_jax_b200 import ops
    g = torch.Generator().manual_seed(0)
    for width in (6, 7):
        table, ids = torch.randn(5, width, generator=g), torch.tensor([4, 0, 4], dtype=torch.int32)
        pos = torch.tensor([0, 3, 100_000], dtype=torch.int32)
        turns = 10000.0 ** (-2.0 * torch.arange((width + 1) // 2, dtype=torch.float64) / width) / (2 * math.pi)
        x, _ = ops.embed_scaled(ids, table, 1.0, pos, turns)
        assert torch.allclose(x.double(), table[ids.long()].double() + oracle.position_vectors(pos, width), atol=1e-6)
    assert torch.equal(oracle.position_vectors(torch.tensor([0]), 4)[0], torch.tensor([0., 1., 0., 1.]).double())


def test_stream_ops():
    from sglang_jax_b200 import ops
    g = torch.Generator().manual_seed(1)
    x, y, s, n = torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g), torch.randn(24, generator=g), torch.randn(24, generator=g)
    want = x.double() + oracle.rms(y.double(), 1e-3) * s.double()
    h = ops.postnorm_add_norm(y, x, s, 1e-3, n, 1e-2)
    assert torch.allclose(x.double(), want, atol=1e-5) and torch.allclose(h.double(), oracle.rms(want, 1e-2) * n.double(), atol=1e-5)
    e, w = torch.randn(9, 24, generator=g), torch.rand(5, 2, generator=g)
    rows = torch.tensor([[0, 1], [8, -1], [3, 3], [-1, -1], [2, 7]], dtype=torch.int32)
    want = x + y + torch.stack([sum((w[t, j] * e[r] for j, r in enumerate(rows[t]) if r >= 0), torch.zeros(24)) for t in range(5)])
    ops.stream_add(y, x, e, w, rows.flatten())
    assert torch.allclose(x, want, atol=1e-5)


def test_clipped_gate_and_token_gate():
    from sglang_jax_b200 import ops
    x = torch.tensor([[-3., 0.4, 5., 2., -9., 0.3]])
    g, u = torch.tensor([-3., 0.4, 1.]), torch.tensor([1., -1., 0.3])             # clipped at 1
    assert torch.allclose(ops.clipped_swiglu(x, 1.0), g * torch.sigmoid(1.702 * g) * (u + 1), atol=1e-6)
    z, table, ids = torch.randn(2, 3), torch.randn(4, 9), torch.tensor([3, 1], dtype=torch.int32)
    assert torch.allclose(ops.token_side_gate(z, table, ids, 3), oracle.gelu_tanh(z) * table[ids.long(), 3:6], atol=1e-6)


def test_router_chooses_by_logit_and_weighs_the_chosen():
    from sglang_jax_b200.layers.gate import GateLogit
    gate = GateLogit(8, 6, torch.float32, use_bias=True)
    g = torch.Generator().manual_seed(0)
    gate.weight.data.copy_(torch.randn(6, 8, generator=g))
    gate.bias.data.copy_(torch.randn(6, generator=g) * 3)
    x = torch.randn(20, 8, generator=g)
    for top in (1, 3, 6):
        w, ids = gate.route_by_logit(x, top)
        want_ids, want_w = oracle.route(x, {"router": gate.weight, "router.b": gate.bias}, "", top)
        assert torch.equal(ids.long(), want_ids) and torch.allclose(w, want_w, atol=1e-6)


def test_window_keeps_the_first_tokens():
    m = oracle.visible(6, 2, 1)
    assert m.int().tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0], [1, 0, 0, 1, 1, 0],
                                [1, 0, 0, 0, 1, 1]]
    assert oracle.visible(4, None, 0).sum() == 10 and torch.equal(oracle.visible(5, 1, 0), torch.eye(5, dtype=torch.bool))


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
def test_unequal_requests_in_mixed_batches_with_pages_and_slots_used_again(models, name):
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
def needle_model(window, keep_first, seed=3):
    """Two attention layers, the second a reader of the first one's keys, whose last token (48) asks for the marker token
    (49): keys are the first half of a token's embedding, queries the second half, and the two agree for that pair only, so
    that its score stands far above all others and whether that key is seen decides the logits.  The embeddings are large
    beside the position vectors.  The reader's window is half as long and keeps one token more."""
    layers = [cases.attention(2, 2, 16, 16, window, keep_first, scale=1.2),
              cases.attention(2, 2, 16, 16, max(window // 2, 1), keep_first + 1, kv_from=0, scale=1.2)]
    cfg = cases.config(layers, 64, 50, 4)
    w = cases.random_weights(cfg, seed)
    w["embed"] = (w["embed"].float() * 20).bfloat16()
    for p in ("l0.mix.", "l1.mix."):
        pick = torch.zeros(2, 16, 64)
        for h in range(2):
            pick[h, torch.arange(16), torch.arange(16) + 16 * h] = 1.0
        if p + "k" in w:
            w[p + "k"] = pick.reshape(32, 64).bfloat16()
        w[p + "q"] = pick.roll(32, 2).reshape(32, 64).bfloat16()
        w[p + "o"] = (w[p + "o"].float() * 20).bfloat16()
        w[p + "g"] = torch.zeros_like(w[p + "g"])
    w["embed"][48, 32:] = w["embed"][49, :32]
    for i in (0, 1):
        w[f"l{i}.norm1"] = torch.ones_like(w[f"l{i}.norm1"])
    return cfg, w


def needle_prompt(distance, length):
    """The asking token at the end, the marker `distance` tokens before it (0: no marker)."""
    ids = cases.tokens(length, 40, distance)
    ids[-1] = 48
    if distance:
        ids[-1 - distance] = 49
    return ids


@pytest.mark.parametrize("distance", [1, 15, 16, 17, 39, 40, 41, 144, 145, 146, 149])
def test_one_key_decides_inside_the_window_and_among_the_first(tmp_path, distance):
    """Window 40 and 4 first tokens of 150 (the reader: 20 and 5): seen or not, the key shows."""
    cfg, w = needle_model(40, 4)
    ids = needle_prompt(distance, 150)
    without = list(ids)
    without[-1 - distance] = 7
    moved = float(cases.error(oracle.forward(ids, w, cfg)[-1:], oracle.forward(without, w, cfg)[-1:]))
    seen = distance < 40 or 149 - distance < 5
    assert (moved > 0.05) == seen, moved
    path = cases.write(str(tmp_path), cfg, w)
    for steps in ([[("a", 150)]], [[("a", 149)], [("a", 1)]], [[("a", n)] for n in cases.cut(150, [60, 2, 31])]):
        cases.check(path, cfg, w, "float32", "cpu", {"a": ids}, steps, 192, want={"a": cases.expectation(ids, w, cfg)}, page_size=16)


def first_token_model(seed=5):
    """The first tokens' keys stand out from everywhere, so that losing or adding one shows at every later position."""
    layers = [cases.attention(4, 2, 32, 24, 9, 2, scale=2.0), cases.delta(2, 2, 16, 16, 3),
              cases.attention(4, 2, 32, 24, 30, 3, kv_from=0, scale=2.0)]
    cfg = cases.config(layers, 96, 64, 4)
    return cfg, cases.random_weights(cfg, seed)


MISTAKES = ["taps", "order", "state", "conv_start", "shared_head", "own_key", "window_short", "window_long", "keep_less",
            "keep_more", "no_key_norm", "gate", "position", "side_slice", "router_all", "limit", "parallel", "decay_per_head",
            "reader_keys"]


@pytest.mark.parametrize("wrong", MISTAKES)
def test_the_oracle_tells_planted_mistakes_apart(models, wrong, monkeypatch):
    """A mistake planted in the oracle moves the logits by far more than the tests' limits."""
    _, cfg, w = models["plain"]
    ids = cases.tokens(40, cfg["vocab"], 9)
    good = oracle.forward(ids, w, cfg)
    was = {n: getattr(oracle, n) for n in ("causal_conv", "channel_delta_recurrence", "masked_attention", "visible", "rms",
                                           "position_vectors", "token_side", "route", "clipped_expert", "channel_decay")}
    conv, rec, att, see = was["causal_conv"], was["channel_delta_recurrence"], was["masked_attention"], was["visible"]
    put = lambda n, f: monkeypatch.setattr(oracle, n, f)
    if wrong == "taps":
        put("causal_conv", lambda x, k: conv(x, k.flip(1)))
    elif wrong == "order":        # the read-out before the write
        def before(*a):
            o = rec(*a)
            return torch.cat([torch.zeros_like(o[:1]), o[:-1]])
        put("channel_delta_recurrence", before)
    elif wrong == "state":        # lost at token 20
        put("channel_delta_recurrence", lambda *a: torch.cat([rec(*(t[:20] for t in a)), rec(*(t[20:] for t in a))]))
    elif wrong == "conv_start":   # the convolution starts anew at token 20
        put("causal_conv", lambda x, k: torch.cat([conv(x[:20], k), conv(x[20:], k)]))
    elif wrong == "shared_head":
        put("masked_attention", lambda q, k, v, s, m: att(q, k.flip(1), v.flip(1), s, m))
    elif wrong == "own_key":      # every token sees its predecessor's key in the place of its own
        put("masked_attention", lambda q, k, v, s, m: att(q, k.roll(1, 0), v.roll(1, 0), s, m))
    elif wrong in ("window_short", "window_long"):
        put("visible", lambda T, n, f: see(T, n + (1 if wrong == "window_long" else -1), f))
    elif wrong in ("keep_less", "keep_more"):
        put("visible", lambda T, n, f: see(T, n, max(f + (1 if wrong == "keep_more" else -1), 0)))
    elif wrong == "no_key_norm":
        put("rms", lambda x, eps: x if x.dim() == 3 else was["rms"](x, eps))
    elif wrong == "gate":
        w = {**w, "l0.mix.g": torch.zeros_like(w["l0.mix.g"])}
    elif wrong == "position":
        put("position_vectors", lambda p, *a: was["position_vectors"](p + 1, *a))
    elif wrong == "side_slice":
        put("token_side", lambda x, t, w, i, d, e: was["token_side"](x, t, {**w, "side.embed": w["side.embed"].roll(d, 1)}, i, d, e))
    elif wrong == "router_all":   # weights from the softmax over all experts
        def all_of_them(h, w, p, top):
            ids, c = was["route"](h, w, p, top)
            return ids, torch.softmax(h @ w[p + "router"].T + w[p + "router.b"], -1).gather(1, ids)
        put("route", all_of_them)
    elif wrong == "limit":
        put("clipped_expert", lambda h, g, u, d, limit: was["clipped_expert"](h, g, u, d, 1.5 * limit))
    elif wrong == "parallel":     # the feed-forward behind the mixer
        def serial(x, tokens, w, i, entry, cfg, shared):
            alone = oracle_layer(x, tokens, w, i, dict(entry, mlp=None), cfg, shared)
            h = was["rms"](alone, cfg["norm"]["eps"]) * w[f"l{i}.norm1"]
            return alone + oracle.sparse_ff(h, w, f"l{i}.mlp.", entry["mlp"])
        oracle_layer = oracle.layer
        put("layer", serial)
    elif wrong == "decay_per_head":
        put("channel_decay", lambda *a: was["channel_decay"](*a).mean(-1, keepdim=True).expand(-1, -1, a[-1]))
    elif wrong == "reader_keys":  # readers look one token back in the keys they share
        def late(q, k, v, s, m, seen=[]):
            first = not any(k is x for x in seen)
            seen.append(k)
            return att(q, k, v, s, m) if first else att(q, k.roll(1, 0), v, s, m)
        put("masked_attention", late)
    assert float(cases.error(oracle.forward(ids, w, cfg), good).max()) > 1e-2


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


@pytest.mark.parametrize("name", ["mixed", "odd", "delta_only", "attention_only"])
def test_greedy_generation_of_every_layout(models, name):
    path, cfg, w = models[name]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (20, 5)]
    eng = _engine(path)
    try:
        got = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 5, **GREEDY})
        assert [o["output_ids"] for o in got] == [oracle.greedy(p, w, cfg, 5) for p in prompts]
    finally:
        eng.shutdown()


@pytest.mark.parametrize("name", ["plain", "mixed", "attention_only"])
def test_shared_prefixes(models, name):
    """With recurrent layers from a checkpoint of the state, without them from the keys and values alone."""
    path, cfg, w = models[name]
    base = cases.tokens(70, cfg["vocab"], 1)
    sp = {"max_new_tokens": 4, **GREEDY}
    eng = _engine(path, recurrent_snapshot_slots=16)
    try:
        eng.generate(input_ids=base, sampling_params=sp)
        again = base[:66] + cases.tokens(20, cfg["vocab"], 2)
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
        top = torch.topk(oracle.forward(ids, w, cfg)[-1], 5).indices.tolist()
        assert out["output_ids"][0] in top
        lp = torch.log_softmax(oracle.forward(ids, w, cfg), -1)
        want = [float(lp[i, ids[i + 1]]) for i in range(29)]
        got = [x[0] for x in out["meta_info"]["input_token_logprobs"] if x[0] is not None]
        assert np.allclose(got, want, atol=1e-3)
    finally:
        eng.shutdown()


# ------------------------------------------------------------------ configuration, loading, pools
def test_unknown_parts_of_a_configuration_are_refused(tmp_path):
    from sglang_jax_b200.configs.model_config import ModelConfig
    good = cases.checkpoint_config(cases.CONFIGS["plain"])
    first = good["layers"][0]
    for change in ({"layers": [dict(first, type="window")]}, {"layers": [dict(first, mlp={"kind": "dense"})]},
                   {"layers": [first, dict(first, mixer=dict(first["mixer"], kv_from=1))]},
                   {"layers": [good["layers"][1], dict(first, mixer=dict(first["mixer"], kv_from=0))]}):
        (tmp_path / "config.json").write_text(json.dumps({**good, **change}))
        with pytest.raises(ValueError):
            ModelConfig(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps(good))
    mc = ModelConfig(str(tmp_path), context_length=100_000)           # positions have no limit of their own
    assert mc.architectures == ["ZidivikForCausalLM"] and mc.context_len == 100_000 and mc.num_experts == 6


def test_widths_that_only_the_tensors_tell(models):
    from sglang_jax_b200.configs.model_config import ModelConfig
    path, cfg, _ = models["mixed"]
    mc = ModelConfig(path)
    assert [(l["mixer"]["decay_rank"], l["mixer"]["gate_rank"]) for l in mc.hf_config.layers if l["type"] == "channel_delta"] \
        == [e["ranks"] for e in cfg["layers"] if e["type"] == "channel_delta"]


@pytest.mark.parametrize("change", ["missing", "unexpected", "reader_keys"])
def test_checkpoints_must_be_complete(tmp_path, change):
    cfg = cases.CONFIGS["plain"]
    w = cases.random_weights(cfg)
    if change == "missing":
        w.pop("l1.mix.dt_bias")
    else:
        w["l1.mix.bias" if change == "unexpected" else "l2.mix.k"] = torch.zeros(4)
    path = cases.write(str(tmp_path), cfg, w)
    with pytest.raises(RuntimeError, match="missing|unexpected"):
        cases.replay(path, "float32", "cpu", {}, [], 64)


def test_pool_of_packed_rows():
    from sglang_jax_b200.mem_cache.memory_pool import PackedKVPool
    shapes = [(2, 48, 7), (1, 10, 16)]
    kv = PackedKVPool(64, 16, torch.float32, shapes, "cpu")
    assert [tuple(b.shape) for b in kv.kv_buffer] == [(5, 2, 16, 56), (5, 1, 16, 32)]
    assert kv.get_kv_size_bytes() == 5 * 16 * PackedKVPool.cell_size(shapes, torch.float32)
    src, dst = torch.tensor([17, 63, 5]), torch.tensor([2, 70, 33])
    want = []
    for i, (h, k, v) in enumerate(shapes):
        want.append((torch.randn(3, h, k), torch.randn(3, h, v)))
        kv.set_kv_buffer(i, src, *want[-1])
    kv.move_kv(src, dst)
    for i in range(2):
        for loc in (src, dst):
            assert all(torch.equal(a, b) for a, b in zip(kv.gather(i, loc), want[i]))


def test_readers_take_no_cache_of_their_own(models):
    from sglang_jax_b200.configs.model_config import ModelConfig
    from sglang_jax_b200.models.registry import get_model_class
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    mc = ModelConfig(models["mixed"][0])
    m = get_model_class(mc.architectures)(mc.hf_config, dtype=torch.float32)
    assert m.kv_layer_shapes == [(3, 24, 40), (1, 40, 24)]
    assert [l.mix.layer_id for l in m.layers if not l.is_delta] == [0, 1, 1]


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


@pytest.mark.parametrize("heads", [2, 1])
def test_two_tensor_ranks_generate_what_one_does(models, tmp_path, heads):
    """Key heads split over the ranks, and one key head that both hold."""
    import torch.multiprocessing as mp
    from sglang_jax_b200.utils.common import get_free_port
    path, cfg, w = models["plain"]
    if heads == 1:
        cfg = cases.config([cases.attention(4, 1, 32, 24, 24, 3, mlp=cases.moe(48, 6, 2)),
                            cases.attention(2, 1, 32, 24, 50, 1, kv_from=0)], 128, 200, 8)
        w = cases.random_weights(cfg, 3)
        path = cases.write(str(tmp_path), cfg, w)
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (21, 40)]
    ctx = mp.get_context("spawn")
    q, port = ctx.Queue(), get_free_port()
    procs = [ctx.Process(target=_tp_rank, args=(r, 2, port, path, prompts, {}, q)) for r in range(2)]
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
