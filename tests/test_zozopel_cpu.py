"""Zozopel on the CPU: every mechanism against the oracle, schedules, caches, loading and generation through the engine."""

import json

import numpy as np
import pytest
import torch

import zozopel_cases as cases
import zozopel_oracle as oracle


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in cases.CONFIGS.items():
        w = cases.random_weights(cfg, seed=len(name))
        out[name] = (cases.write_checkpoint(str(tmp_path_factory.mktemp(name)), cfg, w), cfg, w)
    return out


# ------------------------------------------------------------------ mechanisms alone
def test_stream_ops_against_the_oracle():
    from sglang_jax_b200 import ops
    g = torch.Generator().manual_seed(0)
    x, y = torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g) * 3
    w, ls = torch.randn(24, generator=g), torch.randn(24, generator=g)
    table, ids = torch.randn(11, 24, generator=g), torch.tensor([3, 0, 10, 3, 7], dtype=torch.int32)
    s, h = ops.embed_scaled(ids, table, 0.3)
    assert torch.equal(s, table[ids.long()] * 0.3) and h is s
    want = x.double() + 0.7 * oracle.rms(y.double(), 1e-3) * w.double() * ls.double()
    ops.postnorm_add(y, x, w * ls * 0.7, 1e-3)
    assert torch.allclose(x.double(), want, atol=1e-5)
    assert torch.allclose(ops.rmsnorm_stream(x, w, 1e-3, torch.float32).double(), oracle.rms(want, 1e-3) * w.double(), atol=1e-5)
    ab = torch.randn(5, 30, generator=g) * 3
    assert torch.allclose(ops.gelu_and_mul(ab), oracle.gelu_tanh(ab[:, :15]) * ab[:, 15:], atol=1e-5)
    o = torch.randn(5, 15, generator=g)
    assert torch.allclose(ops.sigmoid_gate(o, ab[:, 4:19]), o * torch.sigmoid(ab[:, 4:19]), atol=1e-6)


def test_post_norm_module_folds_weight_layer_scale_and_multiplier():
    from sglang_jax_b200.layers.layernorm import PostNormResidual
    n = PostNormResidual(8, 1e-6, 0.25, True, torch.float32)
    n.weight.data.copy_(torch.arange(1., 9.))
    n.layer_scale.data.fill_(3.0)
    n.fold()
    assert torch.allclose(n.channel_scale, torch.arange(1., 9.) * 0.75)


def test_rotation_is_interleaved_and_exact():
    from sglang_jax_b200.layers.embeddings import get_rope
    from sglang_jax_b200.ops import reference
    cs = get_rope(12, 12, 4000, 777.0, False, {"rope_type": "exact"}).cos_sin_cache
    x, pos = torch.randn(3, 2, 12), torch.tensor([0, 1, 3999])
    assert torch.allclose(reference.apply_rope(x, pos, cs, False).double(), oracle.rotate(x.double(), pos, 777.0), atol=5e-4)
    assert torch.equal(reference.apply_rope(x[:1], pos[:1], cs, False), x[:1])


@pytest.mark.parametrize("name", list(cases.CONFIGS))
def test_whole_prompts_match_the_oracle(models, name):
    path, cfg, w = models[name]
    reqs = {n: cases.tokens(n, cfg["vocab"], n) for n in (1, 2, 75)}
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


def test_the_last_page_of_the_pool_is_usable_and_no_more(models):
    path, cfg, w = models["plain"]
    reqs = {"a": cases.tokens(128, cfg["vocab"], 1)}
    cases.check(path, cfg, w, "float32", "cpu", reqs, [[("a", 127)], [("a", 1)]], 128)
    with pytest.raises(RuntimeError):
        cases.replay(path, "float32", "cpu", {"a": reqs["a"] + [1]}, [[("a", 129)]], 128)


# ------------------------------------------------------------------ what random weights would hide
def needle_model(seed=3):
    """One latent layer whose last token (48) asks for the marker token (49): keys are the first half of a token's
    embedding, queries the second half, and the two agree for that pair only, so that its score stands far above all
    others and whether that key is seen decides the logits."""
    cfg = cases.config([cases.latent(2, 16, 8, 16, 32, scale=4.0)], 64, 50)
    w = cases.random_weights(cfg, seed)
    p = "l0.mix."
    ident = torch.zeros(32, 64)
    ident[torch.arange(32), torch.arange(32)] = 1.0
    w[p + "dkv"] = torch.cat([ident, torch.zeros(8, 64)]).bfloat16()          # the latent is half of the embedding
    uk = torch.zeros(2, 16, 32)
    for h in range(2):
        uk[h, torch.arange(16), torch.arange(16) + 16 * h] = 1.0
    w[p + "uk"] = uk.reshape(32, 32).bfloat16()
    q = torch.zeros(2, 24, 64)
    for h in range(2):
        q[h, torch.arange(16), torch.arange(16) + 16 * h + 32] = 1.0
    w[p + "q"] = q.reshape(48, 64).bfloat16()
    w["embed"][48, 32:] = w["embed"][49, :32]
    return cfg, w


def needle_prompt(distance, length):
    """The asking token at the end, the marker `distance` tokens before it."""
    ids = cases.tokens(length, 40, distance)
    ids[-1], ids[-1 - distance] = 48, 49
    return ids


@pytest.mark.parametrize("distance", [1, 15, 16, 17, 63, 64, 65, 127, 128, 149])
def test_one_far_key_decides(tmp_path, distance):
    cfg, w = needle_model()
    ids = needle_prompt(distance, 150)
    with_key = oracle.forward(ids, w, cfg)
    ids2 = list(ids)
    ids2[-1 - distance] = 7
    assert float(cases.error(with_key[-1:], oracle.forward(ids2, w, cfg)[-1:])) > 0.05        # it shows
    path = cases.write_checkpoint(str(tmp_path), cfg, w)
    for steps in ([[("a", 150)]], [[("a", 149)], [("a", 1)]], [[("a", n)] for n in cases.cut(150, [60, 2, 31])]):
        cases.check(path, cfg, w, "float32", "cpu", {"a": ids}, steps, 192, want={"a": cases.expectation(ids, w, cfg)}, page_size=16)


@pytest.mark.parametrize("wrong", ["taps", "order", "state", "shared_head", "own_key", "window"])
def test_the_oracle_tells_planted_mistakes_apart(models, wrong, monkeypatch):
    """A mistake planted in the oracle moves the logits by far more than the tests' limits."""
    _, cfg, w = models["plain"]
    ids = cases.tokens(40, cfg["vocab"], 9)
    good = oracle.forward(ids, w, cfg)
    conv, rec, lat = oracle.causal_conv, oracle.delta_recurrence, oracle.softmax_attention
    if wrong == "taps":
        monkeypatch.setattr(oracle, "causal_conv", lambda x, k: conv(x, k.flip(1)))
    elif wrong == "order":        # the read-out before the write
        def before(q, k, v, decay, beta):
            o = rec(q, k, v, decay, beta)
            return torch.cat([torch.zeros_like(o[:1]), o[:-1]])
        monkeypatch.setattr(oracle, "delta_recurrence", before)
    elif wrong == "state":        # lost at token 20
        monkeypatch.setattr(oracle, "delta_recurrence",
                            lambda *a: torch.cat([rec(*(t[:20] for t in a)), rec(*(t[20:] for t in a))]))
    elif wrong == "window":       # the convolution starts anew at token 20
        monkeypatch.setattr(oracle, "causal_conv", lambda x, k: torch.cat([conv(x[:20], k), conv(x[20:], k)]))
    elif wrong == "shared_head":
        monkeypatch.setattr(oracle, "delta_recurrence", lambda q, k, v, d, b: rec(q.flip(1), k.flip(1), v, d, b))
    else:                         # every token sees its predecessor's key in the place of its own
        monkeypatch.setattr(oracle, "softmax_attention", lambda q, k, v, s: lat(q, k.roll(1, 0), v.roll(1, 0), s))
    assert float(cases.error(oracle.forward(ids, w, cfg), good).max()) > 1e-2


# ------------------------------------------------------------------ engine
def _engine(path, **kw):
    from sglang_jax_b200 import Engine
    from sglang_jax_b200.parallel import state as ps
    ps.reset_state()
    return Engine(model_path=path, skip_tokenizer_init=True, enable_single_process=True,
                  **{"device": "cpu", "dtype": "float32", "page_size": 16, "max_total_tokens": 2048, **kw})


PROMPTS = [29, 7, 70, 33]


@pytest.mark.parametrize("kw", [dict(), dict(chunked_prefill_size=16), dict(disable_overlap_schedule=True),
                                dict(chunked_prefill_size=32, enable_mixed_chunk=True),
                                dict(max_total_tokens=176, disable_overlap_schedule=True)])
def test_greedy_generation_through_the_engine(models, kw):
    path, cfg, w = models["plain"]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in PROMPTS]
    want = [oracle.greedy(p, w, cfg, 8) for p in prompts]
    eng = _engine(path, **kw)
    try:
        got = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 8, "temperature": 0, "ignore_eos": True})
        assert [o["output_ids"] for o in got] == want
        eng.scheduler.check_memory()
    finally:
        eng.shutdown()


@pytest.mark.parametrize("name", ["mixed", "odd", "delta_only", "latent_only"])
def test_greedy_generation_of_every_layout(models, name):
    path, cfg, w = models[name]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (20, 5)]
    eng = _engine(path)
    try:
        got = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 5, "temperature": 0, "ignore_eos": True})
        assert [o["output_ids"] for o in got] == [oracle.greedy(p, w, cfg, 5) for p in prompts]
    finally:
        eng.shutdown()


@pytest.mark.parametrize("name", ["plain", "mixed"])
def test_shared_prefixes_restart_from_state_checkpoints(models, name):
    path, cfg, w = models[name]
    base = cases.tokens(70, cfg["vocab"], 1)
    sp = {"max_new_tokens": 4, "temperature": 0, "ignore_eos": True}
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
    good = cases.CONFIGS["plain"]
    for change in ({"architecture": "Other"}, {"layers": [dict(good["layers"][0], type="window")]},
                   {"layers": [dict(good["layers"][0], mlp={"kind": "sparse"})]}):
        (tmp_path / "config.json").write_text(json.dumps({**good, **change}))
        with pytest.raises(ValueError):
            ModelConfig(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps(good))
    mc = ModelConfig(str(tmp_path), context_length=100_000)           # positions have no limit of their own
    assert mc.architectures == ["ZozopelForCausalLM"] and mc.context_len == 100_000


@pytest.mark.parametrize("change", ["missing", "unexpected"])
def test_checkpoints_must_be_complete(tmp_path, change):
    cfg = cases.CONFIGS["plain"]
    w = cases.random_weights(cfg)
    if change == "missing":
        w.pop("l1.mix.dt_bias")
    else:
        w["l1.mix.bias"] = torch.zeros(4)
    path = cases.write_checkpoint(str(tmp_path), cfg, w)
    with pytest.raises(RuntimeError, match="missing|unexpected"):
        cases.replay(path, "float32", "cpu", {}, [], 64)


def test_pools_with_a_size_per_layer():
    from sglang_jax_b200.mem_cache.memory_pool import MLATokenToKVPool
    from sglang_jax_b200.mem_cache.recurrent_state_pool import RecurrentStatePool, slot_bytes
    dims = [(48, 8), (21, 6)]
    kv = MLATokenToKVPool(64, 16, torch.float32, 48, 8, 2, "cpu", layer_dims=dims)
    assert [b.shape[-1] for b in kv.kv_buffer] == [56, 32]
    assert kv.get_kv_size_bytes() == 5 * 16 * MLATokenToKVPool.cell_size(0, 0, 2, torch.float32, layer_dims=dims)
    loc = torch.tensor([17, 63])
    for i, (r, p) in enumerate(dims):
        c, pe = torch.randn(2, r), torch.randn(2, p)
        kv.set_kv_buffer(i, loc, c, pe)
        got = kv.gather(i, loc)
        assert torch.equal(got[0], c) and torch.equal(got[1], pe)
    layers = [dict(conv_dim=10, conv_kernel=4, num_heads=2, head_k_dim=3, head_v_dim=5),
              dict(conv_dim=6, conv_kernel=2, num_heads=1, head_k_dim=4, head_v_dim=2)]
    for spec in (dict(layers=layers), dict(num_layers=2, **layers[0])):
        pool = RecurrentStatePool(3, device="cpu", snapshot_slots=2, **spec)
        assert pool.size_bytes() == 6 * slot_bytes(**spec)
        for i in range(2):
            pool.conv_state[i][1] = 1.0 + i
            pool.recurrent_state[i][1] = 5.0 + i
        pool.copy_slots([1], [4])
        pool.copy_sequence([(4, 5), (5, 2)])
        pool.clear_slots([1])
        for i in range(2):
            assert (pool.conv_state[i][2] == 1.0 + i).all() and (pool.recurrent_state[i][5] == 5.0 + i).all()
            assert (pool.conv_state[i][1] == 0).all() and (pool.recurrent_state[i][3] == 0).all()


def _tp_rank(rank, world, port, path, prompts, q):
    from sglang_jax_b200.parallel import state as ps
    from sglang_jax_b200.server_args import ServerArgs
    torch.set_num_threads(2)
    ps.init_distributed(rank, world, "cpu", init_method=f"tcp://127.0.0.1:{port}", timeout_s=120)
    sa = ServerArgs(model_path=path, device="cpu", dtype="float32", page_size=16, skip_tokenizer_init=True,
                    max_total_tokens=1024, enable_single_process=True, max_running_requests=8, tp_size=world,
                    log_level="error", watchdog_timeout=0)
    if rank:
        from sglang_jax_b200.managers.tp_worker import run_tp_follower
        run_tp_follower(sa)
    else:
        from sglang_jax_b200 import Engine
        eng = Engine(server_args=sa)
        outs = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 8, "temperature": 0, "ignore_eos": True})
        q.put([o["output_ids"] for o in outs])
        eng.shutdown()
    ps.destroy()


def test_two_tensor_ranks_generate_what_one_does(models):
    import torch.multiprocessing as mp
    from sglang_jax_b200.utils.common import get_free_port
    path, cfg, w = models["plain"]
    prompts = [cases.tokens(n, cfg["vocab"], n) for n in (21, 40)]
    ctx = mp.get_context("spawn")
    q, port = ctx.Queue(), get_free_port()
    procs = [ctx.Process(target=_tp_rank, args=(r, 2, port, path, prompts, q)) for r in range(2)]
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
