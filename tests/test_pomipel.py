"""Pomipel: the configuration and checkpoint, each mechanism, and whole models through the engine's scheduler, cache and
model runner, against the plain implementation (tests/pomipel_oracle.py).

Whole-model tests run on the CPU, and on the device in 16 and in 32 bits."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from tests import pomipel_oracle as po
from tests.replay_utils import PLACES, TOL, Engine, check_greedy, generate, make_llm, portions

@pytest.fixture(autouse=True)
def _few_threads():
    """The models are tiny: more threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(min(n, 2))
    yield
    torch.set_num_threads(n)


@pytest.fixture(params=PLACES)
def place(request):
    return request.param


def _model(tmp_path, cfg, seed=0, place=("cpu", "float32"), plant=None, **kw):
    w = po.make_weights(cfg, seed, steady=place[1] == "bfloat16", **kw)
    if plant:
        po.plant_key(cfg, w, *plant)
    return po.save_model(cfg, w, tmp_path / "model"), w


# ------------------------------------------------------------------------------------------------ configuration and checkpoint
def test_configuration_is_read_from_the_model_folder(tmp_path):
    from vllm_b200.config import ModelConfig
    from vllm_b200.models.registry import resolve_model_cls
    cfg = po.small(max_positions=300)
    path, _ = _model(tmp_path, cfg)
    mc = ModelConfig(model=path)
    assert mc.architecture == "PomipelForCausalLM" and mc.is_mla and mc.is_moe
    assert (mc.vocab_size, mc.hidden_size, mc.num_layers, mc.max_model_len) == (208, 96, 4, 300)
    assert resolve_model_cls(mc.architecture).__name__ == "PomipelForCausalLM"
    assert mc.torch_dtype == torch.bfloat16


@pytest.mark.parametrize("change", [lambda c: c["layers"][2]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_from=3),
                                    lambda c: c["layers"][0]["mixer"].update(kv_from=1), lambda c: c["layers"][3]["mixer"].update(kv_from=2),
                                    lambda c: c["layers"][2]["mixer"].update(kv_rank=32)])
def test_a_shared_latent_needs_an_owner_of_the_same_width(change):
    from vllm_b200.config import ModelConfig
    cfg = po.small()
    change(cfg)
    with pytest.raises(ValueError, match="kv_from"):
        ModelConfig(model="x", hf_config=cfg, hf_overrides={})


def test_router_sizes_are_checked():
    from vllm_b200.layers.moe import GroupedRouter
    for top, count, keep in ((9, 4, 2), (2, 3, 2), (2, 4, 5), (5, 4, 2)):
        with pytest.raises(ValueError):
            GroupedRouter(16, 8, top, torch.float32, count, keep)


def test_checkpoint_names_are_all_taken_and_none_else(tmp_path):
    from vllm_b200.engine.replay import StepReplay
    cfg = po.small()
    path, w = _model(tmp_path, cfg)
    r = StepReplay(path, "float32", 256, device="cpu", max_model_len=256)
    model = r.core.model_executor.worker.get_model()
    loaded = model.load_weights((k, v.clone()) for k, v in w.items())
    assert loaded == {n for n, _ in model.named_parameters()}
    for bad in ("l0.mix.foo", "l2.mix.dkv", "l9x.norm1", "other"):
        with pytest.raises(ValueError):
            model.load_weights([(bad, torch.zeros(48, 96))])
    r.shutdown()


def test_more_positions_than_the_model_has_is_an_error(tmp_path):
    from vllm_b200 import LLM
    path, _ = _model(tmp_path, po.small(max_positions=100))
    with pytest.raises(Exception, match="learned positions"):
        LLM(path, device="cpu", dtype="float32", max_model_len=101, kv_cache_memory_bytes=16 << 20, skip_tokenizer_init=True)


def test_layers_with_a_shared_latent_own_no_cache(tmp_path):
    path, _ = _model(tmp_path, po.small())
    with Engine(path, ("cpu", "float32"), 256, max_model_len=256) as e:
        runner = e.replay.core.model_executor.worker.runner
        assert sorted(runner.kv_caches) == ["model.layers.0.mixer.attn", "model.layers.1.mixer.attn"]
        assert sorted(c.shape[-1] for c in runner.kv_caches.values()) == [32, 48]      # the latent and nothing else


# ------------------------------------------------------------------------------------------------ mechanisms (plain ops)
def test_stream_entry_and_post_norm():
    from vllm_b200.ops import ref
    cfg = po.small()
    w = po.make_weights(cfg, 1)
    toks = po.tokens(cfg, 9)
    where = torch.arange(4, 13)
    x, h = ref.embed_stream(torch.tensor(toks), where, w["embed"], w["pos"], 3.0)
    want = po.embed(toks, w["embed"].double(), w["pos"].double(), 3.0, start=4)
    torch.testing.assert_close(x.double(), want, rtol=1e-6, atol=1e-6)
    y = torch.randn(9, 96)
    h = ref.post_norm_add(x, y, w["l0.norm1"], 1e-5, True, w["final.norm"], True)
    want = want + po.centred_norm(y.double(), w["l0.norm1"].double(), 1e-5)
    torch.testing.assert_close(x.double(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(h.double(), po.centred_norm(want, w["final.norm"].double(), 1e-5), rtol=1e-5, atol=1e-5)


def test_the_stream_keeps_what_16_bits_would_lose():
    from vllm_b200.ops import ref
    x = torch.full((1, 64), 256.0)
    for _ in range(8):                                        # eight steps of 1/8: each is below bfloat16's step at 256
        ref.post_norm_add(x, torch.ones(1, 64, dtype=torch.bfloat16), torch.full((64,), -0.875, dtype=torch.bfloat16), 1e-6, True)
    torch.testing.assert_close(x, torch.full((1, 64), 257.0), rtol=0, atol=1e-3)


@pytest.mark.parametrize("E,top,count,keep", [(8, 2, 4, 2), (12, 5, 3, 2), (6, 3, 2, 1), (5, 2, 5, 4), (4, 1, 1, 1), (9, 9, 3, 3)])
def test_router_choice_and_weights(E, top, count, keep):
    from vllm_b200 import ops
    g = torch.Generator().manual_seed(E * top)
    x, w = torch.randn(40, 24, generator=g), torch.randn(E, 24, generator=g) / 5
    corr = torch.randn(E, generator=g) * 0.8 - 1.0            # choice scores are mostly negative: masked ones must not win
    wt, ids = ops.router_topk(x, w, top, count, keep, False, "sigmoid", corr)
    for t in range(40):
        want = po.route(x[t].double(), w.double(), corr.double(), top, count, keep)
        assert sorted(ids[t].tolist()) == sorted(e for e, _ in want)
        got = dict(zip(ids[t].tolist(), wt[t].tolist()))
        for e, s in want:
            assert abs(got[e] - s) < 1e-5                      # the plain score, whatever the correction


def test_ungated_experts():
    from vllm_b200 import ops
    g = torch.Generator().manual_seed(3)
    x, up, down = torch.randn(7, 20, generator=g), torch.randn(4, 12, 20, generator=g), torch.randn(4, 20, 12, generator=g)
    ids, wt = torch.randint(0, 4, (7, 2), generator=g), torch.rand(7, 2, generator=g)
    got = ops.fused_moe(x, up, down, wt, ids, "relu2", None, gated=False)
    for t in range(7):
        want = sum(wt[t, s].double() * po.expert(x[t].double(), up[ids[t, s]].double(), down[ids[t, s]].double()) for s in range(2))
        torch.testing.assert_close(got[t].double(), want, rtol=1e-4, atol=1e-3)


def test_stream_after_every_layer(tmp_path):
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 2)
    toks = po.tokens(cfg, 30)
    want = []
    po.forward(cfg, w, toks, layers=want)
    with Engine(path, ("cpu", "float32"), 256, max_model_len=256) as e:
        got = []
        for layer in e.replay.core.model_executor.worker.get_model().model.layers:
            layer.register_forward_hook(lambda mod, args, out: got.append(args[0].clone()))
        e.feed([("a", toks, True)])
        for g_, w_ in zip(got, want):
            torch.testing.assert_close(g_.double(), w_, rtol=1e-4, atol=1e-4)
        assert len(got) == 4


# ------------------------------------------------------------------------------------------------ whole models
MODELS = {"small": po.small, "uneven": po.uneven, "wide": po.wide}


@pytest.mark.parametrize("name", sorted(MODELS))
def test_prompt_token_by_token_and_portions_agree_with_the_equations(tmp_path, place, name):
    cfg = MODELS[name]()
    path, w = _model(tmp_path, cfg, 3, place)
    toks = po.tokens(cfg, 150)                                 # three pages
    want = po.forward(cfg, w, toks)
    tol = TOL[place[1]]
    with Engine(path, place) as e:
        e.feed([("whole", toks, True)])
        assert po.row_error(e.logits("whole"), want) < tol
        e.feed(*[[("single", [t], i == 149)] for i, t in enumerate(toks)])
        assert po.row_error(e.logits("single"), want) < tol
        for k, sizes in enumerate([(2,), (3, 2, 5), (63, 2, 64, 2), (17, 1, 1, 40), (16, 17, 65), (100, 2, 1)]):
            parts = portions(toks, sizes)
            e.feed(*[[(f"p{k}", p, i == len(parts) - 1)] for i, p in enumerate(parts)])
            assert po.row_error(e.logits(f"p{k}"), want) < tol, sizes


def test_first_tokens(tmp_path, place):
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 4, place)
    with Engine(path, place) as e:
        for n in (1, 2, 3):
            toks = po.tokens(cfg, n, n)
            e.feed([("a", toks, True)])
            assert po.row_error(e.logits("a"), po.forward(cfg, w, toks)) < TOL[place[1]]
        same = [7, 7, 7]                                       # equal tokens differ by their learned positions alone
        e.feed([("b", same, True)])
        assert po.row_error(e.logits("b"), po.forward(cfg, w, same)) < TOL[place[1]]


def test_unequal_requests_in_one_batch(tmp_path, place):
    """Portions beside single tokens; every request as if it were alone."""
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 5, place)
    reqs = {"a": po.tokens(cfg, 140, 1), "b": po.tokens(cfg, 9, 2), "c": po.tokens(cfg, 75, 3), "d": po.tokens(cfg, 33, 4)}
    sizes = {"a": (70, 1, 2, 67), "b": (1,), "c": (2, 40, 1), "d": (33,)}
    parts = {r: portions(t, sizes[r]) for r, t in reqs.items()}
    starts = {"a": 0, "b": 0, "c": 1, "d": 3}
    steps = []
    for n in range(40):
        step = []
        for r in ("c", "a", "d", "b"):
            i = n - starts[r]
            if r == "b" and n in (2, 3):                       # left out of two steps
                continue
            if r == "b" and n > 3:
                i -= 2
            if 0 <= i < len(parts[r]):
                step.append((r, parts[r][i], i == len(parts[r]) - 1))
        if step:
            steps.append(step)
    with Engine(path, place) as e:
        e.feed(*steps)
        for r, t in reqs.items():
            assert po.row_error(e.logits(r), po.forward(cfg, w, t)) < TOL[place[1]], r


def test_pages_and_rows_are_used_again(tmp_path, place):
    """A pool of five pages serves many requests one after another; a new one never sees what a page held before."""
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 6, place)
    with Engine(path, place, 5 * 64) as e:
        mgr = e.replay.core.scheduler.kv_cache_manager
        free = mgr.pool.get_num_free_blocks()
        assert free == 5
        keep = po.tokens(cfg, 100, 50)                         # stays while the others come and go
        e.feed([("keep", keep[:60])])
        for k in range(6):
            n = (64, 65, 130, 2, 128, 127)[k]
            toks = po.tokens(cfg, n, k)
            cut = max(1, n // 2)
            e.feed([(f"r{k}", toks[:cut]), ("keep", keep[60 + 6 * k:66 + 6 * k])], [(f"r{k}", toks[cut:], True)])
            assert po.row_error(e.logits(f"r{k}"), po.forward(cfg, w, toks)) < TOL[place[1]], k
        e.feed([("keep", keep[96:], True)])
        assert po.row_error(e.logits("keep"), po.forward(cfg, w, keep)) < TOL[place[1]]
        assert mgr.pool.get_num_free_blocks() == free


def test_a_pool_that_is_too_small_is_an_error(tmp_path):
    path, _ = _model(tmp_path, po.small())
    with Engine(path, ("cpu", "float32"), 128) as e:
        e.feed([("a", [1] * 64), ("b", [1] * 64)])
        with pytest.raises(RuntimeError, match="no room"):
            e.feed([("a", [2])])


@pytest.mark.parametrize("where", [0, 1, 62, 63, 64, 65, 127, 128, 191, 192])
def test_a_far_key_is_seen(tmp_path, place, where):
    """One key far above the noise, at page borders and elsewhere; the query in a prompt, in a short portion and decoded."""
    cfg = po.small()
    X, Q = 11, 12
    path, w = _model(tmp_path, cfg, 7, place, plant=(X, Q), pos_size=0.02)
    toks = po.tokens(cfg, 199, where, avoid=(X, Q)) + [Q]
    toks[where] = X
    want = po.forward(cfg, w, toks)
    blind = po.row_error(po.forward(cfg, w, toks, hide=(where,))[-1:], want[-1:])
    tol = TOL[place[1]]
    assert blind > 4 * tol                                     # without that one key the logits are others
    with Engine(path, place) as e:
        e.feed([("whole", toks, True)])
        e.feed([("cut", toks[:-2])], [("cut", toks[-2:], True)])
        e.feed([("dec", toks[:-1])], [("dec", toks[-1:], True)])
        for r in ("whole", "cut", "dec"):
            assert po.row_error(e.logits(r)[-1:], want[-1:]) < tol, r


def test_no_query_sees_what_comes_after_it(tmp_path, place):
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 8, place)
    a, b = po.tokens(cfg, 140, 1), po.tokens(cfg, 140, 2)
    b[:70] = a[:70]
    with Engine(path, place) as e:
        e.feed([("a", a, True)], [("b", b, True)])
        la, lb = e.logits("a"), e.logits("b")
        assert po.row_error(la[:70], lb[:70]) < 1e-5 and po.row_error(la[70:], lb[70:]) > 0.3


def test_long_decoding(tmp_path, place):
    cfg = po.config(64, 96, [(po.mixer(2, 24, 16, 32, 40), po.moe(24, 6, 2, 3, 2)), (po.mixer(2, 16, 24, 24, 40, kv_from=0), None)])
    path, w = _model(tmp_path, cfg, 9, place)
    toks = po.tokens(cfg, 300)
    with Engine(path, place) as e:
        e.feed([("a", toks[:5])], *[[("a", [t], i == 294)] for i, t in enumerate(toks[5:])])
        assert po.row_error(e.logits("a"), po.forward(cfg, w, toks)) < TOL[place[1]]


# ------------------------------------------------------------------------------------------------ generation
def _check_greedy(cfg, w, prompts, got, slack):
    check_greedy(lambda toks: po.forward(cfg, w, toks), prompts, got, slack)


def test_greedy_generation(tmp_path, place):
    """Through LLM.generate: chunked prompts (64 tokens a step), decode steps beside them, several requests."""
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 10, place)
    prompts = [po.tokens(cfg, n, n) for n in (1, 3, 40, 100, 130, 17)]
    llm = make_llm(path, place)
    got = generate(llm, prompts, 12)
    assert all(len(g) == 12 for g in got)
    _check_greedy(cfg, w, prompts, got, 1e-3 if place[1] == "float32" else 0.25)
    if place[1] == "float32":
        assert got[2] == po.greedy(cfg, w, prompts[2], 12)
    if place == ("cuda", "bfloat16"):
        runner = llm.llm_engine.engine_core.engine_core.model_executor.worker.runner
        assert runner.graphs and any(getattr(g, "replays", 0) for g in runner.graphs.values())    # decode steps replay graphs
    assert generate(llm, prompts[3:5], 4) == [g[:4] for g in got[3:5]]                           # and the prefix cache serves them
    llm.shutdown()


def test_generation_with_preemption(tmp_path):
    """A pool that cannot hold all requests: some are put back and computed again."""
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 11)
    prompts = [po.tokens(cfg, n, n) for n in (60, 62, 50, 61)]
    llm = make_llm(path, ("cpu", "float32"), num_gpu_blocks_override=7, enable_prefix_caching=False)
    sched = llm.llm_engine.engine_core.engine_core.scheduler
    seen = []
    orig = sched._preempt
    sched._preempt = lambda r: (seen.append(r.request_id), orig(r))[1]
    got = generate(llm, prompts, 20)
    assert seen
    _check_greedy(cfg, w, prompts, got, 1e-3)
    llm.shutdown()


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(tensor_parallel_size=2, enable_expert_parallel=True),
                                dict(pipeline_parallel_size=2)], ids=["tp2", "tp2-ep", "pp2"])
def test_parallel_ranks_generate_the_same(tmp_path, kw):
    cfg = po.config(64, 96, [(po.mixer(2, 24, 16, 32, 40), po.moe(24, 6, 2, 3, 2)), (po.mixer(4, 16, 24, 24, 40, kv_from=0), None),
                             (po.mixer(2, 16, 8, 16, 24), po.moe(16, 4, 2, 1, 1)), (po.mixer(2, 32, 16, 8, 24, kv_from=2), po.moe(8, 4, 3, 2, 2))])
    path, w = _model(tmp_path, cfg, 12)
    prompts = [po.tokens(cfg, n, n) for n in (5, 70, 33)]
    llm = make_llm(path, ("cpu", "float32"), distributed_executor_backend="mp", **kw)
    got = generate(llm, prompts, 6)
    llm.shutdown()
    _check_greedy(cfg, w, prompts, got, 1e-3)


def test_a_shared_latent_stays_on_its_pipeline_stage(tmp_path):
    """Stage 1 would hold a layer whose latent lives on stage 0."""
    from vllm_b200.layers.attention import MLAAttentionCore, clear_attention_layers
    clear_attention_layers()
    with pytest.raises(ValueError, match="shares the cache"):
        MLAAttentionCore(2, 16, 0, 1.0, "model.layers.1.mixer.attn", kv_sharing_target="model.layers.0.mixer.attn")
    MLAAttentionCore(2, 16, 0, 1.0, "model.layers.0.mixer.attn")
    with pytest.raises(ValueError, match="shares the cache"):
        MLAAttentionCore(2, 24, 0, 1.0, "model.layers.1.mixer.attn", kv_sharing_target="model.layers.0.mixer.attn")
    clear_attention_layers()


# ------------------------------------------------------------------------------------------------ the replay program
def test_trace_program(tmp_path, place):
    cfg = po.small()
    path, w = _model(tmp_path, cfg, 13, place)
    a, b = po.tokens(cfg, 70, 1), po.tokens(cfg, 20, 2)
    lines = [dict(step=0, entries=[dict(id="a", tokens=a[:50], want=[])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b, want=[19, 0, 7]), dict(id="a", tokens=a[50:], want=[19])], end=["a", "b"]),
             dict(step=2, entries=[dict(id="a", tokens=b[:3], want=[2])], end=["a"])]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", place[1], "--out", str(out), "--max-tokens",
                        "192", "--device", place[0]], input="".join(json.dumps(s) + "\n" for s in lines), text=True,
                       capture_output=True, cwd=tmp_path, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == ["done 0", "done 1", "done 2"]
    assert sorted(os.listdir(out)) == ["1.f32", "2.f32"]
    got = [torch.from_numpy(np.fromfile(out / f, dtype="<f4").reshape(-1, cfg["vocab"])) for f in ("1.f32", "2.f32")]
    la, lb = po.forward(cfg, w, a), po.forward(cfg, w, b)
    assert po.row_error(got[0], torch.stack([lb[19], lb[0], lb[7], la[69]])) < TOL[place[1]]
    assert po.row_error(got[1], lb[2:3]) < TOL[place[1]]


def test_replay_rejects_malformed_steps(tmp_path):
    path, _ = _model(tmp_path, po.small())
    with Engine(path, ("cpu", "float32"), 256) as e:
        for entries in ([dict(id="a", tokens=[], want=[])], [dict(id="a", tokens=[1]), dict(id="a", tokens=[2])],
                        [dict(id="a", tokens=[1] * 257)], [dict(id=str(i), tokens=[1]) for i in range(5)]):
            with pytest.raises(ValueError):
                e.replay.step(entries)


def test_every_kernel_symbol_has_a_source():
    """A checkout without the full library compiles a symbol's source at its first call."""
    from vllm_b200.csrc.build import source_of
    from vllm_b200.models.pomipel import PomipelForCausalLM
    ops_file = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "vllm_b200", "ops", "cuda.py")
    import re
    names = set(re.findall(r'"(vb_\w+)"', open(ops_file).read()))
    assert len(names) > 50
    sources = {source_of(n) for n in names}
    assert set(PomipelForCausalLM.kernel_sources) <= sources
    with pytest.raises(RuntimeError):
        source_of("vb_no_such_kernel")
