"""Legelix: the configuration and checkpoint, each mechanism, and whole models through the engine's scheduler, cache and state
slots and model runner, against the plain implementation (tests/legelix_oracle.py).

Whole-model tests run on the CPU, and on the device in 16 and in 32 bits."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from tests import legelix_oracle as lo
from tests.replay_utils import (PLACES, TOL, Engine, check_greedy, generate, make_llm, portions, row_error, save_model, tokens)

CPU32 = ("cpu", "float32")


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


def _model(tmp_path, cfg, seed=0, change=None, **kw):
    w = lo.make_weights(cfg, seed, **kw)
    if change:
        change(w)
    return save_model(cfg, w, tmp_path / "model"), w


# ------------------------------------------------------------------------------------------------ configuration and checkpoint
def test_configuration_is_read_from_the_model_folder(tmp_path):
    from vllm_b200.config import ModelConfig
    from vllm_b200.models.registry import resolve_model_cls
    path, _ = _model(tmp_path, lo.small(), rank=11)
    mc = ModelConfig(model=path)
    assert mc.architecture == "LegelixForCausalLM" and not mc.is_mla and not mc.is_moe
    assert (mc.vocab_size, mc.hidden_size, mc.num_layers) == (208, 96, 4)
    assert [l["mixer"].get("rank") for l in mc.hf_config["layers"]] == [None, 11, None, 11]      # from the tensors' shapes
    assert resolve_model_cls(mc.architecture).__name__ == "LegelixForCausalLM"
    assert mc.torch_dtype == torch.bfloat16


@pytest.mark.parametrize("change", [lambda m: m["left"].update(kv_heads=4), lambda m: m["right"].update(groups=3),
                                    lambda m: m["right"].update(norm_groups=7), lambda m: m["left"]["rot"].update(dims=7),
                                    lambda m: m["left"]["rot"].update(dims=26), lambda m: m["left"]["mask"].update(size=0)])
def test_sizes_that_do_not_fit_are_an_error(change):
    from vllm_b200.config import ModelConfig
    cfg = lo.small()
    change(cfg["layers"][0]["mixer"])
    with pytest.raises(ValueError, match="layer 0"):
        ModelConfig(model="x", hf_config=cfg)


@pytest.mark.parametrize("name", sorted(lo.MODELS))
def test_checkpoint_names_are_all_taken_and_none_else(tmp_path, name):
    path, w = _model(tmp_path, lo.MODELS[name]())
    with Engine(path, CPU32, 256) as e:
        model = e.replay.core.model_executor.worker.get_model()
        loaded = model.load_weights((k, v.clone()) for k, v in w.items())
        assert loaded == {n for n, _ in model.named_parameters()}
        for bad in ("l0.mix.foo", "l1.mix.left.sinks", "l9.norm1", "l0x.norm1", "other"):
            with pytest.raises(ValueError):
                model.load_weights([(bad, torch.zeros(48, 96))])


def test_unknown_layer_kinds_are_an_error(tmp_path):
    for i, change in enumerate((lambda c: c["layers"][1].update(type="other"), lambda c: c["layers"][1]["mlp"].update(kind="moe"))):
        cfg = lo.small()
        path, _ = _model(tmp_path / str(i), cfg)
        change(cfg)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(cfg, f)
        with pytest.raises(ValueError, match="unknown"):
            Engine(path, CPU32, 256)


# ------------------------------------------------------------------------------------------------ caches and state slots
def test_one_block_table_and_one_state_slot_for_layers_of_every_size(tmp_path):
    path, _ = _model(tmp_path, lo.small())
    with Engine(path, CPU32, 256) as e:
        runner = e.replay.core.model_executor.worker.runner
        shapes = {n: tuple(c.shape) for n, c in runner.kv_caches.items()}
        assert shapes["model.layers.0.mixer.attn"] == (5, 2, 2, 64, 24) and shapes["model.layers.2.mixer.attn"] == (5, 2, 4, 64, 40)
        states = [n for n in shapes if not n.endswith("attn")]
        assert sorted(states) == [f"model.layers.{i}.mixer{s}" for i, s in ((0, ".mamba"), (1, ""), (2, ".mamba"), (3, ""))]
        assert all(shapes[n][0] == 5 for n in states)            # four live requests and the padding row
        mgr = e.replay.core.scheduler.kv_cache_manager
        assert mgr.num_groups == 2 and mgr.pool.get_num_free_blocks() == 4 and mgr.state_pool.get_num_free_blocks() == 4
        e.feed([("a", [1] * 100), ("b", [2])])
        assert mgr.pool.get_num_free_blocks() == 1 and mgr.state_pool.get_num_free_blocks() == 2
        e.feed([("b", [3], True)])
        assert mgr.pool.get_num_free_blocks() == 2 and mgr.state_pool.get_num_free_blocks() == 3


def test_state_slots_are_counted_by_requests_and_bounded_by_memory():
    from vllm_b200.core.kv_cache_manager import FullAttentionSpec, MambaSpec, get_kv_cache_config
    specs = {"a": FullAttentionSpec(64, 2, 32), "b": FullAttentionSpec(64, 4, 16), "s": MambaSpec(64, 1 << 20), "t": MambaSpec(64, 1 << 18)}
    cfg, _ = get_kv_cache_config(specs, 1 << 30, 1024, max_num_seqs=16)
    assert cfg.num_state_slots == 17 and len(cfg.kv_cache_groups) == 2
    page = 2 * 64 * 2 * 32 * 2 + 2 * 64 * 4 * 16 * 2
    assert cfg.num_blocks == ((1 << 30) - 17 * (5 << 18)) // page
    cfg, _ = get_kv_cache_config(specs, 1 << 30, 1024, max_num_seqs=4000)          # fewer, so that pages have room
    assert cfg.num_state_slots == int((1 << 30) * 0.4) // (5 << 18) and cfg.num_blocks > 1000
    only, _ = get_kv_cache_config({"s": MambaSpec(64, 1 << 20)}, 1 << 30, 1024, max_num_seqs=8)
    assert only.num_state_slots == 9
    with pytest.raises(ValueError):
        get_kv_cache_config({"s": MambaSpec(64, 1 << 30)}, 1 << 28, 1024)


def test_requests_wait_for_a_state_slot():
    from vllm_b200.core.kv_cache_manager import FullAttentionSpec, KVCacheManager, MambaSpec, get_kv_cache_config
    from vllm_b200.core.request import Request
    from vllm_b200.sampling_params import SamplingParams
    cfg, _ = get_kv_cache_config({"a": FullAttentionSpec(16, 1, 16), "s": MambaSpec(16, 4096)}, 1 << 22, 64, max_num_seqs=2)
    mgr = KVCacheManager(cfg, 64, enable_caching=False)
    reqs = [Request(str(i), [1] * 20, SamplingParams(max_tokens=4)) for i in range(3)]
    got = [mgr.allocate_slots(r, 20) for r in reqs]
    assert got[0] is not None and got[1] is not None and got[2] is None
    slots = {tuple(mgr.get_block_ids(r.request_id)[1]) for r in reqs[:2]}
    assert slots == {(1,), (2,)}
    mgr.free(reqs[0])
    assert mgr.allocate_slots(reqs[2], 20) is not None and mgr.get_num_common_prefix_blocks("2", 1)[1] == 0


# ------------------------------------------------------------------------------------------------ mechanisms (plain ops)
def test_stream_step():
    from vllm_b200.ops import ref
    g = torch.Generator().manual_seed(1)
    x, y, yb, w, b, w2, b2 = [torch.randn(*s, generator=g) for s in ((9, 40), (9, 40), (40,), (40,), (40,), (40,), (40,))]
    want = x.double() + 0.3 * lo.layer_norm((y + yb).double(), w.double(), b.double(), 1e-2)
    h = ref.norm_add(x, y, yb, (w, b), 0.3, (w2, b2), 1e-2)
    torch.testing.assert_close(x.double(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(h.double(), lo.layer_norm(want, w2.double(), b2.double(), 1e-2), rtol=1e-5, atol=1e-5)
    x = torch.full((1, 64), 256.0)
    one = torch.zeros(64, dtype=torch.bfloat16), torch.ones(64, dtype=torch.bfloat16)
    for _ in range(8):                                        # steps of 1/8 are below bfloat16's step at 256
        ref.norm_add(x, torch.ones(1, 64, dtype=torch.bfloat16), None, one, 0.125, None, 1e-6)
    torch.testing.assert_close(x, torch.full((1, 64), 257.0), rtol=0, atol=1e-3)


@pytest.mark.parametrize("spec", [dict(base=500.0, dims=16, scaling=dict(factor=8.0, low=1.0, high=4.0, original=128)),
                                  dict(base=9000.0, dims=10, scaling=dict(factor=3.0, low=2.0, high=3.0, original=700)), dict(base=50.0, dims=2)])
def test_rotation_of_neighbours_with_scaled_frequencies(spec):
    from vllm_b200.layers.rotary import get_rope
    sc = spec.get("scaling")
    rope = get_rope(24, spec["dims"], 300, spec["base"], False, sc and dict(
        rope_type="llama3", factor=sc["factor"], low_freq_factor=sc["low"], high_freq_factor=sc["high"], original_max_position_embeddings=sc["original"]))
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(300, 3 * 24, generator=g), torch.randn(300, 24, generator=g)
    f = lo.frequencies(spec)
    assert len(set(f)) == len(f)
    wq, wk = lo.rotate(q.double().view(300, 3, 24), f), lo.rotate(k.double().view(300, 1, 24), f)
    gq, gk = rope(torch.arange(300), q.clone(), k.clone())
    torch.testing.assert_close(gq.double().view(300, 3, 24), wq, rtol=1e-4, atol=1e-4)
    torch.testing.assert_close(gk.double().view(300, 1, 24), wk, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("groups,first,wl", [(1, True, 24), (3, True, 24), (4, False, 6), (24, False, 1)])
def test_gated_norm(groups, first, wl):
    from vllm_b200 import ops
    g = torch.Generator().manual_seed(3)
    y, z, w = torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g), torch.randn(wl, generator=g)
    gate, wd = lo.silu(z.double()), w.double().repeat(24 // wl)
    want = lo.unit_rms((y.double() * (gate if first else 1)).view(5, groups, -1), 1e-2).view(5, 24) * wd * (1 if first else gate)
    torch.testing.assert_close(ops.gated_norm(y, z, w, groups, 1e-2, first).double(), want, rtol=1e-5, atol=1e-5)


def test_gated_scan_continues_a_state():
    from vllm_b200.ops import ref
    g = torch.Generator().manual_seed(4)
    q, k, a = torch.randn(9, 2, 5, generator=g), torch.randn(9, 2, 5, generator=g), torch.rand(9, 2, 5, generator=g)
    v, s0 = torch.randn(9, 2, 7, generator=g), torch.randn(2, 5, 7, generator=g)
    want, sw = lo.gated_scan(*[t.double() for t in (q, k, v, a)], s0.double())
    got, sg = ref.gated_linear_scan(q, k, v, a, s0)
    torch.testing.assert_close(got.double(), want, rtol=1e-4, atol=1e-4)
    torch.testing.assert_close(sg.double(), sw, rtol=1e-4, atol=1e-4)


def test_chunks_and_sinks_in_the_plain_attention():
    from vllm_b200.ops import ref
    g = torch.Generator().manual_seed(5)
    n, H, G, D = 70, 4, 2, 8
    q, k, v, sink = [torch.randn(*s, generator=g) for s in ((n, H, D), (n, G, D), (n, G, D), (H,))]
    cache = torch.zeros(3, 2, G, 32, D)
    for b in range(3):
        part = slice(32 * b, min(32 * b + 32, n))
        m = part.stop - part.start
        cache[b, 0, :, :m], cache[b, 1, :, :m] = k[part].transpose(0, 1), v[part].transpose(0, 1)
    args = (torch.tensor([[0, 1, 2]]), torch.tensor([n]), torch.tensor([0, 30]))
    for size in (1, 25, 64, 100):
        got = ref.paged_attention(q[-30:], cache, *args, 0.5, chunk_size=size, sinks=sink)
        want = lo.attend(q.double(), k.double(), v.double(), 0.5, size, sink.double())[-30:]
        torch.testing.assert_close(got.reshape(30, -1).double(), want, rtol=1e-4, atol=1e-4)


def test_projections_that_share_an_input_or_a_sum():
    from vllm_b200.layers.linear import MergedReplicatedLinear, SummedReplicatedLinear
    g = torch.Generator().manual_seed(6)
    x, parts = torch.randn(3, 10, generator=g), [torch.randn(n, 10, generator=g) for n in (5, 1, 8)]
    m = MergedReplicatedLinear(10, [5, 1, 8], True, torch.float32, align=8)
    bias = torch.randn(1, generator=g)
    for i, w in enumerate(parts):
        m.weight_loader(m.weight, w, i)
    m.weight_loader(m.bias, bias, 1)
    y = m(x)
    assert y.shape == (3, 24)
    for i, (got, w) in enumerate(zip(m.parts(y), parts)):
        torch.testing.assert_close(got, x @ w.T + (bias if i == 1 else 0))
    s = SummedReplicatedLinear([5, 3], 6, torch.float32, align=4)
    a, b = torch.randn(6, 5, generator=g), torch.randn(6, 3, generator=g)
    s.weight_loader(s.weight, a, 0)
    s.weight_loader(s.weight, b, 1)
    buf, (pa, pb) = s.buffer(x)
    pa.copy_(x[:, :5])
    pb.copy_(x[:, 5:8])
    torch.testing.assert_close(s(buf), x[:, :5] @ a.T + x[:, 5:8] @ b.T)


def test_stream_after_every_layer(tmp_path):
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 2)
    toks = tokens(cfg, 60)
    want = []
    lo.forward(cfg, w, toks, layers=want)
    with Engine(path, CPU32, 256) as e:
        got = []
        for layer in e.replay.core.model_executor.worker.get_model().model.layers:
            layer.register_forward_hook(lambda mod, args, out: got.append(args[1].clone()))
        e.feed([("a", toks, True)])
        assert len(got) == 4
        for g_, w_ in zip(got, want):
            torch.testing.assert_close(g_.double(), w_, rtol=1e-4, atol=1e-4)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(lo.MODELS))
def test_prompt_token_by_token_and_portions_agree_with_the_equations(tmp_path, place, name):
    cfg = lo.MODELS[name]()
    path, w = _model(tmp_path, cfg, 3)
    toks = tokens(cfg, 150)                                    # three pages, several chunks
    want = lo.forward(cfg, w, toks)
    tol = TOL[place[1]]
    with Engine(path, place) as e:
        e.feed([("whole", toks, True)])
        assert row_error(e.logits("whole"), want) < tol
        e.feed(*[[("single", [t], i == 149)] for i, t in enumerate(toks)])
        assert row_error(e.logits("single"), want) < tol
        for k, sizes in enumerate([(2,), (3, 2, 5), (63, 2, 64, 2), (17, 1, 1, 40), (50, 49, 2), (100, 2, 1)]):
            parts = portions(toks, sizes)
            e.feed(*[[(f"p{k}", p, i == len(parts) - 1)] for i, p in enumerate(parts)])
            assert row_error(e.logits(f"p{k}"), want) < tol, sizes


def test_first_tokens(tmp_path, place):
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 4)
    with Engine(path, place) as e:
        for n in (1, 2, 3, 4):
            toks = tokens(cfg, n, n)
            e.feed([("a", toks, True)], *[[("b", [t], i == n - 1)] for i, t in enumerate(toks)])
            want = lo.forward(cfg, w, toks)
            assert row_error(e.logits("a"), want) < TOL[place[1]] and row_error(e.logits("b"), want) < TOL[place[1]]


@pytest.mark.parametrize("name", ["small", "wide"])
def test_unequal_requests_in_one_batch(tmp_path, place, name):
    """Portions beside single tokens; every request as if it were alone."""
    cfg = lo.MODELS[name]()
    path, w = _model(tmp_path, cfg, 5)
    reqs = {"a": tokens(cfg, 140, 1), "b": tokens(cfg, 9, 2), "c": tokens(cfg, 75, 3), "d": tokens(cfg, 33, 4)}
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
            assert row_error(e.logits(r), lo.forward(cfg, w, t)) < TOL[place[1]], r


def test_pages_and_slots_are_used_again(tmp_path, place):
    """Five pages and four slots serve many requests one after another; a new one never sees what a page or slot held."""
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 6, lasting=True)
    with Engine(path, place, 5 * 64) as e:
        mgr = e.replay.core.scheduler.kv_cache_manager
        free, slots = mgr.pool.get_num_free_blocks(), mgr.state_pool.get_num_free_blocks()
        assert (free, slots) == (5, 4)
        keep = tokens(cfg, 100, 50)                            # stays while the others come and go
        e.feed([("keep", keep[:60])])
        for k in range(9):
            n = (64, 65, 130, 2, 128, 127, 1, 3, 100)[k]
            toks = tokens(cfg, n, k)
            cut = max(1, n // 2)
            e.feed([(f"r{k}", toks[:cut], n == 1), ("keep", keep[60 + 4 * k:64 + 4 * k])], *([[(f"r{k}", toks[cut:], True)]] if n > 1 else []))
            assert row_error(e.logits(f"r{k}"), lo.forward(cfg, w, toks)) < TOL[place[1]], k
        e.feed([("keep", keep[96:], True)])
        assert row_error(e.logits("keep"), lo.forward(cfg, w, keep)) < TOL[place[1]]
        assert (mgr.pool.get_num_free_blocks(), mgr.state_pool.get_num_free_blocks()) == (free, slots)


def test_a_pool_that_is_too_small_is_an_error(tmp_path):
    path, _ = _model(tmp_path, lo.small())
    with Engine(path, CPU32, 128) as e:
        e.feed([("a", [1] * 64), ("b", [1] * 64)])
        with pytest.raises(RuntimeError, match="no room"):
            e.feed([("a", [2])])
    with Engine(path, CPU32, 512) as e:
        e.feed([(str(i), [1]) for i in range(4)])
        with pytest.raises(ValueError, match="live requests"):
            e.feed([("5", [1])])


# chunk of 150: (key, query) positions; in the same chunk or not, at page borders, first and last places of a chunk
PAIRS = [(0, 149), (0, 1), (63, 149), (64, 130), (1, 128), (149, 150), (150, 199), (149, 299), (150, 299), (191, 192), (148, 149), (0, 150), (192, 299)]


@pytest.mark.parametrize("key,query", PAIRS)
def test_a_far_key_is_seen_inside_its_chunk_only(tmp_path, place, key, query):
    """One key far above the noise; the query in a prompt, in a short portion and decoded."""
    size = 150
    cfg = lo.config(64, 120, [lo.parallel(lo.left(4, 2, 24, 16, size, rot=16), lo.right(2, 8, 8), None, 2.0, 0.3), lo.gated(2, 8, 16, 2.0, 40)])
    X, Q = 11, 12
    path, w = _model(tmp_path, cfg, 7, change=lambda w: lo.plant_key(cfg, w, X, Q))
    toks = tokens(cfg, query, key, avoid=(X, Q)) + [Q]
    toks[key] = X
    want = lo.forward(cfg, w, toks)[-1:]
    if key // size == query // size:
        other = lo.forward(cfg, w, toks, hide=(key,))[-1:]
    else:
        open_cfg = copy.deepcopy(cfg)
        open_cfg["layers"][0]["mixer"]["left"]["mask"]["size"] = 10 ** 6
        other = lo.forward(open_cfg, w, toks)[-1:]
    tol = TOL[place[1]]
    assert row_error(other, want) > 3 * tol                    # seeing it, or not, changes the logits
    with Engine(path, place) as e:
        e.feed([("whole", toks, True)], [("dec", toks[:-1])], [("dec", toks[-1:], True)])
        names = ["whole", "dec"]
        if query > 1:
            e.feed([("cut", toks[:-2])], [("cut", toks[-2:], True)])
            names.append("cut")
        for r in names:
            assert row_error(e.logits(r)[-1:], want) < tol, r


def test_sinks_count(tmp_path, place):
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 8, sink=2.5)
    toks = tokens(cfg, 90)
    want = lo.forward(cfg, w, toks)
    none = {**w, **{k: torch.full_like(v, -50.0) for k, v in w.items() if k.endswith("sink")}}
    assert row_error(lo.forward(cfg, none, toks), want) > 3 * TOL["bfloat16"]
    with Engine(path, place) as e:
        e.feed([("a", toks[:40])], *[[("a", [t], i == 49)] for i, t in enumerate(toks[40:])])
        assert row_error(e.logits("a"), want) < TOL[place[1]]


def test_states_remember_the_first_tokens(tmp_path, place):
    """No key of the first chunk is visible at the end; what is left of the first tokens is in the states."""
    cfg = lo.config(64, 96, [lo.gated(2, 16, 24, 16.0, 40), lo.parallel(lo.left(2, 1, 16, 16, 20), lo.right(2, 16, 12, conv=3), 32)])
    path, w = _model(tmp_path, cfg, 9, lasting=True)
    a = tokens(cfg, 130, 1)
    b = [5] * 40 + a[40:]
    wa, wb = lo.forward(cfg, w, a), lo.forward(cfg, w, b)
    assert row_error(wa[-1:], wb[-1:]) > 3 * TOL["bfloat16"]
    with Engine(path, place) as e:
        e.feed([("a", a[:30]), ("b", b[:64])], [("b", b[64:125])], [("a", a[30:126]), ("b", b[125:127])], [("a", a[126:128])],
               [("a", a[128:129]), ("b", b[127:])], [("a", a[129:])])
        assert row_error(e.logits("a"), wa) < TOL[place[1]] and row_error(e.logits("b"), wb) < TOL[place[1]]


def test_no_query_sees_what_comes_after_it(tmp_path, place):
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 10)
    a, b = tokens(cfg, 140, 1), tokens(cfg, 140, 2)
    b[:70] = a[:70]
    with Engine(path, place) as e:
        e.feed([("a", a, True)], [("b", b, True)])
        la, lb = e.logits("a"), e.logits("b")
        assert row_error(la[:70], lb[:70]) < 1e-5 and row_error(la[70:], lb[70:]) > 0.3


def test_long_decoding(tmp_path, place):
    cfg = lo.config(64, 96, [lo.parallel(lo.left(2, 1, 16, 24, 70, rot=8), lo.right(2, 16, 12), 40), lo.gated(2, 12, 16, 16.0, None)])
    path, w = _model(tmp_path, cfg, 11, lasting=True)
    toks = tokens(cfg, 300)
    with Engine(path, place) as e:
        e.feed([("a", toks[:5])], *[[("a", [t], i == 294)] for i, t in enumerate(toks[5:])])
        assert row_error(e.logits("a"), lo.forward(cfg, w, toks)) < TOL[place[1]]


# ------------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", ["small", "wide", "only_gated"])
def test_greedy_generation(tmp_path, place, name):
    """Through LLM.generate: chunked prompts (64 tokens a step), decode steps beside them, several requests."""
    cfg = lo.MODELS[name]()
    path, w = _model(tmp_path, cfg, 12)
    prompts = [tokens(cfg, n, n) for n in (1, 3, 40, 100, 130, 17)]
    llm = make_llm(path, place, kv_cache_memory_bytes=64 << 20)
    got = generate(llm, prompts, 12)
    assert all(len(g) == 12 for g in got)
    check_greedy(lambda t: lo.forward(cfg, w, t), prompts, got, 1e-3 if place[1] == "float32" else 0.25)
    if place[1] == "float32":
        assert got[2] == lo.greedy(cfg, w, prompts[2], 12)
    if place[0] == "cuda":
        runner = llm.llm_engine.engine_core.engine_core.model_executor.worker.runner
        assert runner.graphs and any(getattr(g, "replays", 0) for g in runner.graphs.values())    # decode steps replay graphs
    assert generate(llm, prompts[3:5], 4) == [g[:4] for g in got[3:5]]
    llm.shutdown()


def test_more_requests_than_state_slots(tmp_path, place):
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 13)
    prompts = [tokens(cfg, 5 + 7 * i, i) for i in range(9)]
    llm = make_llm(path, place, max_num_seqs=2)
    got = generate(llm, prompts, 6)
    check_greedy(lambda t: lo.forward(cfg, w, t), prompts, got, 1e-3 if place[1] == "float32" else 0.25)
    llm.shutdown()


def test_generation_with_preemption(tmp_path):
    """A pool that cannot hold all requests: some are put back and computed again, from an empty state."""
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 14, lasting=True)
    prompts = [tokens(cfg, n, n) for n in (60, 62, 50, 61)]
    llm = make_llm(path, CPU32, num_gpu_blocks_override=7, enable_prefix_caching=False)
    sched = llm.llm_engine.engine_core.engine_core.scheduler
    seen = []
    orig = sched._preempt
    sched._preempt = lambda r: (seen.append(r.request_id), orig(r))[1]
    got = generate(llm, prompts, 20)
    assert seen
    check_greedy(lambda t: lo.forward(cfg, w, t), prompts, got, 1e-3)
    llm.shutdown()


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(pipeline_parallel_size=2)], ids=["tp2", "pp2"])
def test_parallel_ranks_generate_the_same(tmp_path, kw):
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 15)
    prompts = [tokens(cfg, n, n) for n in (5, 70, 33)]
    llm = make_llm(path, CPU32, distributed_executor_backend="mp", **kw)
    got = generate(llm, prompts, 6)
    llm.shutdown()
    check_greedy(lambda t: lo.forward(cfg, w, t), prompts, got, 1e-3)


# ------------------------------------------------------------------------------------------------ the replay program
def test_trace_program(tmp_path, place):
    cfg = lo.small()
    path, w = _model(tmp_path, cfg, 16)
    a, b = tokens(cfg, 70, 1), tokens(cfg, 20, 2)
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
    got = [torch.from_numpy(np.fromfile(out / f, dtype="<f4").reshape(-1, cfg["vocab"])) for f in ("1.f32", "2.f32")]
    la, lb = lo.forward(cfg, w, a), lo.forward(cfg, w, b)
    assert row_error(got[0], torch.stack([lb[19], lb[0], lb[7], la[69]])) < TOL[place[1]]
    assert row_error(got[1], lb[2:3]) < TOL[place[1]]


def test_kernel_sources_exist():
    from vllm_b200.csrc import build
    from vllm_b200.models.legelix import LegelixForCausalLM
    have = {f[:-3] for f in os.listdir(build.HERE) if f.endswith(".cu")}
    for name, want in (("small", "attention_any"), ("wide", "attention_tc")):
        src = set(LegelixForCausalLM.kernel_sources(lo.MODELS[name](), torch.bfloat16))
        assert src <= have and want in src
    assert "attention_any" in LegelixForCausalLM.kernel_sources(lo.wide(), torch.float32)
