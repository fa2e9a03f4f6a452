"""Kopadra: the configuration and checkpoint, each mechanism, and whole models through the engine's scheduler, cache and state
slots and model runner, against the plain implementation (tests/kopadra_oracle.py).

Whole-model tests run on the CPU, and on the device in 16 and in 32 bits."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from tests import kopadra_oracle as ko
from tests.replay_utils import (PLACES, Engine, check_greedy, generate, make_llm, portions, row_error, save_model, tokens)

CPU32 = ("cpu", "float32")
TOL = {"float32": 2e-4, "bfloat16": 0.06}                      # largest row error over the spread of the logits


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


def _model(tmp_path, cfg, seed=0, change=None, place=CPU32, **kw):
    w = ko.make_weights(cfg, seed, steady=place[1] == "bfloat16", **kw)
    if change:
        change(w)
    return save_model(cfg, w, tmp_path / "model"), w


# ------------------------------------------------------------------------------------------------ configuration and checkpoint
def test_configuration_is_read_from_the_model_folder(tmp_path):
    from vllm_b200.config import ModelConfig
    from vllm_b200.models.registry import resolve_model_cls
    path, _ = _model(tmp_path, ko.small())
    mc = ModelConfig(model=path)
    assert mc.architecture == "KopadraForCausalLM" and not mc.is_mla and mc.is_moe
    assert (mc.vocab_size, mc.hidden_size, mc.num_layers) == (208, 96, 6)
    assert resolve_model_cls(mc.architecture).__name__ == "KopadraForCausalLM"
    assert mc.torch_dtype == torch.bfloat16
    assert not ModelConfig(model="x", hf_config=ko.only_memory()).hf_config.get("sliding_window")


@pytest.mark.parametrize("layer,change", [
    (0, lambda m: m.update(kv_heads=4)), (0, lambda m: m["rot"].update(dims=7)), (0, lambda m: m["rot"].update(dims=26)),
    (3, lambda m: m.update(kv_from=3)), (3, lambda m: m.update(kv_from=1)), (3, lambda m: m.update(kv_from=2)),
    (5, lambda m: m.update(kv_from=3)), (5, lambda m: m.update(vdim=24))])
def test_sizes_that_do_not_fit_are_an_error(layer, change):
    from vllm_b200.config import ModelConfig
    cfg = ko.small()
    change(cfg["layers"][layer]["mixer"])
    with pytest.raises(ValueError, match=f"layer {layer}"):
        ModelConfig(model="x", hf_config=cfg)


@pytest.mark.parametrize("name", sorted(ko.MODELS))
def test_checkpoint_names_are_all_taken_and_none_else(tmp_path, name):
    path, w = _model(tmp_path, ko.MODELS[name]())
    with Engine(path, CPU32, 256) as e:
        model = e.replay.core.model_executor.worker.get_model()
        loaded = model.load_weights((k, v.clone()) for k, v in w.items())
        assert loaded == {n for n, _ in model.named_parameters()}
        assert model.lm_head.weight is model.model.embed_tokens.weight
        for bad in ("l0.mix.foo", "l1.mix.left.q", "l9.norm1", "l0x.norm1", "l0.mlp.e9.gate", "l0.mlp.e0.gate.b", "head", "final.norm.b"):
            with pytest.raises(ValueError):
                model.load_weights([(bad, torch.zeros(48, 96))])


def test_a_layer_with_anothers_keys_has_no_tensors_of_them(tmp_path):
    path, _ = _model(tmp_path, ko.small())
    with Engine(path, CPU32, 256) as e:
        model = e.replay.core.model_executor.worker.get_model()
        for bad in ("l3.mix.k", "l3.mix.v.b", "l3.mix.k.norm", "l3.mix.g.b"):
            with pytest.raises(ValueError):
                model.load_weights([(bad, torch.zeros(48, 96))])


def test_unknown_layer_kinds_are_an_error(tmp_path):
    for i, change in enumerate((lambda c: c["layers"][1].update(type="other"), lambda c: c["layers"][1]["mlp"].update(kind="other"))):
        cfg = ko.small()
        path, _ = _model(tmp_path / str(i), cfg)
        change(cfg)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(cfg, f)
        with pytest.raises(ValueError, match="unknown"):
            Engine(path, CPU32, 256)


# ------------------------------------------------------------------------------------------------ caches and state slots
def test_shared_keys_own_no_cache_and_one_block_table_serves_layers_of_every_size(tmp_path):
    path, _ = _model(tmp_path, ko.small())
    with Engine(path, CPU32, 256) as e:
        runner = e.replay.core.model_executor.worker.runner
        shapes = {n: tuple(c.shape) for n, c in runner.kv_caches.items()}
        assert shapes.pop("model.layers.0.mixer.attn") == (5, 2, 2, 64, 40) and shapes.pop("model.layers.2.mixer.attn") == (5, 2, 4, 64, 32)
        assert sorted(shapes) == ["model.layers.1.mixer", "model.layers.4.mixer"] and all(s[0] == 5 for s in shapes.values())
        mgr = e.replay.core.scheduler.kv_cache_manager
        assert mgr.num_groups == 2 and mgr.pool.get_num_free_blocks() == 4 and mgr.state_pool.get_num_free_blocks() == 4
        e.feed([("a", [1] * 100), ("b", [2])])
        assert mgr.pool.get_num_free_blocks() == 1 and mgr.state_pool.get_num_free_blocks() == 2
        e.feed([("b", [3], True)])
        assert mgr.pool.get_num_free_blocks() == 2 and mgr.state_pool.get_num_free_blocks() == 3


def test_a_shared_cache_must_be_on_the_rank():
    from vllm_b200.layers.attention import Attention, clear_attention_layers
    clear_attention_layers()
    Attention(4, 16, 0.25, 2, prefix="own")
    Attention(4, 16, 0.5, 2, prefix="reader", kv_sharing_target="own")
    with pytest.raises(ValueError, match="not an earlier attention layer"):
        Attention(4, 16, 0.5, 2, prefix="r2", kv_sharing_target="elsewhere")
    with pytest.raises(ValueError, match="same head shapes"):
        Attention(4, 16, 0.5, 2, prefix="r3", kv_sharing_target="own", v_head_size=24)
    clear_attention_layers()


# ------------------------------------------------------------------------------------------------ mechanisms (plain ops)
def test_stream_step():
    from vllm_b200 import ops
    g = torch.Generator().manual_seed(1)
    x, y, w = [torch.randn(*s, generator=g) for s in ((9, 40), (9, 40), (40,))]
    want = x.double() + y.double()
    h = ops.add_norm(x, y, (w, None), 1e-2)
    torch.testing.assert_close(x.double(), want, rtol=1e-6, atol=1e-6)
    torch.testing.assert_close(h.double(), ko.layer_norm(want, w.double(), 1e-2), rtol=1e-5, atol=1e-5)
    x = torch.full((1, 64), 256.0)
    for _ in range(8):                                        # steps of 1/8 are below bfloat16's step at 256
        ops.add_norm(x, torch.full((1, 64), 0.125, dtype=torch.bfloat16), None, 0.0)
    torch.testing.assert_close(x, torch.full((1, 64), 257.0), rtol=0, atol=0)


YARN = [dict(base=500.0, dims=16, scaling=dict(factor=8.0, original=128, fast=8.0, slow=1.0)),
        dict(base=9000.0, dims=10, scaling=dict(factor=3.0, original=700, fast=32.0, slow=0.5)),
        dict(base=50.0, dims=24, scaling=dict(factor=0.5, original=64, fast=2.0, slow=2.0)),         # a ramp of no width
        dict(base=3.0, dims=20, scaling=dict(factor=2.0, original=10 ** 6, fast=4.0, slow=1.0)),     # ramp ends behind the last pair
        dict(base=100.0, dims=12, scaling=dict(factor=16.0, original=5, fast=9.0, slow=3.0)), dict(base=50.0, dims=2)]


@pytest.mark.parametrize("spec", YARN)
def test_rotation_of_halves_with_scaled_frequencies(spec):
    from vllm_b200.models.kopadra import GatedAttention
    from vllm_b200.layers.attention import clear_attention_layers
    clear_attention_layers()
    m = dict(heads=3, kv_heads=1, dim=24, vdim=24, scale=1.0, rot=spec)
    rope = GatedAttention(16, m, 1e-5, 300, torch.float32, "x", None).attn.rope
    assert rope.cos_sin_cache.shape == (300, spec["dims"])
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(300, 3 * 24, generator=g), torch.randn(300, 24, generator=g)
    wq, wk = ko.rotate(q.double().view(300, 3, 24), spec), ko.rotate(k.double().view(300, 1, 24), spec)
    gq, gk = rope(torch.arange(300), q.clone(), k.clone())
    torch.testing.assert_close(gq.double().view(300, 3, 24), wq, rtol=2e-6, atol=2e-6)
    torch.testing.assert_close(gk.double().view(300, 1, 24), wk, rtol=2e-6, atol=2e-6)
    clear_attention_layers()


def test_frequencies_are_interpolated_on_a_ramp():
    """Fast pairs keep their frequency, slow ones are divided, those between are mixed, and all are a little longer."""
    plain, _ = ko.frequencies(dict(base=500.0, dims=64))
    got, size = ko.frequencies(dict(base=500.0, dims=64, scaling=dict(factor=5.0, original=1500, fast=24.0, slow=0.8)))
    ratio = [a / b for a, b in zip(got, plain)]
    assert ratio[0] == 1.0 and abs(ratio[-1] - 0.2) < 1e-12 and any(0.3 < r < 0.9 for r in ratio) and size > 1.15


@pytest.mark.parametrize("lasting", [False, True])
def test_matrix_memory_continues_a_state(lasting):
    from vllm_b200.ops import ref
    g = torch.Generator().manual_seed(4)
    q, k, v = [torch.randn(9, 2, n, generator=g) for n in (5, 5, 7)]
    i, f = torch.randn(9, 2, generator=g) * 5, -torch.rand(9, 2, generator=g) * (0.1 if lasting else 4)
    state = torch.randn(2, 5, 7, generator=g), torch.randn(2, 5, generator=g), torch.randn(2, generator=g)
    want, sw = ko.matrix_memory(*[t.double() for t in (q, k, v, i, f)], [t.double() for t in state])
    got, *sg = ref.matrix_memory_scan(q, k, v, i, f, *state)
    torch.testing.assert_close(got.double(), want, rtol=1e-4, atol=1e-4)
    for a, b in zip(sg, sw):
        torch.testing.assert_close(a.double(), b, rtol=1e-4, atol=1e-4)


def test_the_running_maximum_starts_at_zero():
    """A first token with a small input gate: the divisor is exp(-0), not exp(-i)."""
    one = torch.ones(1, 1, 1, dtype=torch.float64)
    i, f = torch.full((1, 1), -3.0, dtype=torch.float64), torch.full((1, 1), -0.1, dtype=torch.float64)
    o, (_, _, m) = ko.matrix_memory(one, one, one, i, f)
    assert abs(float(m) + 0.1) < 1e-12 and abs(float(o) - np.exp(-3.0)) < 1e-6


def test_gated_norm_with_a_sigmoid():
    from vllm_b200 import ops
    g = torch.Generator().manual_seed(3)
    y, z, w = torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g), torch.randn(24, generator=g)
    want = ko.unit_rms(y.double().view(5, 3, 8), 1e-2).view(5, 24) * w.double() * ko.sigmoid(z.double())
    torch.testing.assert_close(ops.gated_norm(y, z, w, 3, 1e-2, False, gate="sigmoid").double(), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("E,top,count,keep", [(14, 5, 2, 1), (12, 3, 4, 2), (9, 5, 3, 2), (6, 1, 6, 1), (8, 8, 1, 1), (1, 1, 1, 1)])
def test_router_choice_and_weights(E, top, count, keep):
    """Groups count by their best choice score; a group of one good expert beats one of two fair ones."""
    from vllm_b200 import ops
    g = torch.Generator().manual_seed(E)
    x, w = torch.randn(200, 20, generator=g), torch.randn(E, 20, generator=g) * 0.3
    corr = torch.randn(E, generator=g) * 0.3 - 0.5
    wt, ids = ops.router_topk(x, w, top, count, keep, True, "softmax", corr, 2.5, group_score="max")
    s = torch.softmax(x.double() @ w.double().T, -1)
    want = ko.choose(s, corr.double(), top, count, keep)
    assert torch.equal(ids.long(), want)
    sw = s.gather(1, want)
    torch.testing.assert_close(wt.double(), sw / sw.sum(-1, keepdim=True) * 2.5, rtol=1e-5, atol=1e-6)
    if keep < count and E // count > 1:
        _, other = ops.router_topk(x, w, top, count, keep, True, "softmax", corr, 2.5, group_score="top2")
        assert not torch.equal(other, ids)


def test_identity_experts_pass_the_input_on():
    from vllm_b200 import ops
    cfg = ko.config(16, 50, [(ko.memory(1, 4, 4), ko.moe(12, 5, 3, 3, (4, 3), 20, 1.4))])
    w = {k: v.double() for k, v in ko.make_weights(cfg, 5).items()}
    mlp = cfg["layers"][0]["mlp"]
    h = torch.randn(40, 16, generator=torch.Generator().manual_seed(6), dtype=torch.float64)
    s = torch.softmax(h @ w["l0.mlp.router"].T, -1)
    ids = ko.choose(s, w["l0.mlp.correction"], 3, 4, 3)
    assert (ids >= 5).any() and (ids < 5).any()
    sw = s.gather(1, ids)
    pw = (sw / sw.sum(-1, keepdim=True) * 1.4).float()
    w13 = torch.stack([torch.cat([w[f"l0.mlp.e{e}.gate"], w[f"l0.mlp.e{e}.up"]]) for e in range(5)]).float()
    w2 = torch.stack([w[f"l0.mlp.e{e}.down"] for e in range(5)]).float()
    emap = torch.tensor([0, 1, 2, 3, 4, -1, -1, -1], dtype=torch.int32)
    x = torch.zeros(40, 16)
    shared = ko.gated(h, w, "l0.mlp.shared.", ko.silu).float()
    ops.fused_moe_add_norm(x, h.float(), w13, w2, pw, ids.int(), "silu", emap, True, 5, shared, None, 0.0)
    torch.testing.assert_close(x.double(), ko.experts(h, w, "l0.mlp.", mlp), rtol=1e-4, atol=1e-4)


def test_stream_after_every_layer(tmp_path):
    cfg = ko.small()
    path, w = _model(tmp_path, cfg, 2)
    toks = tokens(cfg, 60)
    want = []
    ko.forward(cfg, w, toks, layers=want)
    with Engine(path, CPU32, 256) as e:
        got = []
        for layer in e.replay.core.model_executor.worker.get_model().model.layers:
            layer.register_forward_hook(lambda mod, args, out: got.append(args[1].clone()))
        e.feed([("a", toks, True)])
        assert len(got) == 6
        for g_, w_ in zip(got, want):
            torch.testing.assert_close(g_.double(), w_, rtol=2e-4, atol=2e-4)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(ko.MODELS))
def test_prompt_token_by_token_and_portions_agree_with_the_equations(tmp_path, place, name):
    cfg = ko.MODELS[name]()
    path, w = _model(tmp_path, cfg, 3, place=place)
    toks = tokens(cfg, 150)                                    # three pages
    want = ko.forward(cfg, w, toks)
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
    cfg = ko.small()
    path, w = _model(tmp_path, cfg, 4, place=place, input_bias=-2.0)
    with Engine(path, place) as e:
        for n in (1, 2, 3, 4):
            toks = tokens(cfg, n, n)
            e.feed([("a", toks, True)], *[[("b", [t], i == n - 1)] for i, t in enumerate(toks)])
            want = ko.forward(cfg, w, toks)
            assert row_error(e.logits("a"), want) < TOL[place[1]] and row_error(e.logits("b"), want) < TOL[place[1]]


@pytest.mark.parametrize("name", ["small", "wide"])
def test_unequal_requests_in_one_batch(tmp_path, place, name):
    """Portions beside single tokens; every request as if it were alone."""
    cfg = ko.MODELS[name]()
    path, w = _model(tmp_path, cfg, 5, place=place)
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
            assert row_error(e.logits(r), ko.forward(cfg, w, t)) < TOL[place[1]], r


def test_pages_and_slots_are_used_again(tmp_path, place):
    """Five pages and four slots serve many requests one after another; a new one never sees what a page or slot held."""
    cfg = ko.small()
    path, w = _model(tmp_path, cfg, 6, place=place, lasting=True, input_bias=1.0)
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
            assert row_error(e.logits(f"r{k}"), ko.forward(cfg, w, toks)) < TOL[place[1]], k
        e.feed([("keep", keep[96:], True)])
        assert row_error(e.logits("keep"), ko.forward(cfg, w, keep)) < TOL[place[1]]
        assert (mgr.pool.get_num_free_blocks(), mgr.state_pool.get_num_free_blocks()) == (free, slots)


# (key, query) positions: page borders, first and last places, near and far
PAIRS = [(0, 1), (0, 299), (63, 64), (64, 130), (1, 128), (127, 300), (128, 191), (191, 192), (298, 299)]


@pytest.mark.parametrize("reader", [0, 1])
@pytest.mark.parametrize("key,query", PAIRS)
def test_a_far_key_is_seen(tmp_path, place, key, query, reader):
    """One key far above the noise; the query in a prompt, in a short portion and decoded.  ``reader`` 1: the layer that looks at it
    has no keys of its own."""
    cfg = ko.config(64, 120, [(ko.attn(4, 2, 24, 16, 16), None), (ko.attn(4, 2, 24, 16, 8, scale=0.3, base=700.0, kv_from=0), ko.dense(40)),
                              (ko.memory(2, 8, 16), ko.dense(40))])
    X, Q = 11, 12
    path, w = _model(tmp_path, cfg, 7, place=place, change=lambda w: ko.plant_key(cfg, w, X, Q, reader))
    toks = tokens(cfg, query, key, avoid=(X, Q)) + [Q]
    toks[key] = X
    want = ko.forward(cfg, w, toks)[-1:]
    tol = TOL[place[1]]
    assert row_error(ko.forward(cfg, w, toks, hide=(key,))[-1:], want) > 3 * tol            # seeing it changes the logits
    with Engine(path, place) as e:
        e.feed([("whole", toks, True)], [("dec", toks[:-1])], [("dec", toks[-1:], True)])
        names = ["whole", "dec"]
        if query > 1:
            e.feed([("cut", toks[:-2])], [("cut", toks[-2:], True)])
            names.append("cut")
        for r in names:
            assert row_error(e.logits(r)[-1:], want) < tol, r


def test_rows_of_a_tile_whose_maxima_move_differently(tmp_path, place):
    """Scores that grow by far more than the lazy rescaling of the tensor-core kernel allows, in some rows of a tile and not in others."""
    cfg = ko.config(128, 120, [(ko.attn(2, 1, 128, 128, 48), ko.dense(64))])
    X, Q = 11, 12
    path, w = _model(tmp_path, cfg, 8, place=place, change=lambda w: ko.plant_key(cfg, w, X, Q, gain=2.5))
    toks = tokens(cfg, 600, 1, avoid=(X, Q))
    for i in (130, 300, 520):
        toks[i] = X
    for i in (140, 301, 302, 310, 400, 530, 599):
        toks[i] = Q
    want = ko.forward(cfg, w, toks)
    with Engine(path, place) as e:
        e.feed([("a", toks, True)], [("b", toks[:299])], [("b", toks[299:405])], [("b", toks[405:599])], [("b", toks[599:], True)])
        assert row_error(e.logits("a"), want) < TOL[place[1]] and row_error(e.logits("b"), want) < TOL[place[1]]


@pytest.mark.parametrize("bias", [-7.0, 0.0, 9.0])
def test_memories_of_weak_and_strong_inputs(tmp_path, place, bias):
    """Input gates so small that exp(-m) is the divisor, and so large that m carries the first tokens' size on."""
    cfg = ko.config(64, 96, [(ko.memory(2, 16, 24, cap=12.0), None), (ko.memory(3, 12, 20, cap=9.0), ko.dense(40))], eps=1e-3)
    path, w = _model(tmp_path, cfg, 9, place=place, input_bias=bias)
    toks = tokens(cfg, 300, 3)
    want = ko.forward(cfg, w, toks)
    with Engine(path, place) as e:
        e.feed([("a", toks, True)], [("b", toks[:257])], [("b", toks[257:259])], *[[("b", [t], i == 40)] for i, t in enumerate(toks[259:])])
        assert row_error(e.logits("a"), want) < TOL[place[1]] and row_error(e.logits("b"), want) < TOL[place[1]]


def test_states_remember_the_first_tokens(tmp_path, place):
    cfg = ko.config(64, 96, [(ko.memory(2, 16, 24), ko.dense(40)), (ko.memory(2, 12, 16), None)])
    path, w = _model(tmp_path, cfg, 10, place=place, lasting=True)
    a = tokens(cfg, 130, 1)
    b = [5] * 40 + a[40:]
    wa, wb = ko.forward(cfg, w, a), ko.forward(cfg, w, b)
    assert row_error(wa[-1:], wb[-1:]) > 2 * TOL["bfloat16"]
    with Engine(path, place) as e:
        e.feed([("a", a[:30]), ("b", b[:64])], [("b", b[64:125])], [("a", a[30:126]), ("b", b[125:127])], [("a", a[126:128])],
               [("a", a[128:129]), ("b", b[127:])], [("a", a[129:])])
        assert row_error(e.logits("a"), wa) < TOL[place[1]] and row_error(e.logits("b"), wb) < TOL[place[1]]


def test_no_query_sees_what_comes_after_it(tmp_path, place):
    cfg = ko.small()
    path, w = _model(tmp_path, cfg, 11, place=place)
    a, b = tokens(cfg, 140, 1), tokens(cfg, 140, 2)
    b[:70] = a[:70]
    with Engine(path, place) as e:
        e.feed([("a", a, True)], [("b", b, True)])
        la, lb = e.logits("a"), e.logits("b")
        assert row_error(la[:70], lb[:70]) < 1e-5 and row_error(la[70:], lb[70:]) > 0.3


def test_long_decoding(tmp_path, place):
    cfg = ko.config(64, 96, [(ko.attn(2, 1, 16, 24, 8), ko.moe(24, 4, 2, 2, (2, 1), 16)), (ko.memory(2, 12, 16), None)])
    path, w = _model(tmp_path, cfg, 12, place=place, lasting=True)
    toks = tokens(cfg, 300)
    with Engine(path, place) as e:
        e.feed([("a", toks[:5])], *[[("a", [t], i == 294)] for i, t in enumerate(toks[5:])])
        assert row_error(e.logits("a"), ko.forward(cfg, w, toks)) < TOL[place[1]]


def test_logits_are_capped(tmp_path, place):
    cfg = ko.middling()
    cfg["logit_softcap"] = 2.0
    path, w = _model(tmp_path, cfg, 13, place=place)
    toks = tokens(cfg, 30)
    want = ko.forward(cfg, w, toks)
    assert float(want.abs().max()) > 1.9
    with Engine(path, place) as e:
        e.feed([("a", toks, True)])
        got = e.logits("a")
        assert float(got.abs().max()) <= 2.0 and row_error(got, want) < TOL[place[1]]


# ------------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", ["small", "wide", "only_memory", "only_attention"])
def test_greedy_generation(tmp_path, place, name):
    """Through LLM.generate: chunked prompts (64 tokens a step), decode steps beside them, several requests."""
    cfg = ko.MODELS[name]()
    path, w = _model(tmp_path, cfg, 14, place=place)
    prompts = [tokens(cfg, n, n) for n in (1, 3, 40, 100, 130, 17)]
    llm = make_llm(path, place, kv_cache_memory_bytes=64 << 20)
    got = generate(llm, prompts, 12)
    assert all(len(g) == 12 for g in got)
    check_greedy(lambda t: ko.forward(cfg, w, t), prompts, got, 1e-3 if place[1] == "float32" else 0.25)
    if place[1] == "float32":
        assert got[2] == ko.greedy(cfg, w, prompts[2], 12)
    if place[0] == "cuda":
        runner = llm.llm_engine.engine_core.engine_core.model_executor.worker.runner
        assert runner.graphs and any(getattr(g, "replays", 0) for g in runner.graphs.values())    # decode steps replay graphs
    assert generate(llm, prompts[3:5], 4) == [g[:4] for g in got[3:5]]
    llm.shutdown()


def test_generation_with_preemption(tmp_path):
    """A pool that cannot hold all requests: some are put back and computed again, from an empty state."""
    cfg = ko.small()
    path, w = _model(tmp_path, cfg, 15, lasting=True)
    prompts = [tokens(cfg, n, n) for n in (60, 62, 50, 61)]
    llm = make_llm(path, CPU32, num_gpu_blocks_override=7, enable_prefix_caching=False)
    sched = llm.llm_engine.engine_core.engine_core.scheduler
    seen = []
    orig = sched._preempt
    sched._preempt = lambda r: (seen.append(r.request_id), orig(r))[1]
    got = generate(llm, prompts, 20)
    assert seen
    check_greedy(lambda t: ko.forward(cfg, w, t), prompts, got, 1e-3)
    llm.shutdown()


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(tensor_parallel_size=2, enable_expert_parallel=True),
                                dict(pipeline_parallel_size=2)], ids=["tp2", "ep2", "pp2"])
def test_parallel_ranks_generate_the_same(tmp_path, kw):
    cfg = ko.small()
    if "pipeline_parallel_size" in kw:                         # a shared cache lives on its stage
        cfg["layers"] = [cfg["layers"][i] for i in (0, 1, 4, 2)]
    path, w = _model(tmp_path, cfg, 16)
    prompts = [tokens(cfg, n, n) for n in (5, 70, 33)]
    llm = make_llm(path, CPU32, distributed_executor_backend="mp", **kw)
    got = generate(llm, prompts, 6)
    llm.shutdown()
    check_greedy(lambda t: ko.forward(cfg, w, t), prompts, got, 1e-3)


# ------------------------------------------------------------------------------------------------ the replay program
def test_trace_program(tmp_path, place):
    cfg = ko.small()
    path, w = _model(tmp_path, cfg, 17, place=place)
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
    la, lb = ko.forward(cfg, w, a), ko.forward(cfg, w, b)
    assert row_error(got[0], torch.stack([lb[19], lb[0], lb[7], la[69]])) < TOL[place[1]]
    assert row_error(got[1], lb[2:3]) < TOL[place[1]]


def test_kernel_sources_exist():
    from vllm_b200.csrc import build
    from vllm_b200.models.kopadra import KopadraForCausalLM
    have = {f[:-3] for f in os.listdir(build.HERE) if f.endswith(".cu")}
    for name, want in (("small", "attention_any"), ("wide", "attention_tc"), ("middling", "attention_simt"), ("only_memory", "linear_attn")):
        src = set(KopadraForCausalLM.kernel_sources(ko.MODELS[name](), torch.bfloat16))
        assert src <= have and want in src
    assert "attention_any" in KopadraForCausalLM.kernel_sources(ko.wide(), torch.float32)


@pytest.mark.parametrize("name", ["kopadra-tiny", "kopadra-small"])
def test_presets_are_valid(name):
    from vllm_b200.config import ModelConfig
    assert ModelConfig(model=name).architecture == "KopadraForCausalLM"
