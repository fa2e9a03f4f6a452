"""Gizilorn: the configuration and checkpoint, each mechanism, and whole models through the engine's scheduler, cache and model runner,
against the plain implementation (tests/gizilorn_oracle.py).

Whole-model tests run on the CPU, and on the device in 16 and in 32 bits."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from tests import gizilorn_oracle as go
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


def _model(tmp_path, cfg, seed=0, change=None):
    w = go.make_weights(cfg, seed)
    if change:
        change(w)
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    return save_model(cfg, w, tmp_path / "model"), w


def _rand(*shape, seed=0, size=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * size


# ------------------------------------------------------------------------------------------------ configuration and checkpoint
def test_configuration_is_read_from_the_model_folder(tmp_path):
    from vllm_b200.config import ModelConfig
    from vllm_b200.models.registry import resolve_model_cls
    path, _ = _model(tmp_path, go.small())
    mc = ModelConfig(model=path)
    assert mc.architecture == "GizilornForCausalLM" and not mc.is_mla and not mc.is_moe
    assert (mc.vocab_size, mc.hidden_size, mc.num_layers) == (208, 96, 7)
    assert resolve_model_cls(mc.architecture).__name__ == "GizilornForCausalLM"
    assert mc.torch_dtype == torch.bfloat16


@pytest.mark.parametrize("layer,change", [
    (0, lambda m: m.update(kv_heads=4)), (0, lambda m: m["rot"].update(dims=7)), (0, lambda m: m["rot"].update(dims=26)),
    (0, lambda m: m.update(vdim=39)), (2, lambda m: m["mask"].update(size=0)), (1, lambda m: m.update(rot_dim=10)),
    (3, lambda m: m.update(kv_from=3)), (3, lambda m: m.update(kv_from=0)), (6, lambda m: m.update(kv_from=3)),
    (6, lambda m: m.update(kv_rank=48)), (6, lambda m: m["rot"].update(base=71.0))])
def test_sizes_that_do_not_fit_are_an_error(layer, change):
    from vllm_b200.config import ModelConfig
    cfg = go.small()
    change(cfg["layers"][layer]["mixer"])
    with pytest.raises(ValueError, match=f"layer {layer}"):
        ModelConfig(model="x", hf_config=cfg)


@pytest.mark.parametrize("name", sorted(go.MODELS))
def test_checkpoint_names_are_all_taken_and_none_else(tmp_path, name):
    path, w = _model(tmp_path, go.MODELS[name]())
    with Engine(path, CPU32, 256) as e:
        model = e.replay.core.model_executor.worker.get_model()
        loaded = model.load_weights((k, v.clone()) for k, v in w.items())
        assert loaded == {n for n, _ in model.named_parameters()}
        for bad in ("l0.mix.foo", "l1.mix.left.q", "l9.norm1", "l0x.norm1", "l0.hc3.in", "l0.mlp.gate", "l0.mix.o.b", "final.norm.b", "pos"):
            with pytest.raises(ValueError):
                model.load_weights([(bad, torch.zeros(48, 96))])


def test_a_layer_with_anothers_latents_has_no_tensors_of_them(tmp_path):
    path, _ = _model(tmp_path, go.small())
    with Engine(path, CPU32, 256) as e:
        model = e.replay.core.model_executor.worker.get_model()
        for bad in ("l3.mix.dkv", "l3.mix.dkv.norm", "l2.norm2", "l2.hc2.mix", "l1.mix.k", "l0.mix.uk"):
            with pytest.raises(ValueError):
                model.load_weights([(bad, torch.zeros(48, 96))])


def test_unknown_kinds_are_an_error(tmp_path):
    for i, change in enumerate((lambda c: c["layers"][1].update(type="other"), lambda c: c["layers"][1]["mlp"].update(kind="other"))):
        cfg = go.small()
        path, _ = _model(tmp_path / str(i), cfg)
        change(cfg)
        if i == 0:
            for l in cfg["layers"]:
                l["mixer"].pop("kv_from", None)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(cfg, f)
        with pytest.raises(ValueError, match="unknown"):
            Engine(path, CPU32, 256)


# ------------------------------------------------------------------------------------------------ caches
def test_one_block_table_serves_keys_and_latents_and_forgets_old_pages(tmp_path):
    cfg = go.small()                                           # the longest window is 129
    path, _ = _model(tmp_path, cfg)
    with Engine(path, CPU32, 512) as e:
        runner = e.replay.core.model_executor.worker.runner
        shapes = {n.split(".")[2]: tuple(c.shape) for n, c in runner.kv_caches.items()}
        assert shapes == {"0": (9, 2, 2, 64, 40), "1": (9, 64, 60), "2": (9, 2, 4, 64, 32), "4": (9, 64, 60), "5": (9, 2, 1, 64, 24)}
        mgr = e.replay.core.scheduler.kv_cache_manager
        assert mgr.num_groups == 1 and mgr.pool.get_num_free_blocks() == 8
        e.feed([("a", [1] * 192)])
        assert mgr.pool.get_num_free_blocks() == 5
        e.feed([("a", [1])])                                   # position 192 sees 64 and later ones: page 0 goes, page 3 comes
        assert mgr.pool.get_num_free_blocks() == 5
        e.feed([("a", [1] * 64)])
        e.feed([("a", [1] * 2, True)])
        assert mgr.pool.get_num_free_blocks() == 8


def test_a_request_may_fill_the_pool():
    """A window never needs more pages than the whole sequence."""
    from vllm_b200.core.kv_cache_manager import SlidingWindowMLASpec, SlidingWindowSpec, get_kv_cache_config, group_specs
    specs = {"a": SlidingWindowSpec(64, num_kv_heads=2, head_size=128, sliding_window=100),
             "b": SlidingWindowMLASpec(64, head_size=576, sliding_window=100), "c": SlidingWindowMLASpec(64, head_size=576, sliding_window=90)}
    assert [g.layer_names for g in group_specs(specs)] == [["a", "b"], ["c"]]
    del specs["c"]
    cfg, n = get_kv_cache_config(specs, 1 << 30, 512, num_gpu_blocks_override=9)
    assert n == 512 and cfg.num_blocks == 9
    with pytest.raises(ValueError, match="too small"):
        get_kv_cache_config(specs, 1 << 30, 512, num_gpu_blocks_override=8)


def test_a_shared_cache_must_be_kept_long_enough():
    from vllm_b200.layers.attention import MLAAttentionCore, clear_attention_layers
    clear_attention_layers()
    MLAAttentionCore(2, 32, 8, 1.0, prefix="own", sliding_window=50, cache_window=70)
    MLAAttentionCore(2, 32, 8, 1.0, prefix="near", kv_sharing_target="own", sliding_window=70)
    for kw in (dict(sliding_window=71), dict()):
        with pytest.raises(ValueError, match="further back"):
            MLAAttentionCore(2, 32, 8, 1.0, prefix="far", kv_sharing_target="own", **kw)
    clear_attention_layers()


# ------------------------------------------------------------------------------------------------ mechanisms (plain ops)
@pytest.mark.parametrize("S", [1, 2, 3, 5])
def test_hyper_connections(S):
    from vllm_b200 import ops
    x, y = _rand(7, S, 24, seed=1), _rand(7, 24, seed=2)
    into, out, mix, nxt, w = _rand(S, seed=3), _rand(S, seed=4), _rand(S, S, seed=5), _rand(S, seed=6), _rand(24, seed=7) + 1
    p = {"hc.in": into.double(), "hc.out": out.double(), "hc.mix": mix.double()}
    got = []
    want = go.hyper(x.double().transpose(0, 1), p, "hc.", lambda u: (got.append(u), y.double())[1])
    h = ops.hyper_step(x.clone(), None, None, into, w, 1e-3, torch.float32)
    torch.testing.assert_close(h.double(), go.rms_norm(got[0], w.double(), 1e-3), rtol=1e-5, atol=1e-5)
    xs = x.clone()
    h = ops.hyper_step(xs, y, torch.cat([out, mix.flatten()]), nxt, w, 1e-3)
    torch.testing.assert_close(xs.double().transpose(0, 1), want, rtol=1e-5, atol=1e-5)
    u = sum(nxt[s].double() * want[s] for s in range(S))
    torch.testing.assert_close(h.double(), go.rms_norm(u, w.double(), 1e-3), rtol=1e-4, atol=1e-5)


def test_mix_weights_are_indexed_from_then_to():
    from vllm_b200 import ops
    x = torch.zeros(1, 2, 4)
    x[0, 0] = 1.0
    coef = torch.tensor([0.0, 0.0, 0.0, 1.0, 0.0, 0.0])       # out = 0, mix[0, 1] = 1: stream 0 goes to stream 1
    ops.hyper_step(x, torch.ones(1, 4), coef, torch.ones(2), torch.ones(4), 1e-6)
    assert x[0, 0].eq(0).all() and x[0, 1].eq(1).all()


def test_streams_start_as_the_normed_embedding():
    from vllm_b200 import ops
    table, we, w, into = _rand(11, 16, seed=1) * 3, _rand(16, seed=2) + 1, _rand(16, seed=3) + 1, torch.tensor([0.5, -2.0, 0.25])
    ids = torch.tensor([4, 0, 10, 4], dtype=torch.int32)
    x, h = ops.hyper_entry(ids, table, 3, we, into, w, 1e-2)
    e = go.rms_norm(table[ids.long()].double(), we.double(), 1e-2)
    for s in range(3):
        torch.testing.assert_close(x[:, s].double(), e, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(h.double(), go.rms_norm(-1.25 * e, w.double(), 1e-2), rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("p,q", [(0.3, -1.2), (-40.0, 30.0), (25.0, -60.0)])
def test_xielu(p, q):
    from vllm_b200.layers.common import XIELU
    act = XIELU()
    act.weight_loader(act.coef, torch.tensor([p, q]))
    z = torch.tensor([-200.0, -30.0, -3.0, -1e-3, -1e-6, 0.0, 1e-6, 0.2, 4.0, 100.0])
    torch.testing.assert_close(act(z).double(), go.xielu(z.double(), p, q), rtol=1e-5, atol=1e-9)


def test_values_turn_forward_into_the_cache_and_back_in_the_output():
    """A value reaches the output turned by the distance between its position and the query's, whatever the positions are."""
    v = _rand(9, 1, 10, seed=1).double()
    back = go.turn(go.turn(v, 50.0, 10, True, first=70), 50.0, 10, True, back=True, first=70)
    torch.testing.assert_close(back, v)
    a = go.turn(go.turn(v, 50.0, 10, True, first=70), 50.0, 10, True, back=True, first=75)
    b = go.turn(go.turn(v, 50.0, 10, True, first=0), 50.0, 10, True, back=True, first=5)
    torch.testing.assert_close(a, b)
    from vllm_b200.layers.rotary import get_rope
    rope = get_rope(10, 10, 100, 50.0, True, dict(exact=True))
    got, _ = rope(torch.arange(70, 79), v.float().view(9, 10).clone(), None)
    torch.testing.assert_close(got.double(), go.turn(v, 50.0, 10, True, first=70).view(9, 10), rtol=1e-5, atol=1e-6)


def test_the_sink_takes_weight_and_is_not_mixed():
    """One visible key of score s: weight e^s / (1 + e^s); a talk matrix of zeros leaves nothing."""
    q, k, v = _rand(1, 2, 4, seed=1).double(), _rand(1, 1, 4, seed=2).double(), _rand(1, 1, 6, seed=3).double()
    s = 5 * torch.tanh((q[0] @ k[0, 0]) * 0.5 / 5)
    w = torch.exp(s) / (1 + torch.exp(s))
    talk = _rand(2, 2, seed=4).double()
    torch.testing.assert_close(go.talking_attention(q, k, v, 0.5, 5.0, 9, talk)[0], (talk @ w)[:, None] * v[0, 0])
    assert go.talking_attention(q, k, v, 0.5, 5.0, 9, torch.zeros(2, 2)).eq(0).all()


@pytest.mark.parametrize("H,G", [(6, 2), (4, 4), (3, 1)])
def test_mixed_heads_over_pages(H, G):
    from types import SimpleNamespace
    from vllm_b200 import ops
    n, d, dv, W = 150, 12, 20, 40
    q, k, v, talk = _rand(n, H, d, seed=1), _rand(n, G, d, seed=2), _rand(n, G, dv, seed=3), _rand(H, H, seed=4)
    cache = torch.full((6, 2, G, 64, dv), 9.0)
    table = torch.tensor([[4, 1, 5, 0]], dtype=torch.int32)
    for j in range(n):
        cache[table[0, j // 64], 0, :, j % 64, :d], cache[table[0, j // 64], 1, :, j % 64] = k[j], v[j]
    want = go.talking_attention(q.double(), k.double(), v.double(), 0.6, 2.0, W, talk.double())
    for first in (0, 149, 100):
        md = SimpleNamespace(block_table=table, seq_lens=torch.tensor([n]), query_start_loc=torch.tensor([0, n - first]), seq_lens_cpu=None,
                             query_start_loc_cpu=None)
        got = ops.talking_attention(q[first:], cache, md, 0.6, W, 2.0, talk, torch.zeros(H), dv)
        torch.testing.assert_close(got.double(), want[first:], rtol=1e-4, atol=1e-5)


def test_streams_after_every_layer(tmp_path):
    cfg = go.small()
    path, w = _model(tmp_path, cfg, 2)
    toks = tokens(cfg, 60)
    want = []
    go.forward(cfg, w, toks, layers=want)
    with Engine(path, CPU32, 256) as e:
        model = e.replay.core.model_executor.worker.get_model().model
        from vllm_b200 import ops
        got, orig = [], ops.hyper_step
        ops.hyper_step = lambda x, *a: (orig(x, *a), got.append(x.sum(1)))[0]
        try:
            e.feed([("a", toks, True)])
        finally:
            ops.hyper_step = orig
        ends = np.cumsum([1 + (layer.mlp is not None) for layer in model.layers]) - 1
        assert len(got) == ends[-1] + 1
        for i, t in zip(ends, want):
            torch.testing.assert_close(got[i].double(), t, rtol=2e-4, atol=2e-4)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(go.MODELS))
def test_prompt_token_by_token_and_portions_agree_with_the_equations(tmp_path, place, name):
    cfg = go.MODELS[name]()
    path, w = _model(tmp_path, cfg, 3)
    toks = tokens(cfg, 150)                                    # three pages
    want = go.forward(cfg, w, toks)
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


def test_long_prompts(tmp_path, place):
    """Several tiles of queries and keys, windows shorter and longer than a tile."""
    cfg = go.wide()
    cfg["layers"][2]["mixer"]["mask"]["size"] = 300
    path, w = _model(tmp_path, cfg, 4)
    a, b = tokens(cfg, 500, 1), tokens(cfg, 390, 2)
    with Engine(path, place) as e:
        e.feed([("a", a, True), ("b", b[:260])], [("b", b[260:], True)])
        assert row_error(e.logits("a"), go.forward(cfg, w, a)) < TOL[place[1]]
        assert row_error(e.logits("b"), go.forward(cfg, w, b)) < TOL[place[1]]


def test_first_tokens(tmp_path, place):
    """A sequence's first tokens have few keys: there the sink takes a good part of the weight."""
    cfg = go.small()
    path, w = _model(tmp_path, cfg, 5)
    with Engine(path, place) as e:
        for n in (1, 2, 3, 4):
            toks = tokens(cfg, n, n)
            e.feed([("a", toks, True)], *[[("b", [t], i == n - 1)] for i, t in enumerate(toks)])
            want = go.forward(cfg, w, toks)
            assert row_error(e.logits("a"), want) < TOL[place[1]] and row_error(e.logits("b"), want) < TOL[place[1]]
    orig = go.sink_weights
    go.sink_weights = go.softmax_weights
    try:
        assert row_error(go.forward(cfg, w, toks), want) > 3 * TOL["bfloat16"]
    finally:
        go.sink_weights = orig


@pytest.mark.parametrize("name", ["small", "wide"])
def test_unequal_requests_in_one_batch(tmp_path, place, name):
    """Portions beside single tokens; every request as if it were alone."""
    cfg = go.MODELS[name]()
    path, w = _model(tmp_path, cfg, 6)
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
            assert row_error(e.logits(r), go.forward(cfg, w, t)) < TOL[place[1]], r


def test_pages_are_used_again(tmp_path, place):
    """Five pages serve many requests one after another; a new one never sees what a page held."""
    cfg = go.small()
    path, w = _model(tmp_path, cfg, 7)
    with Engine(path, place, 5 * 64) as e:
        mgr = e.replay.core.scheduler.kv_cache_manager
        free = mgr.pool.get_num_free_blocks()
        assert free == 5
        keep = tokens(cfg, 100, 50)                            # stays while the others come and go
        e.feed([("keep", keep[:60])])
        for k in range(9):
            n = (64, 65, 130, 2, 128, 127, 1, 3, 100)[k]
            toks = tokens(cfg, n, k)
            cut = max(1, n // 2)
            e.feed([(f"r{k}", toks[:cut], n == 1), ("keep", keep[60 + 4 * k:64 + 4 * k])], *([[(f"r{k}", toks[cut:], True)]] if n > 1 else []))
            assert row_error(e.logits(f"r{k}"), go.forward(cfg, w, toks)) < TOL[place[1]], k
        e.feed([("keep", keep[96:], True)])
        assert row_error(e.logits("keep"), go.forward(cfg, w, keep)) < TOL[place[1]]
        assert mgr.pool.get_num_free_blocks() == free


def test_pages_behind_the_windows_serve_others_at_once(tmp_path, place):
    """A long decode gives pages back; another request takes them while the first goes on."""
    cfg = go.only_latent()                                     # windows of 40 and 70
    path, w = _model(tmp_path, cfg, 8)
    a, b = tokens(cfg, 260, 1), tokens(cfg, 120, 2)
    with Engine(path, place, 6 * 64) as e:
        e.feed([("a", a[:180])], *[[("a", [t])] for t in a[180:200]], [("a", a[200:201]), ("b", b[:119])], [("b", b[119:], True), ("a", a[201:203])],
               [("a", a[203:], True)])
        assert row_error(e.logits("a"), go.forward(cfg, w, a)) < TOL[place[1]]
        assert row_error(e.logits("b"), go.forward(cfg, w, b)) < TOL[place[1]]


READERS = {"attention": [(go.attn(4, 2, 24, 16, 16, 100, softcap=30.0), None), (go.latent(2, 8, 4, 16, 24, 30), 40)],
           "attention-wide": [(go.attn(4, 2, 128, 128, 96, 100, softcap=30.0), None), (go.latent(2, 8, 4, 16, 24, 30), 40)],
           "latent": [(go.latent(3, 16, 8, 24, 32, 100, scale=0.3), None), (go.attn(2, 1, 8, 16, 8, 30), 40)],
           "shared": [(go.latent(3, 16, 8, 24, 32, 30, scale=0.3), None), (go.latent(2, 24, 8, 16, 32, 100, scale=0.3, kv_from=0), 40)]}


def _planted(tmp_path, kind, window, X=11, Q=12):
    cfg = go.config(64, 120, READERS[kind], 2)
    layer = 1 if kind == "shared" else 0
    cfg["layers"][layer]["mixer"]["mask"]["size"] = window
    path, w = _model(tmp_path, cfg, 9, change=lambda w: go.plant_key(cfg, w, X, Q, layer))
    return cfg, path, w


def _asked(e, toks):
    """Logits of the last token: in a prompt, decoded, and in a portion of two."""
    e.feed([("whole", toks, True)], [("dec", toks[:-1])], [("dec", toks[-1:], True)])
    out = [e.logits("whole")[-1:], e.logits("dec")[-1:]]
    if len(toks) > 2:
        e.feed([("cut", toks[:-2])], [("cut", toks[-2:], True)])
        out.append(e.logits("cut")[-1:])
    return out


# (window, query): page and tile borders on either side of the window's edge
EDGES = [(2, 64), (63, 127), (64, 128), (65, 129), (100, 163), (100, 227), (128, 191), (129, 300), (200, 263)]


@pytest.mark.parametrize("kind", sorted(READERS))
@pytest.mark.parametrize("window,query", EDGES)
def test_the_windows_edge(tmp_path, place, kind, window, query):
    """The last key inside the window is seen, the next one is not."""
    X, Q = 11, 12
    cfg, path, w = _planted(tmp_path, kind, window)
    tol = TOL[place[1]]
    with Engine(path, place) as e:
        for inside in (True, False):
            key = query - window + (1 if inside else 0)
            toks = tokens(cfg, query, key, avoid=(X, Q)) + [Q]
            toks[key] = X
            want = go.forward(cfg, w, toks)[-1:]
            wider = dict(cfg, layers=[dict(l, mixer=dict(l["mixer"], mask=dict(size=l["mixer"]["mask"]["size"] + 1))) for l in cfg["layers"]])
            other = go.forward(cfg, w, toks, hide=(key,))[-1:] if inside else go.forward(wider, w, toks)[-1:]
            assert row_error(other, want) > 3 * tol            # it makes a difference
            for got in _asked(e, toks):
                assert row_error(got, want) < tol, inside


@pytest.mark.parametrize("kind", sorted(READERS))
@pytest.mark.parametrize("key,query", [(0, 1), (0, 299), (63, 64), (64, 130), (1, 128), (127, 300), (128, 191), (298, 299)])
def test_a_far_key_is_seen(tmp_path, place, kind, key, query):
    X, Q = 11, 12
    cfg, path, w = _planted(tmp_path, kind, 320)
    toks = tokens(cfg, query, key, avoid=(X, Q)) + [Q]
    toks[key] = X
    want = go.forward(cfg, w, toks)[-1:]
    tol = TOL[place[1]]
    assert row_error(go.forward(cfg, w, toks, hide=(key,))[-1:], want) > 3 * tol
    with Engine(path, place) as e:
        for got in _asked(e, toks):
            assert row_error(got, want) < tol


@pytest.mark.parametrize("cap", [0.5, 8.0, 60.0, 200.0])
@pytest.mark.parametrize("dim", [24, 128])
def test_caps_of_every_size(tmp_path, place, cap, dim):
    """Scores far below, around and far above the cap; caps that the tensor-core kernels do not take."""
    cfg = go.config(64, 90, [(go.attn(4, 2, dim, dim, dim // 2, 50, softcap=cap, scale=0.5 if cap < 100 else 1.0), 40)], 2)
    path, w = _model(tmp_path, cfg, 10)
    toks = tokens(cfg, 140)
    want = go.forward(cfg, w, toks)
    with Engine(path, place) as e:
        e.feed([("a", toks, True)], [("b", toks[:120])], *[[("b", [t], i == 19)] for i, t in enumerate(toks[120:])])
        assert row_error(e.logits("a"), want) < 1.5 * TOL[place[1]] and row_error(e.logits("b"), want) < 1.5 * TOL[place[1]]


def test_no_query_sees_what_comes_after_it(tmp_path, place):
    cfg = go.small()
    path, w = _model(tmp_path, cfg, 11)
    a, b = tokens(cfg, 140, 1), tokens(cfg, 140, 2)
    b[:70] = a[:70]
    with Engine(path, place) as e:
        e.feed([("a", a, True)], [("b", b, True)])
        la, lb = e.logits("a"), e.logits("b")
        assert row_error(la[:70], lb[:70]) < 1e-5 and row_error(la[70:], lb[70:]) > 0.3


@pytest.mark.parametrize("name", ["only_latent", "only_attention", "plain"])
def test_long_decoding(tmp_path, place, name):
    cfg = go.MODELS[name]()
    path, w = _model(tmp_path, cfg, 12)
    toks = tokens(cfg, 300)
    with Engine(path, place) as e:
        e.feed([("a", toks[:5])], *[[("a", [t], i == 294)] for i, t in enumerate(toks[5:])])
        assert row_error(e.logits("a"), go.forward(cfg, w, toks)) < TOL[place[1]]


# ------------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", ["small", "wide", "broad", "only_latent"])
def test_greedy_generation(tmp_path, place, name):
    """Through LLM.generate: chunked prompts (64 tokens a step), decode steps beside them, several requests."""
    cfg = go.MODELS[name]()
    path, w = _model(tmp_path, cfg, 14)
    prompts = [tokens(cfg, n, n) for n in (1, 3, 40, 100, 130, 17)]
    llm = make_llm(path, place, kv_cache_memory_bytes=256 << 20)
    got = generate(llm, prompts, 12)
    assert all(len(g) == 12 for g in got)
    check_greedy(lambda t: go.forward(cfg, w, t), prompts, got, 1e-3 if place[1] == "float32" else 0.25)
    if place[1] == "float32":
        assert got[2] == go.greedy(cfg, w, prompts[2], 12)
    if place[0] == "cuda":
        runner = llm.llm_engine.engine_core.engine_core.model_executor.worker.runner
        assert runner.graphs and any(getattr(g, "replays", 0) for g in runner.graphs.values())    # decode steps replay graphs
    assert generate(llm, prompts[3:5], 4) == [g[:4] for g in got[3:5]]                            # (from the prefix cache)
    llm.shutdown()


def test_generation_with_preemption(tmp_path):
    """A pool that cannot hold all requests: some are put back and computed again."""
    cfg = go.small()
    path, w = _model(tmp_path, cfg, 15)
    prompts = [tokens(cfg, n, n) for n in (60, 62, 50, 61)]
    llm = make_llm(path, CPU32, num_gpu_blocks_override=7, enable_prefix_caching=False)
    sched = llm.llm_engine.engine_core.engine_core.scheduler
    seen = []
    orig = sched._preempt
    sched._preempt = lambda r: (seen.append(r.request_id), orig(r))[1]
    got = generate(llm, prompts, 20)
    assert seen
    check_greedy(lambda t: go.forward(cfg, w, t), prompts, got, 1e-3)
    llm.shutdown()


@pytest.mark.parametrize("kw", [dict(tensor_parallel_size=2), dict(pipeline_parallel_size=2)], ids=["tp2", "pp2"])
def test_parallel_ranks_generate_the_same(tmp_path, kw):
    cfg = go.small()
    if "pipeline_parallel_size" in kw:                         # a shared cache lives on its stage
        cfg["layers"] = [cfg["layers"][i] for i in (0, 1, 2, 5)]
    path, w = _model(tmp_path, cfg, 16)
    prompts = [tokens(cfg, n, n) for n in (5, 70, 33)]
    llm = make_llm(path, CPU32, distributed_executor_backend="mp", **kw)
    got = generate(llm, prompts, 6)
    llm.shutdown()
    check_greedy(lambda t: go.forward(cfg, w, t), prompts, got, 1e-3)


# ------------------------------------------------------------------------------------------------ the replay program
def test_trace_program(tmp_path, place):
    cfg = go.small()
    path, w = _model(tmp_path, cfg, 17)
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
    la, lb = go.forward(cfg, w, a), go.forward(cfg, w, b)
    assert row_error(got[0], torch.stack([lb[19], lb[0], lb[7], la[69]])) < TOL[place[1]]
    assert row_error(got[1], lb[2:3]) < TOL[place[1]]


def test_kernel_sources_exist():
    from vllm_b200.csrc import build
    from vllm_b200.models.gizilorn import GizilornForCausalLM
    have = {f[:-3] for f in os.listdir(build.HERE) if f.endswith(".cu")}
    for name, want in (("small", "attention_any"), ("wide", "attention_talk_decode"), ("only_latent", "mla_prefill")):
        src = set(GizilornForCausalLM.kernel_sources(go.MODELS[name](), torch.bfloat16))
        assert src <= have and want in src
    assert "attention_any" in GizilornForCausalLM.kernel_sources(go.wide(), torch.float32)


@pytest.mark.parametrize("name", ["gizilorn-tiny", "gizilorn-small"])
def test_presets_are_valid(name):
    from vllm_b200.config import ModelConfig
    assert ModelConfig(model=name).architecture == "GizilornForCausalLM"
