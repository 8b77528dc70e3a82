"""Vurazen without a GPU: configuration, model description, tensor names and shapes, cache and state needs, and the plain
implementation's own properties (what a window, its kept tokens, a sink, the recurrences, the loop and the routing must and
must not do)."""
import copy
import json

import numpy as np
import pytest
import torch

import plain_vurazen as plain
from tiny_inference_engine_b200.config import load_config, parse_vurazen_config, vurazen_spec
from tiny_inference_engine_b200.errors import LoadError, UnsupportedError
from tiny_inference_engine_b200.parts.model import Model, expected_tensors
from tiny_inference_engine_b200.weights.loader import SafetensorsSource, bind_check

S, P, L, moe = plain.scan_layer, plain.parallel_layer, plain.lightning_layer, plain.moe
CFG = plain.make_config([S(inner=40, state=6, dt_rank=3, mlp=moe(ff=20, experts=6, top=3, shared_ff=28, limit=0.9, shared_limit=1.1)),
                         P(heads=6, kv_heads=3, dim=10, window=9, keep_first=4, rheads=4, rkv_heads=2, rdim=6, rvdim=14, conv=3, rconv=5),
                         L(heads=5, dim=6, vdim=10, mlp=None),
                         P(heads=2, kv_heads=2, dim=8, window=30, keep_first=0, rot=4, mlp=moe())], vocab=97, width=72, loop=(1, 3, 2))


def test_config_json_picks_the_architecture_and_every_size_comes_from_it(tmp_path):
    w = plain.random_weights(CFG, 1, ranks=(3, 7))
    plain.write_model_dir(tmp_path, CFG, w)
    arch, cfg, spec = load_config(tmp_path)
    assert arch.name == "Vurazen" and spec.architecture == "Vurazen"
    assert (spec.hidden_size, spec.vocab_size, len(spec.layers)) == (72, 97, 4)
    assert cfg.ranks == {1: (3, 7), 3: (3, 7)}            # read from the checkpoint's shapes: config.json has no key for them
    assert cfg.to_dict() == CFG
    model = Model(spec, torch.float32)
    assert {n: tuple(t.shape) for n, t in model.needs().items()} == {n: tuple(s) for n, s in plain.tensor_shapes(CFG, (3, 7)).items()}
    bind_check(model.needs(), SafetensorsSource(tmp_path), what="Vurazen")
    assert [l.mixer.kind for l in spec.layers] == ["selective_scan", "mixer_sum", "constant_decay_attention", "mixer_sum"]
    assert [None if l.ffn is None else l.ffn.kind for l in spec.layers] == ["feed_forward_sum", "swiglu", None, "feed_forward_sum"]
    assert all(l.block.kind == "shared_norm" and l.mixer_norm.kind == "layer_norm" and l.ffn_norm is None for l in spec.layers)
    assert spec.embedding["scale"] == 3.0 and spec.head["softcap"] == 25.0 and not spec.head["tied"]
    # the loop: each pass has entries (with caches and states) of its own; the embedding's output joins from the second pass on
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 1, 2, 3]
    assert [None if e.before is None else (e.before["index"], e.before["add_origin"]) for e in spec.run_order] == \
        [None, (0, False), None, (1, True), None, None]
    cache, state = model.cache_needs(), model.state_needs()
    assert [c is None for c in cache] == [True, False, True, False, True, False]
    assert (cache[1].kind, cache[1].kv_heads, cache[1].head_dim, cache[1].window, cache[1].keep_first) == ("window", 3, 10, 9, 4)
    assert cache[3] == cache[1] and cache[5].keep_first == 0
    assert state[0].shape == (40 * 6 + 3 * 40,) and state[2].shape == (5 * 6 * 10,)
    # both halves of a parallel layer keep state: one row behind the other, each on a 16-byte boundary
    left, right = 2 * (64 + 30), 4 * 6 * 14 + 4 * (2 * 12 + 56)       # q channels padded to 64, then k; S, then the last inputs
    assert state[1].shape == (left + right,) and model.layers[1].mixer.state_at == [(0, left), (left, left + right)]


def test_cache_groups_by_window_and_kept_tokens():
    from tiny_inference_engine_b200.cache.manager import CacheManager
    model = Model(vurazen_spec(parse_vurazen_config(CFG)), torch.float32)
    cm = CacheManager(model.cache_needs(), 8, num_pages=10, dtype=torch.float32)
    assert [(g.kind, g.kv_heads, g.head_dim, g.window, g.keep_first, g.entries) for g in cm.groups] == \
        [("window", 3, 10, 9, 4, (1, 3)), ("window", 2, 8, 30, 0, (5,))]


def test_what_the_configuration_rejects():
    def broken(change):
        cfg = copy.deepcopy(CFG)
        change(cfg)
        return cfg
    with pytest.raises(UnsupportedError, match="type 'mamba3'"):
        parse_vurazen_config(broken(lambda c: c["layers"][0].update(type="mamba3")))
    with pytest.raises(LoadError, match="no 'dt_rank'"):
        parse_vurazen_config(broken(lambda c: c["layers"][0]["mixer"].pop("dt_rank")))
    with pytest.raises(LoadError, match="differs from dim"):
        parse_vurazen_config(broken(lambda c: c["layers"][1]["mixer"]["left"].update(vdim=12)))
    with pytest.raises(LoadError, match="not a multiple"):
        parse_vurazen_config(broken(lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4)))
    with pytest.raises(LoadError, match="rot.dims"):
        parse_vurazen_config(broken(lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=12)))
    with pytest.raises(LoadError, match="keep_first"):
        parse_vurazen_config(broken(lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1)))
    with pytest.raises(LoadError, match="no 'right_scale'"):
        parse_vurazen_config(broken(lambda c: c["layers"][1]["mixer"].pop("right_scale")))
    with pytest.raises(LoadError, match="a number for each of the 5 heads"):
        parse_vurazen_config(broken(lambda c: c["layers"][2]["mixer"]["decay"].pop()))
    with pytest.raises(LoadError, match="cannot choose"):
        parse_vurazen_config(broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=7)))
    with pytest.raises(LoadError, match="shared has no 'limit'"):
        parse_vurazen_config(broken(lambda c: c["layers"][0]["mlp"]["shared"].pop("limit")))
    with pytest.raises(UnsupportedError, match="kind 'glu'"):
        parse_vurazen_config(broken(lambda c: c["layers"][1]["mlp"].update(kind="glu")))
    with pytest.raises(LoadError, match="does not name layers"):
        parse_vurazen_config(broken(lambda c: c["loop"].update(stop=5)))
    with pytest.raises(LoadError, match="no 'vocab'"):
        parse_vurazen_config(broken(lambda c: c.pop("vocab")))


def test_a_configuration_without_a_loop_a_cap_or_a_shared_expert():
    cfg = copy.deepcopy(CFG)
    cfg.pop("loop"), cfg.pop("logit_softcap"), cfg.pop("embedding")
    cfg["layers"][0]["mlp"].pop("shared")
    cfg["layers"][1]["mixer"]["left"].pop("mask")
    spec = vurazen_spec(parse_vurazen_config(cfg))
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 3] and all(e.before is None for e in spec.run_order)
    needs = expected_tensors(spec)
    assert "loop.step" not in needs and "l0.mlp.shared.gate" not in needs and needs["l1.mix.right.a1"].shape == (16, 72)
    model = Model(spec, torch.float32)
    assert model.cache_needs()[1].kind == "full" and model.embedding.scale == 1.0 and model.head.softcap == 0.0


def test_a_random_model_folder_from_a_configuration(tmp_path):
    from tiny_inference_engine_b200.cli.main import main
    cfg_path, out = tmp_path / "c.json", tmp_path / "m"
    cfg_path.write_text(json.dumps(CFG))
    assert main(["make-random", "--config", str(cfg_path), "--out", str(out), "--seed", "3", "--device", "cpu"]) == 0
    arch, cfg, spec = load_config(out)
    assert arch.name == "Vurazen" and cfg.ranks == {1: (16, 16), 3: (16, 16)}
    bind_check(Model(spec, torch.float32).needs(), SafetensorsSource(out), what="Vurazen")


def test_plain_windows_kept_tokens_and_recurrences_see_what_they_should():
    r = np.random.default_rng(0)
    toks = r.integers(0, 40, 23).tolist()
    other = list(toks)
    other[11] = (toks[11] + 1) % 40

    def moved(cfg, seed, at=other):
        w = plain.random_weights(cfg, seed)
        return np.abs(plain.forward(w, cfg, toks) - plain.forward(w, cfg, at)).max(axis=1) > 1e-9
    # the left mixer alone, a window of 5 and taps of 1: the rows whose window holds the changed token, and no other
    cfg = plain.make_config([P(window=5, keep_first=2, conv=1, right_scale=0.0, mlp=None)], vocab=40, width=32)
    assert moved(cfg, 2).tolist() == [11 <= i < 16 for i in range(23)]
    # a kept token moves every later row; the token behind the kept ones does not
    for at, seen in ((1, True), (2, False)):
        changed = list(toks)
        changed[at] = (toks[at] + 1) % 40
        assert moved(cfg, 2, changed)[at + 5:].all() == seen and moved(cfg, 2, changed)[at + 5:].any() == seen
    # taps reach further back: a changed token also changes the keys of the three tokens behind it
    cfg = plain.make_config([P(window=5, keep_first=0, conv=4, right_scale=0.0, mlp=None)], vocab=40, width=32)
    assert moved(cfg, 3).tolist() == [11 <= i < 19 for i in range(23)]
    # the recurrences: every later row moves, earlier rows do not
    for cfg in (plain.make_config([P(left_scale=0.0, mlp=None)], vocab=40, width=32), plain.make_config([S(mlp=None)], vocab=40, width=32),
                plain.make_config([L(mlp=None)], vocab=40, width=32)):
        assert moved(cfg, 4).tolist() == [i >= 11 for i in range(23)]
        w = plain.random_weights(cfg, 4)
        assert np.abs(plain.forward(w, cfg, toks[:9]) - plain.forward(w, cfg, toks)[:9]).max() < 1e-9


def test_plain_mechanisms_by_hand():
    assert plain.window_mask(5, 2, 1).astype(int).tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [1, 1, 1, 0, 0], [1, 0, 1, 1, 0], [1, 0, 0, 1, 1]]
    p = plain.softmax_with_sink(np.zeros((1, 3)), np.array([[True, True, False]]), np.log(2.0))
    assert np.allclose(p, [[0.25, 0.25, 0.0]])
    # rotation by a quarter turn of the first pair (2i with 2i+1), the rest passes
    x = plain.rotate_pairs(np.ones((1, 1, 4)), [np.pi / 2], 7.0, 2)
    assert np.allclose(x[0, 0], [-1.0, 1.0, 1.0, 1.0])
    assert np.allclose(plain.short_conv(np.array([[1.0], [2.0], [3.0]]), np.array([[10.0, 1.0]]))[:, 0], [1.0, 12.0, 23.0])
    # one channel, one state: S = exp(dt A) S + dt x B, y = S C + D x
    y = plain.selective_scan(np.array([[2.0], [3.0]]), np.array([[0.5], [1.0]]), np.array([[-np.log(2.0)]]), np.array([[1.0], [1.0]]),
                             np.array([[1.0], [10.0]]), np.array([0.25]))
    assert np.allclose(y[:, 0], [1.0 + 0.5, 10 * (0.5 * 1.0 + 3.0) + 0.75])
    # the delta rule writes what the (decayed) state does not say yet, and reads its own write
    k = np.array([[[1.0, 0.0]], [[1.0, 0.0]]])
    o = plain.delta_recurrence(k, k, np.array([[[4.0]], [[6.0]]]), np.ones((2, 1)), np.full((2, 1, 2), 0.5))
    assert np.allclose(o[:, 0, 0], [4.0, 6.0])
    o = plain.constant_decay_recurrence(np.ones((2, 1, 1)), np.ones((2, 1, 1)), np.array([[[4.0]], [[6.0]]]), [0.5])
    assert np.allclose(o[:, 0, 0], [4.0, 8.0])
    chosen, weights = plain.route(np.array([1.0, 3.0, 3.0, 0.0]), 2)
    assert chosen == [1, 2] and np.allclose(weights, 0.5)
    assert plain.run_order(CFG) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
