"""Sebalorn without a GPU: configuration, model description, tensor names and shapes, cache and state needs, and the plain
implementation's own properties (what rotations, sinks, the recurrence, the norm over a whole projection and the loop must do)."""
import copy
import json

import numpy as np
import pytest
import torch

import plain_sebalorn as plain
from tiny_inference_engine_b200.config import load_config, parse_sebalorn_config, sebalorn_spec
from tiny_inference_engine_b200.errors import InvalidArgument, LoadError, UnsupportedError
from tiny_inference_engine_b200.parts.model import Model, expected_tensors
from tiny_inference_engine_b200.weights.loader import SafetensorsSource, bind_check

LA, A, R = plain.latent_layer, plain.attention_layer, plain.retention_layer
CFG = plain.make_config([A(heads=6, kv_heads=3, dim=10, vdim=14, rot=4, mlp=plain.dense(40)), LA(heads=5, dim=6, rot_dim=8, vdim=11, kv_rank=21, q_rank=18),
                         R(heads=4, dim=12, vdim=9, rot=6, mlp=None), LA(heads=2, mlp=plain.dense(31))], vocab=97, width=72, loop=(1, 3, 2))


def test_config_json_picks_the_architecture_and_every_size_comes_from_it(tmp_path):
    w = plain.random_weights(CFG, 1)
    plain.write_model_dir(tmp_path, CFG, w)
    arch, cfg, spec = load_config(tmp_path)
    assert arch.name == "Sebalorn" and spec.architecture == "Sebalorn"
    assert (spec.hidden_size, spec.vocab_size, len(spec.layers)) == (72, 97, 4)
    assert cfg.to_dict() == CFG
    model = Model(spec, torch.float32)
    needs = {n: tuple(t.shape) for n, t in model.needs().items() if not t.optional}
    assert needs == {n: tuple(s) for n, s in plain.tensor_shapes(CFG).items()}
    bind_check(model.needs(), SafetensorsSource(tmp_path), what="Sebalorn")
    assert [l.mixer.kind for l in spec.layers] == ["gated_window_attention", "latent_attention", "constant_decay_attention", "latent_attention"]
    assert [None if l.ffn is None else (l.ffn.kind, l.ffn["intermediate_size"]) for l in spec.layers] == \
        [("squared_relu_mlp", 40), ("squared_relu_mlp", 72), None, ("squared_relu_mlp", 31)]
    assert all(l.block.kind == "shared_norm" and l.mixer_norm.kind == "rmsnorm_one_plus" and l.ffn_norm is None for l in spec.layers)
    assert spec.embedding["scale"] == 3.0 and spec.head["softcap"] == 25.0 and not spec.head["tied"]
    # the loop: each pass has entries (with caches and states) of its own, and a vector of its own joins ahead of it
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 1, 2, 3]
    assert [None if e.before is None else e.before["index"] for e in spec.run_order] == [None, 0, None, 1, None, None]
    assert not any(p.reads_origin for p in model.stream_inputs.values())
    cache, state = model.cache_needs(), model.state_needs()
    assert (cache[0].kind, cache[0].kv_heads, cache[0].head_dim, cache[0].value_dim) == ("full", 3, 10, 14)
    assert (cache[1].kind, cache[1].kv_heads, cache[1].head_dim, cache[1].value_dim) == ("full", 1, 21 + 8, -1)      # latent and key part, no values
    assert cache[3] == cache[1] and cache[2] is None and state[2].shape == (4 * 12 * 9,) and state[4] == state[2] and state[0] is None
    # pairs and angles of the three rotations
    lay = model.layers
    assert lay[1].mixer.position.neighbours and not lay[0].mixer.position.neighbours and not lay[2].mixer.position.neighbours
    assert all(lay[i].mixer.position.double_angles for i in range(3)) and [lay[i].mixer.position.rotary_dim for i in range(3)] == [4, 8, 6]
    assert lay[0].mixer.output_gate == "head" and lay[1].mixer.output_gate == "channel" and lay[2].mixer.k_scale == 12 ** -0.5


def test_cache_groups_and_their_bytes():
    from tiny_inference_engine_b200.cache.manager import CacheManager
    model = Model(sebalorn_spec(parse_sebalorn_config(CFG)), torch.float32)
    cm = CacheManager(model.cache_needs(), 8, num_pages=10, dtype=torch.float32)
    assert [(g.kind, g.kv_heads, g.head_dim, g.value_dim, g.entries) for g in cm.groups] == \
        [("full", 3, 10, 14, (0,)), ("full", 1, 29, -1, (1, 3)), ("full", 1, 30, -1, (5,))]
    assert cm.bytes_per_page == 8 * 4 * (3 * 24 + 2 * 29 + 30)


def test_what_the_configuration_rejects():
    def broken(change):
        cfg = copy.deepcopy(CFG)
        change(cfg)
        return cfg
    mixer = lambda c, i: c["layers"][i]["mixer"]
    with pytest.raises(UnsupportedError, match="type 'retention2'"):
        parse_sebalorn_config(broken(lambda c: c["layers"][2].update(type="retention2")))
    for key in ("q_rank", "kv_rank", "rot_dim", "vdim", "scale"):
        with pytest.raises(LoadError, match=f"no '{key}'"):
            parse_sebalorn_config(broken(lambda c: mixer(c, 1).pop(key)))
    with pytest.raises(LoadError, match="the whole rotated part"):
        parse_sebalorn_config(broken(lambda c: mixer(c, 1)["rot"].update(dims=6)))
    with pytest.raises(LoadError, match="rot.dims 12"):
        parse_sebalorn_config(broken(lambda c: mixer(c, 0)["rot"].update(dims=12)))
    with pytest.raises(LoadError, match="rot.dims 3"):
        parse_sebalorn_config(broken(lambda c: mixer(c, 2)["rot"].update(dims=3)))
    with pytest.raises(LoadError, match="base must be positive"):
        parse_sebalorn_config(broken(lambda c: mixer(c, 2)["rot"].update(base=0)))
    with pytest.raises(LoadError, match="not a multiple"):
        parse_sebalorn_config(broken(lambda c: mixer(c, 0).update(kv_heads=4)))
    with pytest.raises(LoadError, match="a number for each of the 4 heads"):
        parse_sebalorn_config(broken(lambda c: mixer(c, 2)["decay"].pop()))
    with pytest.raises(UnsupportedError, match="kind 'moe'"):
        parse_sebalorn_config(broken(lambda c: c["layers"][0]["mlp"].update(kind="moe")))
    with pytest.raises(LoadError, match="no 'ff'"):
        parse_sebalorn_config(broken(lambda c: c["layers"][0]["mlp"].pop("ff")))
    with pytest.raises(LoadError, match="does not name layers"):
        parse_sebalorn_config(broken(lambda c: c["loop"].update(stop=5)))
    with pytest.raises(LoadError, match="no 'vocab'"):
        parse_sebalorn_config(broken(lambda c: c.pop("vocab")))


def test_parts_reject_options_they_do_not_know():
    from tiny_inference_engine_b200.config.spec import PartSpec
    from tiny_inference_engine_b200.parts import build_part
    def part(family, kind, **params):
        return build_part(family, PartSpec(kind, params), torch.float32)
    with pytest.raises(InvalidArgument, match="halves or neighbours"):
        part("position", "rope", theta=10.0, head_dim=8, pairing="thirds")
    latent = dict(hidden_size=8, num_heads=2, head_dim=4, rot_dim=0, value_dim=4, kv_rank=4, q_rank=4)
    with pytest.raises(InvalidArgument, match="output_gate"):
        part("mixer", "latent_attention", **latent, output_gate="row")
    assert part("mixer", "latent_attention", **latent).needs()["g"].shape == (2, 8)                # a gate per head, as before
    assert "sink" not in part("mixer", "latent_attention", **latent).needs()
    linear = dict(hidden_size=8, num_heads=2, head_dim=4, value_dim=4, decay=[0.5, 0.5])
    with pytest.raises(InvalidArgument, match="without an activation"):
        part("mixer", "constant_decay_attention", **linear, k_scale=0.5)
    assert part("mixer", "constant_decay_attention", **linear).needs()["norm"].shape == (8,)
    assert part("mixer", "constant_decay_attention", **linear, norm_per_head=True).needs()["norm"].shape == (4,)


def test_a_configuration_without_a_loop_a_cap_or_a_rotation():
    cfg = copy.deepcopy(CFG)
    cfg.pop("loop"), cfg.pop("logit_softcap"), cfg.pop("embedding")
    cfg["layers"][0]["mixer"]["rot"]["dims"] = 0
    cfg["layers"][1]["mixer"].update(rot_dim=0, rot={"base": 10.0, "dims": 0})
    cfg["layers"][2]["mixer"].pop("rot")
    spec = sebalorn_spec(parse_sebalorn_config(cfg))
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 3] and all(e.before is None for e in spec.run_order)
    assert "loop.step" not in expected_tensors(spec)
    model = Model(spec, torch.float32)
    assert model.embedding.scale == 1.0 and model.head.softcap == 0.0
    assert model.layers[0].mixer.position.is_identity and model.layers[1].mixer.position is None and model.layers[2].mixer.position is None


def test_a_random_model_folder_from_a_configuration(tmp_path):
    from tiny_inference_engine_b200.cli.main import main
    cfg_path, out = tmp_path / "c.json", tmp_path / "m"
    cfg_path.write_text(json.dumps(CFG))
    assert main(["make-random", "--config", str(cfg_path), "--out", str(out), "--seed", "3", "--device", "cpu"]) == 0
    arch, cfg, spec = load_config(out)
    assert arch.name == "Sebalorn"
    bind_check(Model(spec, torch.float32).needs(), SafetensorsSource(out), what="Sebalorn")


def test_plain_mixers_see_every_earlier_token_and_no_later_one():
    toks = np.random.default_rng(0).integers(0, 40, 19).tolist()
    other = list(toks)
    other[11] = (toks[11] + 1) % 40
    for layer in (LA(mlp=None), A(mlp=None), R(mlp=None), R(mlp="dense")):
        cfg = plain.make_config([layer], vocab=40, width=32)
        w = plain.random_weights(cfg, 4)
        moved = np.abs(plain.forward(w, cfg, toks) - plain.forward(w, cfg, other)).max(axis=1) > 1e-9
        assert moved.tolist() == [i >= 11 for i in range(19)]
        assert np.abs(plain.forward(w, cfg, toks[:9]) - plain.forward(w, cfg, toks)[:9]).max() < 1e-9


def test_plain_mechanisms_by_hand():
    # a quarter turn of the first pair: neighbours 0 and 1, or 0 and 2 (halves of 4); what is not rotated passes
    x = np.array([[[1.0, 2.0, 3.0, 4.0, 5.0]]])
    turned = plain.rotate_neighbours(x, [np.pi / 2], 1e30, 4)[0, 0]
    assert np.allclose(turned, [-2.0, 1.0, 3.0, 4.0, 5.0])
    turned = plain.rotate_halves(x, [np.pi / 2], 1e30, 4)[0, 0]
    assert np.allclose(turned, [-3.0, 2.0, 1.0, 4.0, 5.0])
    p = plain.causal_softmax(np.zeros((2, 2)), np.log(2.0))
    assert np.allclose(p, [[1 / 3, 0.0], [0.25, 0.25]]) and np.allclose(plain.causal_softmax(np.zeros((2, 2))), [[1.0, 0.0], [0.5, 0.5]])
    o = plain.constant_decay_recurrence(np.ones((2, 1, 1)), np.ones((2, 1, 1)), np.array([[[4.0]], [[6.0]]]), [0.5])
    assert np.allclose(o[:, 0, 0], [4.0, 8.0])
    assert np.allclose(plain.norm_one_plus([[3.0, 4.0]], [0.0, 1.0], 0.0), np.array([[3.0, 8.0]]) / np.sqrt(12.5))
    w = {"m.up": np.array([[1.0], [-1.0]]), "m.down": np.array([[1.0, 10.0]])}
    assert np.allclose(plain.dense_mlp(np.array([[2.0], [-3.0]]), w, "m."), [[4.0], [90.0]])
    assert plain.run_order(CFG) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]


def test_plain_query_norm_spans_all_heads():
    """One head's projection scaled up shrinks the other heads' normed queries: the norm is not per head."""
    cfg = plain.make_config([A(heads=2, kv_heads=1, dim=8, vdim=4, rot=4, mlp=None)], vocab=30, width=24)
    w = plain.random_weights(cfg, 2)
    other = {k: v.copy() for k, v in w.items()}
    other["l0.mix.q"][8:] *= 50.0
    h = np.random.default_rng(1).standard_normal((9, 24))
    w["l0.mix.o"][:, 4:] = 0.0
    other["l0.mix.o"][:, 4:] = 0.0          # the first head's output alone
    a, b = (plain.attention_mixer(h, x, "l0.mix.", cfg["layers"][0]["mixer"], 1e-6) for x in (w, other))
    assert np.abs(a - b)[1:].max() > 1e-2
