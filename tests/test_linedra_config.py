"""Linedra without a GPU: the configuration (registry, round trip, rules reported by name), its layout (parts, tensor names, states
of blocks and mixers), a random folder that the plain implementation reads, and the plain mechanisms against hand-made cases."""
import copy
import json
import os

import numpy as np
import pytest
import torch

from plain import linedra_plain as LP

MOE = {"kind": "moe", "expert": {"ff": 12, "limit": 0.8}, "router": {"experts": 5, "top": 2}}
LEFT = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.3, "mask": {"size": 5}}
PAR = {"type": "parallel", "mlp": MOE, "mixer": {"left": LEFT, "right": {"width": 30, "blocks": 3, "conv": 2},
                                                 "left_scale": 0.7, "right_scale": 1.4}}
LAT = {"type": "latent_attention", "mlp": None,
       "mixer": {"heads": 3, "dim": 6, "rot_dim": 4, "vdim": 10, "q_rank": 14, "kv_rank": 9, "scale": 0.4, "rot": {"base": 300.0, "dims": 4}}}
RAW = dict(architecture="Linedra", vocab=90, width=24, embedding={"scale": 2.0}, norm={"eps": 1e-5}, canon={"taps": 3},
           residual_mult=0.6, logit_softcap=12.0, initializer_range=0.08, layers=[PAR, LAT, dict(PAR, mlp=None)])


def changed(**paths):
    """RAW with values at dotted paths replaced (double underscores for dots, numbers for list places)."""
    raw = copy.deepcopy(RAW)
    for path, value in paths.items():
        at = raw
        *way, last = path.split("__")
        for k in way:
            at = at[int(k)] if isinstance(at, list) else at[k]
        if value is KeyError:
            del at[last]
        else:
            at[last] = value
    return raw


def test_registry_round_trip_and_every_constant_from_the_file():
    from quicknn_b200.config import LINEDRA, LinedraConfig, find_architecture
    assert find_architecture({"architecture": "Linedra"}) is LINEDRA
    cfg = LinedraConfig.from_dict(RAW)
    assert LinedraConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict() == RAW
    spec = LINEDRA.build_spec(cfg)
    assert spec.depth_history and spec.head.tied and spec.head.softcap == 12.0 and spec.embedding.scale == 2.0
    for i, layer in enumerate(spec.layers):
        assert layer.block.kind == "sandwich" and layer.block.get("residual_mult") == 0.6
        assert layer.block.get("input_conv") == 3 and layer.block.get("depth_average") == i + 2
        assert all(n.get("unit_offset") and n.get("eps") == 1e-5 for n in layer.norms.values())
    left = spec.layers[0].mixer.get("branches")["left"]
    assert left.get("window") == 5 and left.get("sink") and left.get("head_gate") and left.get("v_head_dim") == 12
    assert left.get("distance_slopes") == (0.25, 0.0625, 0.015625, 0.00390625)
    assert spec.layers[0].mixer.get("scales") == {"left": 0.7, "right": 1.4}
    assert spec.layers[1].mixer.get("window") is None and spec.layers[1].mixer.get("gate") == "element"
    assert spec.layers[1].feed_forward is None and set(spec.layers[1].norms) == {"pre_mixer", "post_mixer"}
    no_mask = LinedraConfig.from_dict(changed(layers__0__mixer__left__mask=KeyError, logit_softcap=KeyError))
    assert no_mask.layers[0].left.window is None and no_mask.logit_softcap is None


def test_layout_and_tensor_names():
    from quicknn_b200.config import LINEDRA, LinedraConfig
    from quicknn_b200.parts import expected_tensors
    spec = LINEDRA.build_spec(LinedraConfig.from_dict(RAW))
    shapes = {n: s for n, (s, _) in expected_tensors(spec).items()}
    assert shapes["embed"] == (90, 24) and "head" not in shapes and shapes["final.norm"] == (24,)
    assert shapes["l0.mix.left.q"] == (32, 24) and shapes["l0.mix.left.v"] == (24, 24) and shapes["l0.mix.left.o"] == (24, 48)
    assert shapes["l0.mix.left.g"] == (4, 24) and shapes["l0.mix.left.sink"] == (4,)
    assert shapes["l0.mix.right.conv"] == (30, 2) and shapes["l0.mix.right.ra"] == (3, 10, 10) and shapes["l0.mix.right.ri.b"] == (3, 10)
    assert shapes["l0.mix.right.lam"] == (30,) and shapes["l0.mix.right.x.b"] == (30,) and shapes["l0.mix.right.o"] == (24, 30)
    assert shapes["l1.mix.uq"] == (30, 14) and shapes["l1.mix.dkv"] == (13, 24) and shapes["l1.mix.uk"] == (18, 9)
    assert shapes["l1.mix.uv"] == (30, 9) and shapes["l1.mix.g"] == (30, 24) and shapes["l1.mix.dkv.norm"] == (9,)
    assert shapes["l0.mlp.router"] == (5, 24) and shapes["l0.mlp.e4.down"] == (24, 12)
    assert [shapes[f"l{i}.dwa"] for i in range(3)] == [(2,), (3,), (4,)] and shapes["l2.canon1"] == (24, 3)
    assert "l1.norm2" not in shapes and set(spec.optional_tensors) == {"l1.norm2", "l1.norm2b", "l2.norm2", "l2.norm2b"}


@pytest.mark.parametrize("paths,word", [
    ({"width": 0}, "width"), ({"norm__eps": 0.0}, "norm.eps"), ({"canon__taps": 0}, "canon.taps"), ({"logit_softcap": -1.0}, "logit_softcap"),
    ({"residual_mult": float("inf")}, "residual_mult"), ({"residual_mult": KeyError}, "residual_mult"), ({"layers": []}, "layers"),
    ({"layers__0__type": "hgrn2"}, "layer type"), ({"layers__0__mlp__kind": "dense"}, "mlp.kind"),
    ({"layers__0__mlp__router__top": 6}, "router.top"), ({"layers__0__mlp__expert__limit": 0.0}, "limit"),
    ({"layers__0__mixer__left__kv_heads": 3}, "kv_heads"), ({"layers__0__mixer__left__mask__size": 0}, "mask.size"),
    ({"layers__0__mixer__right__blocks": 4}, "blocks"), ({"layers__0__mixer__right__conv": 0}, "conv"),
    ({"layers__1__mixer__rot__dims": 2}, "rot.dims"), ({"layers__1__mixer__rot__base": 0.0}, "rot.base"),
    ({"layers__1__mixer__kv_rank": 0}, "kv_rank"), ({"embedding": 3}, "embedding")])
def test_every_broken_rule_is_named(paths, word):
    from quicknn_b200.config import ConfigError, LinedraConfig
    with pytest.raises(ConfigError) as e:
        LinedraConfig.from_dict(changed(**paths))
    assert word in str(e.value)


def test_a_random_folder_loads_and_its_averages_are_averages(tmp_path):
    from quicknn_b200.config import LINEDRA, LinedraConfig, load_config
    from quicknn_b200.weights import write_model_folder
    cfg = LinedraConfig.from_dict(RAW)
    d = write_model_folder(str(tmp_path / "m"), LINEDRA, cfg, 5, torch.bfloat16, 0.05)
    arch, back = load_config(d)
    assert arch is LINEDRA and back == cfg
    plain = LP.PlainLinedra(d)
    for i in range(3):
        assert abs(plain.w[f"l{i}.dwa"].mean() - 1.0 / (i + 2)) < 0.1
    logits = plain.logits([1, 2, 3, 4, 5, 6, 7])
    assert logits.shape == (7, 90) and np.isfinite(logits).all() and np.abs(logits).max() <= 12.0
    assert plain.layers([1, 2, 3]).shape == (3, 3, 24)


def test_states_of_a_block_live_beside_its_mixers():
    from quicknn_b200.cache import KVCache
    from quicknn_b200.parts import CacheNeed, StateNeed
    c = KVCache([CacheNeed(1, 8, None), None, None], [None, StateNeed((3, 2)), None], 128, 2, 128, torch.float32, "cpu",
                [StateNeed((2, 4)), StateNeed((5,)), StateNeed((1,), "compute")])
    assert c.line(0).state is None and c.line(0).block_state.shape == (2, 2, 4) and c.line(0).k is not None
    assert c.line(1).state.shape == (2, 3, 2) and c.line(1).block_state.shape == (2, 5)
    assert c.line(2).state is None and c.line(2).k is None and c.line(2).block_state.dtype == torch.float32
    s = c.allocate()
    for i in range(3):
        c.line(i).block_state[s] = 7.0
    c.extend([(s, 10)])
    assert c.rewind_limit(s) == 10                            # a state describes the whole sequence
    c.free(s)
    again = c.allocate()
    assert again == s and all(float(c.line(i).block_state[s].abs().sum()) == 0.0 for i in range(3))
    assert c.bytes() > KVCache([CacheNeed(1, 8, None)], [None], 128, 2, 128, torch.float32, "cpu").bytes()


# ---- the plain mechanisms against other ways of writing them ------------------------------------------------------------

def test_convolutions_and_averages():
    x = np.arange(1.0, 6.0)[:, None]
    w = np.array([[100.0, 10.0, 1.0]])                        # the last number meets the row itself
    assert LP.causal_conv(x, w)[:, 0].tolist() == [1, 12, 123, 234, 345]
    assert np.allclose(LP.depth_average([x, 2 * x, 5 * x], np.array([1.0, -1.0, 0.5])), 1.5 * x)
    assert np.allclose(LP.norm_about_zero(np.array([[3.0, 4.0]]), np.array([0.0, 1.0]), 0.0), np.array([[3.0, 8.0]]) / np.sqrt(12.5))


def test_sinks_windows_and_slopes():
    see = LP.causal(4, 2)
    assert see.tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False], [False, False, True, True]]
    p = LP.softmax_with_sink(np.zeros((4, 4)), see, 0.0)
    assert np.allclose(p[0], [0.5, 0, 0, 0]) and np.allclose(p[3], [0, 0, 1 / 3, 1 / 3])
    assert np.allclose(LP.softmax_with_sink(np.zeros((4, 4)), see, -np.inf)[3], [0, 0, 0.5, 0.5])
    assert np.allclose(LP.softmax_with_sink(np.full((1, 1), 900.0), np.ones((1, 1), bool), 900.0), 0.5)
    assert np.allclose(LP.distance_slopes(8), [2.0 ** -(h + 1) for h in range(8)])


def test_the_rotation_turns_pairs_half_a_width_apart():
    x = np.zeros((3, 1, 6))
    x[:, 0, 0], x[:, 0, 5] = 1.0, 3.0
    y = LP.rotate_half(x, 100.0, 4)                           # pairs (0, 2) and (1, 3); columns 4 and 5 pass
    assert np.allclose(y[:, 0, 0], np.cos([0, 1, 2])) and np.allclose(y[:, 0, 2], np.sin([0, 1, 2])) and np.allclose(y[:, 0, 5], 3.0)
    x[:, 0, :] = [0, 1, 0, 0, 0, 0]
    assert np.allclose(LP.rotate_half(x, 100.0, 4)[2, 0, [1, 3]], [np.cos(0.2), np.sin(0.2)])


def test_the_recurrence_is_a_sum_over_earlier_rows():
    rng = np.random.default_rng(0)
    a, b = rng.uniform(0.2, 1.0, (7, 3)), rng.normal(size=(7, 3))
    S = LP.linear_recurrence(a, b)
    for t in range(7):
        assert np.allclose(S[t], sum(np.prod(a[s + 1:t + 1], axis=0) * b[s] for s in range(t + 1)))
    u = rng.normal(size=(2, 4))
    w = rng.normal(size=(2, 2, 2))
    bias = rng.normal(size=(2, 2))
    assert np.allclose(LP.block_product(u, w, bias)[:, 2:], u[:, 2:] @ w[1].T + bias[1])
    z = {"ra": np.zeros((2, 2, 2)), "ra.b": np.zeros((2, 2)), "ri": np.zeros((2, 2, 2)), "ri.b": np.zeros((2, 2)), "lam": np.zeros(4)}
    at, term = LP.recurrence_inputs(u, z, "")
    assert np.allclose(at, np.exp(-4.0 * np.log(2.0))) and np.allclose(term, np.sqrt(1 - at ** 2) * 0.5 * u)


def test_routing_weighs_by_the_chosen_logits_alone():
    h = np.array([[1.0, 0.0]])
    w = {"router": np.array([[1.0, 0], [3.0, 0], [2.0, 0], [-9.0, 0]])}
    chosen, weights = LP.route(h, w, "", 2)
    assert chosen.tolist() == [[1, 2]] and np.allclose(weights, [[np.e / (1 + np.e), 1 / (1 + np.e)]])
    one = {"e.gate": np.array([[5.0, 0]]), "e.up": np.array([[-7.0, 0]]), "e.down": np.eye(2)[:, :1]}
    assert np.allclose(LP.clamped_expert(h, one, "e.", 2.0), [[2.0 / (1 + np.exp(-3.404)) * -1.0, 0.0]])


def test_the_command_line_writes_and_describes_a_random_model(tmp_path, capsys):
    from quicknn_b200.cli import main
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(RAW))
    out = tmp_path / "model"
    assert main(["random", "--config", str(cfg), "--seed", "3", "--out", str(out)]) == 0
    capsys.readouterr()
    assert main(["info", "--model", str(out)]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Linedra" and info["layers"] == 3 and os.path.exists(out / "model.safetensors")
