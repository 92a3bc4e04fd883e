"""Vonulorn without a GPU: the configuration (registry, round trip, rules reported by name), its layout (parts, tensor names, state),
a random folder that the plain implementation reads, and the plain mechanisms against hand-made cases."""
import copy
import json
import os

import numpy as np
import pytest
import torch

from plain import vonulorn_plain as VP

DENSE = {"kind": "dense", "ff": 20}
DELTA = {"type": "delta", "mlp": DENSE, "mixer": {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 14, "conv": 2}}
ATT = {"type": "attention", "mlp": None,
       "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 9, "scale": 0.35, "diff": 0.6, "softcap": 11.0,
                 "q_temp": {"coef": 0.2, "every": 5.0}}}
LAT = {"type": "latent_attention", "mlp": DENSE,
       "mixer": {"heads": 3, "dim": 6, "rot_dim": 4, "vdim": 10, "q_rank": 14, "kv_rank": 9, "scale": 0.4, "rot": {"base": 300.0, "dims": 4}}}
RAW = dict(architecture="Vonulorn", vocab=90, width=24, norm={"eps": 1e-5}, residual_mult=0.7, initializer_range=0.08,
           layers=[ATT, DELTA, LAT])


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
    from quicknn_b200.config import VONULORN, VonulornConfig, find_architecture
    assert find_architecture({"architecture": "Vonulorn"}) is VONULORN
    cfg = VonulornConfig.from_dict(RAW)
    assert VonulornConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict() == RAW
    spec = VONULORN.build_spec(cfg)
    assert not spec.head.tied and spec.head.softcap is None and spec.embedding.scale == 1.0
    for layer in spec.layers:
        assert layer.block.kind == "prenorm" and layer.block.get("residual_mult") == 0.7
        assert all(not n.get("unit_offset") and n.get("eps") == 1e-5 for n in layer.norms.values())
    att, delta, lat = (l.mixer for l in spec.layers)
    assert att.kind == "differential_attention" and att.get("diff") == 0.6 and att.get("softcap") == 11.0 and att.get("eps") == 1e-5
    assert att.get("query_temperature") == {"coef": 0.2, "every": 5.0} and att.get("window") is None and att.get("scale") == 0.35
    assert delta.kind == "delta_rule" and delta.get("conv") == 2 and delta.get("n_kv_heads") == 3 and delta.get("eps") == 1e-5
    assert lat.get("sink") and lat.get("gate") == "none" and lat.get("position").get("layout") == "interleaved"
    assert lat.get("position").get("theta") == 300.0 and lat.get("position").get("rotary_dim") == 4
    assert spec.layers[0].feed_forward is None and spec.layers[1].feed_forward.get("activation") == "gelu_tanh"
    bare = VonulornConfig.from_dict(changed(layers__0__mixer__q_temp=KeyError, layers__0__mixer__softcap=KeyError))
    assert bare.layers[0].mixer.softcap is None and bare.layers[0].mixer.temp_coef is None
    assert VonulornConfig.from_dict(bare.to_dict()) == bare


def test_layout_and_tensor_names():
    from quicknn_b200.config import VONULORN, VonulornConfig
    from quicknn_b200.parts import expected_tensors
    spec = VONULORN.build_spec(VonulornConfig.from_dict(RAW))
    shapes = {n: s for n, (s, _) in expected_tensors(spec).items()}
    assert shapes["embed"] == (90, 24) and shapes["head"] == (90, 24) and shapes["final.norm"] == (24,)
    assert shapes["l0.mix.q"] == (48, 24) and shapes["l0.mix.k"] == (24, 24) and shapes["l0.mix.v"] == (18, 24)
    assert shapes["l0.mix.o"] == (24, 36) and all(shapes[f"l0.mix.{n}"] == (6,) for n in ("lq1", "lk1", "lq2", "lk2"))
    assert shapes["l1.mix.q"] == (30, 24) and shapes["l1.mix.k.conv"] == (30, 2) and shapes["l1.mix.v.conv"] == (84, 2)
    assert shapes["l1.mix.b"] == (6, 24) and shapes["l1.mix.A_log"] == (6,) and shapes["l1.mix.norm"] == (14,)
    assert shapes["l1.mix.g"] == (84, 24) and shapes["l1.mix.o"] == (24, 84) and shapes["l1.mlp.down"] == (24, 20)
    assert shapes["l2.mix.uq"] == (30, 14) and shapes["l2.mix.dkv"] == (13, 24) and shapes["l2.mix.sink"] == (3,)
    assert "l2.mix.g" not in shapes and "l0.norm2" not in shapes and spec.optional_tensors == ("l0.norm2",)


@pytest.mark.parametrize("paths,word", [
    ({"width": 0}, "width"), ({"norm__eps": 0.0}, "norm.eps"), ({"residual_mult": float("nan")}, "residual_mult"),
    ({"residual_mult": KeyError}, "residual_mult"), ({"layers": []}, "layers"), ({"layers__0__type": "gla"}, "layer type"),
    ({"layers__1__mlp__kind": "moe"}, "mlp.kind"), ({"layers__1__mlp__ff": 0}, "mlp.ff"), ({"layers__1__mixer__kv_heads": 4}, "kv_heads"),
    ({"layers__1__mixer__conv": 0}, "conv"), ({"layers__1__mixer__dim": 257}, "dim"), ({"layers__1__mixer__vdim": KeyError}, "layers"),
    ({"layers__0__mixer__kv_heads": 3}, "kv_heads"), ({"layers__0__mixer__softcap": 0.0}, "softcap"),
    ({"layers__0__mixer__q_temp__every": 0}, "q_temp.every"), ({"layers__0__mixer__diff": float("inf")}, "diff"),
    ({"layers__2__mixer__rot__dims": 2}, "rot.dims"), ({"layers__2__mixer__rot__base": 0.0}, "rot.base"), ({"norm": 3}, "norm")])
def test_every_broken_rule_is_named(paths, word):
    from quicknn_b200.config import ConfigError, VonulornConfig
    with pytest.raises(ConfigError) as e:
        VonulornConfig.from_dict(changed(**paths))
    assert word in str(e.value)


def test_a_random_folder_loads(tmp_path):
    from quicknn_b200.config import VONULORN, VonulornConfig, load_config
    from quicknn_b200.weights import write_model_folder
    cfg = VonulornConfig.from_dict(RAW)
    d = write_model_folder(str(tmp_path / "m"), VONULORN, cfg, 5, torch.bfloat16, 0.05)
    arch, back = load_config(d)
    assert arch is VONULORN and back == cfg
    plain = VP.PlainVonulorn(d)
    logits = plain.logits([1, 2, 3, 4, 5, 6, 7])
    assert logits.shape == (7, 90) and np.isfinite(logits).all()
    assert plain.layers([1, 2, 3]).shape == (3, 3, 24)
    assert np.allclose(plain.logits([1, 2, 3])[2], logits[2])             # no row sees a later one


# ---- the plain mechanisms against other ways of writing them ------------------------------------------------------------

def test_the_delta_rule_is_a_product_of_transitions():
    """S_t = g_t (I - beta_t k_t k_t^T) S_(t-1) + beta_t k_t v_t^T."""
    rng = np.random.default_rng(0)
    n, D, V = 9, 5, 4
    q, k, v = rng.normal(size=(n, D)), VP.unit_vectors(rng.normal(size=(n, D))), rng.normal(size=(n, V))
    beta, g = rng.uniform(0.1, 0.9, n), rng.uniform(0.3, 1.0, n)
    out, S = VP.delta_rule(q, k, v, beta, g)
    R = np.zeros((D, V))
    for t in range(n):
        R = g[t] * (np.eye(D) - beta[t] * np.outer(k[t], k[t])) @ R + beta[t] * np.outer(k[t], v[t])
        assert np.allclose(out[t], R.T @ q[t])
    assert np.allclose(S, R)
    a, S1 = VP.delta_rule(q[:4], k[:4], v[:4], beta[:4], g[:4])
    b, S2 = VP.delta_rule(q[4:], k[4:], v[4:], beta[4:], g[4:], S1)
    assert np.allclose(np.concatenate([a, b]), out) and np.allclose(S2, S)
    # a full step writes exactly the value at its key, whatever was there
    one = np.ones(n)
    out, S = VP.delta_rule(k, k, v, one, one)
    assert np.allclose(out, v)


def test_the_chunked_form_of_the_delta_rule():
    """(I + L) U = diag(beta) (V - P K S) for a chunk of rows, what the kernels compute."""
    rng = np.random.default_rng(1)
    n, D, V = 16, 6, 3
    q, k, v = rng.normal(size=(n, D)), VP.unit_vectors(rng.normal(size=(n, D))), rng.normal(size=(n, V))
    beta, g, S0 = rng.uniform(0.1, 1.0, n), rng.uniform(0.2, 1.0, n), rng.normal(size=(D, V))
    P = np.cumprod(g)
    Dm = np.array([[np.prod(g[j + 1:t + 1]) if j <= t else 0.0 for j in range(n)] for t in range(n)])
    L = np.tril(beta[:, None] * Dm * (k @ k.T), -1)
    U = np.linalg.solve(np.eye(n) + L, beta[:, None] * (v - P[:, None] * (k @ S0)))
    O = P[:, None] * (q @ S0) + np.tril(Dm * (q @ k.T)) @ U
    out, S = VP.delta_rule(q, k, v, beta, g, S0)
    assert np.allclose(O, out) and np.allclose(P[-1] * S0 + (Dm[-1][:, None] * k).T @ U, S)


def test_convolutions_and_unit_vectors():
    x = np.arange(1.0, 6.0)[:, None]
    w = np.array([[100.0, 10.0, 1.0]])                        # the last number meets the row itself
    assert VP.causal_conv(x, w)[:, 0].tolist() == [1, 12, 123, 234, 345]
    assert np.allclose(VP.unit_vectors(np.array([[3.0, 4.0], [0.0, 0.0]])), [[0.6, 0.8], [0, 0]], atol=1e-6)
    assert np.allclose(VP.unit_vectors(np.array([[1e-3, 0.0]])), [[1e-3 / np.sqrt(2e-6), 0.0]])


def test_query_temperature_and_the_difference_of_maps():
    t = VP.query_temperature(9, {"coef": 0.5, "every": 4})
    assert np.allclose(t, 1 + 0.5 * np.log([1, 1, 1, 2, 2, 2, 2, 3, 3]))     # the step comes at position every - 1
    assert np.allclose(VP.query_temperature(3, None), 1.0)
    w = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.0]), "lq2": np.zeros(2), "lk2": np.ones(2)}
    assert np.isclose(VP.differential_lambda(w, "", 0.3), np.exp(0.5) - 1.0 + 0.3)
    q = k = np.zeros((3, 2))
    assert np.allclose(VP.softmax_map(q, k, 1.0, None), [[1, 0, 0], [0.5, 0.5, 0], [1 / 3] * 3])
    big = np.full((2, 1), 30.0)
    assert np.allclose(VP.softmax_map(big, np.array([[1.0], [2.0]]), 1.0, 2.0)[1], [0.5, 0.5], atol=1e-6)    # both at the cap


def test_sinks_and_the_rotation_of_neighbours():
    p = VP.softmax_rows(np.zeros((3, 3)), VP.causal(3), 0.0)
    assert np.allclose(p[0], [0.5, 0, 0]) and np.allclose(p[2], [0.25] * 3)
    assert np.allclose(VP.softmax_rows(np.full((1, 1), 900.0), VP.causal(1), 900.0), 0.5)
    x = np.zeros((3, 1, 6))
    x[:, 0, 0], x[:, 0, 5] = 1.0, 3.0
    y = VP.rotate_neighbours(x, 100.0, 4)                     # pairs (0, 1) and (2, 3); columns 4 and 5 pass
    assert np.allclose(y[:, 0, 0], np.cos([0, 1, 2])) and np.allclose(y[:, 0, 1], np.sin([0, 1, 2])) and np.allclose(y[:, 0, 5], 3.0)
    x[:, 0, :] = [0, 0, 0, 1, 0, 0]
    assert np.allclose(VP.rotate_neighbours(x, 100.0, 4)[2, 0, [2, 3]], [-np.sin(0.2), np.cos(0.2)])


def test_the_command_line_writes_and_describes_a_random_model(tmp_path, capsys):
    from quicknn_b200.cli import main
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(RAW))
    out = tmp_path / "model"
    assert main(["random", "--config", str(cfg), "--seed", "3", "--out", str(out)]) == 0
    capsys.readouterr()
    assert main(["info", "--model", str(out)]) == 0
    info = json.loads(capsys.readouterr().out)
    assert info["architecture"] == "Vonulorn" and info["layers"] == 3 and os.path.exists(out / "model.safetensors")
