"""Vonulorn on the GPU against the plain implementation (tests/plain/vonulorn_plain.py): the small kernels (convolutions with silu and
unit vectors, rows packed for several maps, the difference of maps); the delta rule's scan and its decode step; the three mixers
alone over caches of their own (prompts, single tokens, portions, slots handed out again, keys and associations that stand out
hundreds of positions back); then whole models through bin/trace_run under every cutting, in portions down to two tokens, through
the entry point's generation loop, the command line, and configurations drawn at random.  The configurations are small and differ
from one another in every size and constant."""
import json
import os

import numpy as np
import pytest
import torch

from plain import vonulorn_plain as VP
from test_gpu_fuposun import part_step
from test_gpu_linedra import bf, dev, f64, host, i32, rnd, walk_a_mixer
from test_gpu_replay import Replay, run_all_cuttings

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BOTH = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module", autouse=True)
def _need_gpu():
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")


def near(got, ref, dtype, float32=1e-4):
    """How whole models are compared.  float32: the largest difference, 1e-4 of the largest logit: the sharp check, since a wrong
    mask, key, filter, sink, temperature or state moves these models' logits by 1e-2 and more.  bfloat16: a row by the root mean
    square of its difference (mean taken off) against that of the logits, at most a tenth; one row in thirty may lie beyond (a
    difference of two maps that nearly cancel is divided by its own size)."""
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    if dtype == "float32":
        tol = float32 * max(1.0, float(np.abs(ref).max()))
        err = float(np.abs(got - ref).max()) if got.size else 0.0
        return err <= tol, err, tol
    if not got.size:
        return True, 0.0, 0.1
    d = got - ref
    d = d - d.mean(axis=-1, keepdims=True)
    r = ref - ref.mean(axis=-1, keepdims=True)
    e = np.sqrt((d * d).mean(axis=-1)) / np.sqrt((r * r).mean())
    over, allowed = int((e > 0.1).sum()), max(1, len(e) // 30)
    return over <= allowed, float(np.sort(e)[-1 - min(over, allowed, len(e) - 1)]), 0.1


@pytest.fixture
def whole_model_tolerance(monkeypatch):
    import test_gpu_replay
    monkeypatch.setattr(test_gpu_replay, "close", near)


# ---- configurations -------------------------------------------------------------------------------------

def _dense(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def _delta(heads, kv, dim, vdim, conv, ff):
    return {"type": "delta", "mlp": _dense(ff), "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def _att(heads, kv, dim, vdim, scale, diff, cap, temp, ff):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if cap is not None:
        m["softcap"] = cap
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mlp": _dense(ff), "mixer": m}


def _lat(heads, dim, rot, vdim, q_rank, kv_rank, scale, base, ff):
    return {"type": "latent_attention", "mlp": _dense(ff),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot}}}


def _model(vocab, width, eps, mult, std, layers):
    return dict(architecture="Vonulorn", vocab=vocab, width=width, norm={"eps": eps}, residual_mult=mult, initializer_range=std,
                layers=layers)


# A: attention first; values wider and narrower than keys; a temperature that steps every 7 positions; one key head for all; taps
#    of 2 and 5; layers without a feed-forward; a residual multiplier of 1
VON_A = _model(300, 64, 1e-6, 1.0, 0.08, [
    _att(4, 2, 16, 40, 0.35, 0.5, 9.0, (0.25, 7), 48),
    _delta(6, 2, 16, 24, 2, None),
    _lat(3, 16, 8, 24, 40, 24, 0.3, 1000.0, 40),
    _delta(2, 2, 32, 16, 5, 72)])
# B: sizes for the tensor-core kernels (both maps in 64 columns, latent rows of 64), four value heads on a key head, no softcap in
#    one layer and no temperature in the other
VON_B = _model(512, 128, 1e-5, 0.6, 0.06, [
    _delta(4, 1, 64, 64, 4, 96),
    _att(4, 1, 32, 64, 0.21, 0.2, None, (0.4, 33), 128),
    _lat(4, 32, 16, 32, 64, 48, 0.17, 30000.0, None),
    _att(2, 2, 32, 48, 0.18, 0.7, 25.0, None, 64),
    _delta(3, 3, 128, 32, 3, 64)])
# C: a width, head sizes, ranks and a vocabulary that are no multiple of 8; one tap (no past); one head; a large multiplier
VON_C = _model(301, 100, 1e-4, 1.3, 0.07, [
    _lat(1, 20, 6, 28, 30, 21, 0.25, 500.0, 60),
    _delta(5, 5, 12, 20, 1, 36),
    _att(3, 1, 10, 12, 0.3, -0.2, 4.0, (1.5, 64), None),
    _delta(1, 1, 20, 7, 3, 44),
    _att(1, 1, 21, 50, 0.25, 0.9, 50.0, (0.1, 1), 20)])
CONFIGS = {"A": (VON_A, 3), "B": (VON_B, 4), "C": (VON_C, 5)}
LENGTHS = [70, 33, 129, 45, 100, 64]
LENGTHS_B = [170, 33, 257, 45, 100, 64]


def stand_out(tensors, peaky):
    """What random draws would leave trivial: sinks of the size of the scores, decays from nearly none to nearly all, filters with
    sizeable numbers of both signs, a lambda far from its constant; ``peaky``: scores scaled up."""
    for k in list(tensors):
        t = tensors[k]
        if k.endswith(".sink"):
            tensors[k] = t * 8.0
        elif k.endswith(".A_log"):
            tensors[k] = torch.linspace(-3.0, 1.5, t.numel())
        elif k.endswith(".dt_bias"):
            tensors[k] = torch.linspace(0.5, -4.0, t.numel())
        elif k.endswith(".mix.a") or k.endswith(".mix.b"):
            tensors[k] = t * 4.0
        elif k.endswith(".conv"):
            tensors[k] = t * 0.5 * torch.cos(torch.arange(t.numel()).view(t.shape) * 1.3 + 0.4)
        elif k.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            tensors[k] = torch.full_like(t, {"lq1": 0.2, "lk1": 0.2, "lq2": 0.3, "lk2": -0.2}[k[-3:]])
        elif peaky and k.endswith((".mix.q", ".mix.uq")):
            tensors[k] = t * 4.0
    return tensors


def make_folder(base, name, storage, peaky):
    from quicknn_b200.config import VONULORN, VonulornConfig
    from quicknn_b200.weights import random_tensors, write_safetensors
    raw, seed = CONFIGS[name]
    cfg = VonulornConfig.from_dict(raw)
    d = os.path.join(str(base), f"von{name}_{storage}{'_peaky' if peaky else ''}")
    os.makedirs(d, exist_ok=True)
    tensors = stand_out(dict(random_tensors(VONULORN, cfg, seed, torch.float32, 0.2)), peaky)
    dt = torch.float32 if storage == "float32" else torch.bfloat16
    with open(os.path.join(d, "config.json"), "w") as fh:
        json.dump(cfg.to_dict(), fh)
    write_safetensors(os.path.join(d, "model.safetensors"), {k: v.to(dt).contiguous() for k, v in tensors.items()})
    return d


@pytest.fixture(scope="module")
def von(tmp_path_factory):
    base = tmp_path_factory.mktemp("vonulorn")
    made = {}

    def get(name, storage="float32", peaky=False):
        key = (name, storage, peaky)
        if key not in made:
            folder = make_folder(base, name, storage, peaky)
            made[key] = (folder, VP.PlainVonulorn(folder))
        return made[key]
    return get


def prompts(name, lengths, seed=0):
    rng = np.random.default_rng(100 + seed)
    return [rng.integers(1, CONFIGS[name][0]["vocab"], n).tolist() for n in lengths]


# ---- the small kernels ------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("heads,size,C,taps", [(4, 16, 112, 4), (2, 64, 160, 3), (3, 24, 96, 2), (2, 8, 24, 4), (1, 256, 264, 3),
                                               (5, 12, 84, 4), (2, 32, 64, 1), (2, 128, 320, 6), (6, 7, 45, 2)])
def test_convolutions_with_silu_and_unit_vectors(dtype, heads, size, C, taps):
    """Prompts of unequal lengths, a portion, single tokens, a row of no sequence; heads of one to thirty-two eights inside the
    convolution's kernel, others behind it."""
    from quicknn_b200.kernels import ops
    w = bf(rnd((C, taps), 1, 0.6))
    lens, extra = [37, 1, 20], [11, 2, 9]
    xs = [bf(rnd((n + m + 3, C + 5), 10 + i)) for i, (n, m) in enumerate(zip(lens, extra))]
    ref = [VP.silu(VP.causal_conv(x[:, 3:3 + C].astype(np.float64), w.astype(np.float64))) for x in xs]
    state = torch.full((4, taps * C + 2), 5.0, device=DEV)               # what lies before a start is never read
    wd = dev(w, dtype)
    tol = 3e-6 if dtype == torch.float32 else 1e-2

    def check(out, inv, want):
        y = host(out)
        assert np.abs(y - want).max() < tol * max(1.0, np.abs(want).max())
        h = y[:, :heads * size].reshape(len(y), heads, size)             # 1 / length of the rows as they are stored
        assert np.allclose(host(inv), 1.0 / np.sqrt((h * h).sum(-1) + 1e-6), rtol=2e-6)

    def run(ns, starts, which, longest):
        rows = np.concatenate([xs[i][s:s + n] for i, s, n in zip(which, starts, ns)])
        pos = np.concatenate([np.arange(s, s + n) for s, n in zip(starts, ns)])
        first = np.cumsum([0] + list(ns[:-1]))
        decode = longest == 0
        out, inv = ops.causal_conv(dev(rows, dtype), wd, state, None if decode else i32(first), None if decode else i32(ns),
                                   i32(pos), i32([s + 1 for s in which]), len(ns), max(1, longest), col0=3, activation="silu",
                                   unit_heads=(heads, size, 1e-6))
        check(out, inv, np.concatenate([ref[i][s:s + n] for i, s, n in zip(which, starts, ns)]))
    run(lens, [0, 0, 0], [0, 1, 2], max(lens))
    run(extra, lens, [0, 1, 2], max(extra))
    for t in range(3):
        run([1, 1, 1], [n + m + t for n, m in zip(lens, extra)], [0, 1, 2], 0)
    out, inv = ops.causal_conv(dev(xs[0][:2], dtype), wd, state, None, None, i32([5, 0]), i32([-1, 0]), 2, col0=3, activation="silu",
                               unit_heads=(heads, size, 1e-6))
    assert float(out[0].abs().max()) == 0.0 and float(inv[0].abs().max()) == 0.0
    check(out[1:], inv[1:], VP.silu(VP.causal_conv(xs[0][1:2, 3:3 + C].astype(np.float64), w.astype(np.float64))))


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("nq,nk,maps,dim,vdim,hd", [(4, 2, 2, 16, 40, 64), (2, 2, 2, 32, 64, 64), (3, 1, 2, 10, 12, 24), (2, 1, 1, 24, 16, 24),
                                                    (1, 1, 3, 8, 32, 32), (6, 3, 2, 64, 128, 128)])
def test_rows_packed_for_several_maps(dtype, nq, nk, maps, dim, vdim, hd):
    from quicknn_b200.cache import KVCache
    from quicknn_b200.kernels import ops
    from quicknn_b200.parts import CacheNeed
    coef, every = 0.3, 6.0
    cache = KVCache([CacheNeed(nk, hd, None)], [None], 512, 3, 256, dtype, DEV)
    slots = [cache.allocate(), cache.allocate()]
    cache.extend([(slots[0], 70), (slots[1], 9)])
    cache.sync()
    line = cache.line(0)
    T = 79
    src = bf(rnd((T, (nq + nk) * maps * dim + nk * vdim), 4))
    pos = np.concatenate([np.arange(70), np.arange(9)])
    slot = np.concatenate([np.full(70, slots[0]), np.full(9, slots[1])])
    slot[75] = -1                                                     # a row of no sequence writes nothing
    got = host(ops.map_prep(dev(src, dtype), nq, nk, maps, dim, vdim, hd, i32(pos), i32(slot), line, True, True, coef, every))
    temp = 1 + coef * np.log(np.floor((pos + 1) / every) + 1)
    want = np.zeros((T, nq * maps + 2 * nk, hd))
    for h in range(nq):
        for m in range(maps):
            u = h * maps + m
            want[:, u, m * dim:(m + 1) * dim] = src[:, u * dim:(u + 1) * dim] * temp[:, None]
    k0, v0 = nq * maps * dim, (nq + nk) * maps * dim
    for g in range(nk):
        want[:, nq * maps + g, :maps * dim] = src[:, k0 + g * maps * dim:k0 + (g + 1) * maps * dim]
        want[:, nq * maps + nk + g, :vdim] = src[:, v0 + g * vdim:v0 + (g + 1) * vdim]
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    assert np.allclose(got, want.reshape(T, -1), rtol=tol, atol=tol)
    table = line.page_table.cpu().numpy()
    for t in (0, 1, 63, 64, 69, 70, 74, 78):
        page, off = table[slot[t], pos[t] // line.page_size], pos[t] % line.page_size
        assert np.allclose(host(line.k[page, :, off]), want[t, nq * maps:nq * maps + nk], rtol=tol, atol=tol)
        assert np.allclose(host(line.v[page, :, off]), want[t, nq * maps + nk:], rtol=tol, atol=tol)
    alone = host(ops.map_prep(dev(src, dtype), nq, nk, maps, dim, vdim, hd, i32(pos), i32(slot), line, False, False, 0.0, 1.0))
    assert np.allclose(alone, (want[:, :nq * maps] / temp[:, None, None]).reshape(T, -1), rtol=tol, atol=tol)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,vdim,hd", [(4, 64, 64), (3, 40, 64), (1, 12, 24), (5, 256, 256), (2, 300, 304), (7, 7, 8)])
def test_the_difference_of_two_maps(dtype, H, vdim, hd):
    from quicknn_b200.kernels import ops
    a = bf(rnd((33, H * 2 * hd), 2))
    a[5] = 0.0
    got = host(ops.map_difference(dev(a, dtype), H, vdim, 0.37, 1e-5, 0.8))
    x = a.reshape(33, H, 2, hd)[..., :vdim].astype(np.float64)
    want = VP.rms_unit(x[:, :, 0] - 0.37 * x[:, :, 1], 1e-5) * 0.8
    tol = 3e-6 if dtype == torch.float32 else 1e-2
    assert np.allclose(got, want.reshape(33, -1), rtol=tol, atol=tol)


# ---- the delta rule ---------------------------------------------------------------------------------------------

def scan_inputs(T, H, G, D, V, seed=0, repeat=False):
    """Raw rows (before the unit vectors), logits and constants; ``repeat``: few distinct keys, so that writes meet one another."""
    q, k, v = rnd((T, G, D), seed + 1), rnd((T, G, D), seed + 2), rnd((T, H, V), seed + 3)
    if repeat:
        k = k[np.random.default_rng(seed).integers(0, min(5, T), T)] + 0.05 * k
    pre = rnd((T, 2 * H), seed + 4, 2.0)
    rate, bias = np.exp(np.linspace(-4, 1.5, H)).astype(np.float32), np.linspace(-5, 0.5, H).astype(np.float32)[::-1].copy()
    if H == 1:
        rate, bias = np.float32([0.05]), np.float32([-3.0])
    return [bf(q), bf(k), bf(v)], pre, rate, bias


def plain_scan(qkv, pre, rate, bias, S0=None):
    q, k, v = (a.astype(np.float64) for a in qkv)
    H, per = v.shape[1], v.shape[1] // q.shape[1]
    q, k = VP.unit_vectors(q) / np.sqrt(q.shape[-1]), VP.unit_vectors(k)
    beta = VP.sigmoid(pre[:, :H].astype(np.float64))
    g = np.exp(-rate.astype(np.float64) * VP.softplus(pre[:, H:].astype(np.float64) + bias))
    outs = [VP.delta_rule(q[:, h // per], k[:, h // per], v[:, h], beta[:, h], g[:, h], None if S0 is None else S0[h]) for h in range(H)]
    return np.stack([o for o, _ in outs], 1), np.stack([s for _, s in outs])


def run_scan(qkvs, pres, rate, bias, state, slots, dtype, col0):
    from quicknn_b200.kernels import ops
    ns = [len(p) for p in pres]
    G, D = qkvs[0][0].shape[1:]
    H, V = qkvs[0][2].shape[1:]
    rows = np.concatenate([np.concatenate([a.reshape(len(a), -1) for a in qkv], 1) for qkv in qkvs])
    heads = rows[:, :2 * G * D].reshape(len(rows), 2 * G, D).astype(np.float64)
    inv = 1.0 / np.sqrt((heads ** 2).sum(-1) + 1e-6)
    return host(ops.delta_scan(dev(rows, dtype), dev(inv), dev(np.concatenate(pres)), dev(rate), dev(bias), D ** -0.5, state, col0,
                               i32(np.cumsum([0] + ns[:-1])), i32(ns), i32(slots), len(ns), max(ns), H, G, D, V)).reshape(-1, H, V)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,D,V", [(2, 2, 16, 16), (4, 2, 64, 32), (6, 1, 32, 40), (3, 3, 128, 64), (1, 1, 256, 24), (5, 5, 12, 20),
                                     (2, 1, 21, 7), (4, 4, 128, 128), (3, 1, 200, 33), (8, 2, 64, 128)])
@pytest.mark.parametrize("repeat", [False, True])
def test_the_delta_rules_scan_over_prompts_and_portions(dtype, H, G, D, V, repeat):
    """Unequal sequences (below, at and beyond chunks of 16), then portions from the state that they left; decays from none to all
    within a few rows; keys that write over one another."""
    lens, more = [100, 1, 33, 16, 47], [17, 2, 1, 31, 5]
    rng = np.random.default_rng(3)
    state = torch.zeros((7, 3 + H * D * V), device=DEV)
    data = [scan_inputs(n + m, H, G, D, V, seed=20 * i, repeat=repeat) for i, (n, m) in enumerate(zip(lens, more))]
    rate, bias = data[0][2], data[0][3]
    ref = [plain_scan(d[0], d[1], rate, bias) for d in data]
    slots = [5, 0, 3, 2, 6]
    state[4] = 7.0
    cut = lambda d, a, b: ([x[a:b] for x in d[0]], d[1][a:b])  # noqa: E731
    top = max(np.abs(r[0]).max() for r in ref)
    tol = 1e-5 * top
    first = [cut(d, 0, n) for d, n in zip(data, lens)]
    got = run_scan([f[0] for f in first], [f[1] for f in first], rate, bias, state, slots, dtype, 3)
    assert np.abs(got - np.concatenate([r[0][:n] for r, n in zip(ref, lens)])).max() < tol
    second = [cut(d, n, n + m) for d, n, m in zip(data, lens, more)]
    got = run_scan([f[0] for f in second], [f[1] for f in second], rate, bias, state, slots, dtype, 3)
    assert np.abs(got - np.concatenate([r[0][n:] for r, n in zip(ref, lens)])).max() < tol
    for r, s in zip(ref, slots):
        S = host(state[s, 3:]).reshape(H, D, V)
        assert np.abs(S - r[1]).max() < 1e-5 * max(1.0, np.abs(r[1]).max())
    assert float((state[4] - 7.0).abs().max()) == 0.0 and float(state[:, :3][[0, 2, 3]].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", BOTH)
def test_many_sequences_take_the_wide_blocks_and_rows_of_no_sequence_give_zeros(dtype):
    H, G, D, V, B = 6, 3, 64, 96, 12
    data = [scan_inputs(18 + 3 * i, H, G, D, V, seed=7 * i) for i in range(B)]
    rate, bias = data[0][2], data[0][3]
    ref = [plain_scan(d[0], d[1], rate, bias)[0] for d in data]
    state = torch.zeros((B, H * D * V), device=DEV)
    slots = list(range(B))[::-1]
    slots[4] = -1
    got = run_scan([d[0] for d in data], [d[1] for d in data], rate, bias, state, slots, dtype, 0)
    at = 0
    for i, r in enumerate(ref):
        want = np.zeros_like(r) if i == 4 else r
        assert np.abs(got[at:at + len(r)] - want).max() < 1e-5 * np.abs(r).max()
        at += len(r)
    assert float(state[B - 1 - 4].abs().max()) == 0.0


def delta_part(H, G, D, V, taps, dtype, W=48, seed=0, eps=1e-5):
    from quicknn_b200.parts import MIXERS, PartSpec
    mixer = MIXERS.get("delta_rule")(PartSpec("delta_rule", {
        "hidden_size": W, "n_heads": H, "n_kv_heads": G, "dim": D, "vdim": V, "conv": taps, "eps": eps}))
    w = {"q": rnd((G * D, W), seed + 1, 0.3), "k": rnd((G * D, W), seed + 2, 0.3), "v": rnd((H * V, W), seed + 3, 0.3),
         "q.conv": rnd((G * D, taps), seed + 4, 0.6), "k.conv": rnd((G * D, taps), seed + 5, 0.6), "v.conv": rnd((H * V, taps), seed + 6, 0.6),
         "b": rnd((H, W), seed + 7, 0.3), "a": rnd((H, W), seed + 8, 0.2), "A_log": np.linspace(-3, 1, H), "dt_bias": np.linspace(0.5, -4, H),
         "norm": rnd(V, seed + 9, 0.2) + 1.0, "g": rnd((H * V, W), seed + 10, 0.3), "o": rnd((W, H * V), seed + 11, 0.2)}
    w = {k: bf(v) for k, v in w.items()}
    names = {k: k.replace(".", "_") for k in w}
    names["g"] = "gate"
    mixer.load({names[k]: dev(v, dtype) for k, v in w.items()}, dtype, DEV)
    return mixer, w, {"heads": H, "kv_heads": G, "dim": D, "vdim": V}


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,D,V,taps", [(4, 2, 16, 24, 4), (2, 2, 64, 32, 2), (3, 1, 32, 130, 3), (5, 5, 12, 20, 1), (1, 1, 21, 7, 5),
                                          (2, 1, 128, 256, 4), (2, 2, 256, 64, 3), (1, 1, 8, 600, 2), (6, 3, 40, 12, 6)])
def test_the_delta_rule_alone_and_what_is_lost_or_left_out_would_show(dtype, H, G, D, V, taps):
    W = 48
    mixer, w, m = delta_part(H, G, D, V, taps, dtype)
    w64 = f64(w)
    plain = lambda x, w=w64: VP.delta(x, w, "", m, 1e-5)  # noqa: E731
    xs, ref, tol = walk_a_mixer(mixer, plain, dtype, W, lambda top: (4e-5 if dtype == torch.float32 else 5e-2) * top)
    if dtype == torch.float32:
        x = xs[0].astype(np.float64)
        assert np.abs(plain(x[60:]) - ref[0][60:]).max() > 20 * tol              # a state that starts anew
        for name, change in (("A_log", lambda t: t + 1.0), ("dt_bias", lambda t: t + 1.0), ("b", lambda t: t * 0.0), ("norm", lambda t: t * 0 + 1)):
            assert np.abs(plain(x, dict(w64, **{name: change(w64[name])})) - ref[0]).max() > 20 * tol, name
        if taps > 1:
            lost = dict(w64, **{t + ".conv": np.concatenate([w64[t + ".conv"][:, :1] * 0, w64[t + ".conv"][:, 1:]], 1) for t in "qkv"})
            assert np.abs(plain(x, lost) - ref[0]).max() > 20 * tol


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows", [1, 3, 8, 17, 40])
def test_decode_batches_of_the_delta_rule(dtype, rows):
    """Single tokens of many sequences, some rows of no sequence, against every sequence alone."""
    from quicknn_b200.cache import KVCache
    W = 72
    mixer, w, m = delta_part(4, 2, 32, 96, 4, dtype, W=W, seed=40)
    w64 = f64(w)
    cache = KVCache([None], [mixer.state_need()], 4096, rows, 64, dtype, DEV)
    slots = [cache.allocate() for _ in range(rows)]
    n, extra = 5, 6
    xs = [bf(rnd((n + extra, W), 200 + i)) for i in range(rows)]
    ref = [VP.delta(x.astype(np.float64), w64, "", m, 1e-5) for x in xs]
    tol = (4e-5 if dtype == torch.float32 else 5e-2) * max(np.abs(r).max() for r in ref)
    step = part_step([n] * rows, [0] * rows, slots, "prefill", dtype, cache, mixer)
    y = host(mixer.forward(dev(np.concatenate([x[:n] for x in xs]), dtype), step, cache.line(0)))
    assert np.abs(y - np.concatenate([r[:n] for r in ref])).max() < tol
    for t in range(n, n + extra):
        step = part_step([1] * rows, [t] * rows, slots, "decode", dtype, cache, mixer)
        idle = [] if rows < 8 else [2, rows - 1]                   # (their sequences stay where they are)
        for i in idle:
            step.slots[i] = -1
            step.tok_slot[i] = -1
        y = host(mixer.forward(dev(np.stack([x[t] for x in xs]), dtype), step, cache.line(0)))
        for i in range(rows):
            if i in idle:
                assert np.abs(y[i]).max() == 0.0
            else:
                assert np.abs(y[i] - ref[i][t]).max() < tol, (i, t)


@pytest.mark.parametrize("where", ["prefill", "decode"])
def test_an_association_hundreds_of_rows_back_is_found(where):
    """Keys of the rows between are orthogonal to the one that is asked for, decays are nearly 1: the value written at row 30 comes
    back at row 530, and a state lost or decayed a little more on the way would show."""
    H, G, D, V, n = 1, 1, 32, 32, 531
    (q, k, v), pre, rate, bias = scan_inputs(n, H, G, D, V, seed=9)
    k[:, 0, 0] = 0.0                                               # column 0 belongs to rows 30 and 530 alone
    q[:, 0, 0] = 0.0
    k[30, 0] = 0.0
    k[30, 0, 0] = q[530, 0, 0] = 4.0
    q[530, 0, 1:] = 0.0
    pre[30, 0], pre[530, 0] = 6.0, -6.0                            # written in full; hardly anything at the end
    pre[:, 1] = -4.0
    rate, bias = np.float32([0.02]), np.float32([-2.0])
    ref, S = plain_scan((q, k, v), pre, rate, bias)
    kept = np.abs(ref[530, 0] * np.sqrt(D) - v[30, 0]).max()
    assert kept < 0.1 * np.abs(v[30, 0]).max()                     # the plain answer is the value of row 30
    state = torch.zeros((1, H * D * V), device=DEV)
    if where == "prefill":
        got = run_scan([(q, k, v)], [pre], rate, bias, state, [0], torch.bfloat16, 0)
    else:
        got = run_scan([(q[:40], k[:40], v[:40])], [pre[:40]], rate, bias, state, [0], torch.bfloat16, 0)
        for t in range(40, n):                                     # single rows through the scan
            got = run_scan([(q[t:t + 1], k[t:t + 1], v[t:t + 1])], [pre[t:t + 1]], rate, bias, state, [0], torch.bfloat16, 0)
    assert np.abs(got[-1] - ref[-1]).max() < 1e-4 * np.abs(ref[-1]).max()      # (500 equal decays, each rounded to float32)


# ---- the attentions alone ------------------------------------------------------------------------------------------

def differential_part(H, G, D, V, scale, diff, cap, temp, dtype, W=48, seed=0, eps=1e-5):
    from quicknn_b200.parts import MIXERS, PartSpec
    mixer = MIXERS.get("differential_attention")(PartSpec("differential_attention", {
        "hidden_size": W, "n_heads": H, "n_kv_heads": G, "dim": D, "vdim": V, "scale": scale, "softcap": cap, "window": None,
        "diff": diff, "eps": eps, "query_temperature": None if temp is None else {"coef": temp[0], "every": temp[1]}}))
    w = {"q": rnd((H * 2 * D, W), seed + 1, 0.4), "k": rnd((G * 2 * D, W), seed + 2, 0.4), "v": rnd((G * V, W), seed + 3, 0.3),
         "lq1": rnd(D, seed + 4, 0.2), "lk1": rnd(D, seed + 5, 0.2) + 0.3 / np.sqrt(D), "lq2": rnd(D, seed + 6, 0.2),
         "lk2": rnd(D, seed + 7, 0.2), "o": rnd((W, H * V), seed + 8, 0.2)}
    w = {k: bf(v) for k, v in w.items()}
    mixer.load({k: dev(v, dtype) for k, v in w.items()}, dtype, DEV)
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale, "diff": diff}
    if cap is not None:
        m["softcap"] = cap
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return mixer, w, m


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,D,V,diff,cap,temp", [
    (4, 2, 16, 40, 0.5, 6.0, (0.3, 7)), (2, 2, 32, 64, 0.2, None, (0.5, 64)), (6, 1, 24, 16, 0.8, 20.0, None), (3, 3, 10, 12, -0.3, 3.0, (1.0, 33)),
    (1, 1, 64, 128, 0.6, 30.0, (0.2, 1)), (8, 4, 32, 48, 0.4, 8.0, (0.3, 50)), (2, 1, 128, 256, 0.35, 50.0, (0.1, 100)), (5, 5, 8, 300, 0.1, None, None),
    (2, 2, 150, 40, 0.3, 15.0, (0.4, 20))])
def test_differential_attention_alone_and_what_is_left_out_would_show(dtype, H, G, D, V, diff, cap, temp):
    W = 48
    mixer, w, m = differential_part(H, G, D, V, 1.5 / np.sqrt(D), diff, cap, temp, dtype)
    w64 = f64(w)
    plain = lambda x, m=m, w=w64: VP.differential_attention(x, w, "", m, 1e-5)  # noqa: E731
    xs, ref, tol = walk_a_mixer(mixer, plain, dtype, W, lambda top: (4e-5 if dtype == torch.float32 else 6e-2) * top)
    if dtype == torch.float32:
        x = xs[0].astype(np.float64)
        assert np.abs(plain(x, m, dict(w64, lq1=w64["lq1"] * 0)) - ref[0]).max() > 20 * tol
        assert np.abs(plain(x, dict(m, diff=diff + 0.1)) - ref[0]).max() > 20 * tol
        if cap is not None and cap < 20:
            assert np.abs(plain(x, dict(m, softcap=cap * 1.3)) - ref[0]).max() > 20 * tol
        if temp is not None and temp[1] > 1:                       # a step that comes one position late
            assert np.abs(plain(x, dict(m, q_temp={"coef": temp[0], "every": temp[1] + 1})) - ref[0]).max() > 20 * tol


def latent_part(H, D, R, V, QR, KR, scale, base, dtype, W=48, seed=0):
    from quicknn_b200.parts import MIXERS, PartSpec
    mixer = MIXERS.get("latent_attention")(PartSpec("latent_attention", {
        "hidden_size": W, "n_heads": H, "dim": D, "vdim": V, "q_rank": QR, "kv_rank": KR, "scale": scale, "window": None, "eps": 1e-5,
        "sink": True, "gate": "none", "position": PartSpec("rotary", {"head_dim": R, "theta": base, "rotary_dim": R, "layout": "interleaved"})}))
    w = {"dq": rnd((QR, W), seed + 1, 0.3), "dq.norm": rnd(QR, seed + 2, 0.2) + 1.0, "uq": rnd((H * (D + R), QR), seed + 3, 0.3),
         "dkv": rnd((KR + R, W), seed + 4, 0.3), "dkv.norm": rnd(KR, seed + 5, 0.2) + 1.0, "uk": rnd((H * D, KR), seed + 6, 0.3),
         "uv": rnd((H * V, KR), seed + 7, 0.3), "sink": rnd(H, seed + 8, 2.0), "o": rnd((W, H * V), seed + 10, 0.2)}
    w = {k: bf(v) for k, v in w.items()}
    mixer.load({k.replace(".", "_"): dev(v, dtype) for k, v in w.items()}, dtype, DEV)
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "q_rank": QR, "kv_rank": KR, "scale": scale, "rot": {"base": base, "dims": R}}
    return mixer, w, m


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,D,R,V,QR,KR,W", [(3, 16, 8, 24, 40, 24, 48), (2, 8, 16, 8, 24, 40, 96), (1, 20, 6, 28, 30, 21, 52), (4, 32, 16, 32, 64, 48, 48),
                                             (2, 64, 64, 16, 48, 192, 128), (2, 24, 2, 20, 16, 290, 48)])
def test_latent_attention_without_a_gate_in_neighbouring_pairs(dtype, H, D, R, V, QR, KR, W):
    mixer, w, m = latent_part(H, D, R, V, QR, KR, 0.9 / np.sqrt(D + R), 700.0, dtype, W=W)
    folded = W * mixer.rank_pad <= 2 * V * (mixer.rank_pad + W)
    assert (mixer.w_ov is not None) == folded and (mixer.w_uv is None) == folded
    w64 = f64(w)
    plain = lambda x, m=m, w=w64: VP.latent_attention(x, w, "", m, 1e-5)  # noqa: E731
    xs, ref, tol = walk_a_mixer(mixer, plain, dtype, W, lambda top: (4e-5 if dtype == torch.float32 else 4e-2) * top)
    if dtype == torch.float32:
        x = xs[0].astype(np.float64)
        assert np.abs(plain(x, m, dict(w64, sink=w64["sink"] - 40.0)) - ref[0]).max() > 20 * tol
        if R > 2:
            assert np.abs(plain(x, dict(m, rot={"base": 500.0, "dims": R})) - ref[0]).max() > 20 * tol
            half = np.concatenate([np.arange(0, R, 2), np.arange(1, R, 2)])          # pairs half a width apart
            uq = w64["uq"].reshape(H, D + R, QR).copy()
            uq[:, D:] = uq[:, D:][:, half]
            other = dict(w64, uq=uq.reshape(-1, QR))
            assert np.abs(plain(x, m, other) - ref[0]).max() > 20 * tol


@pytest.mark.parametrize("where", ["prefill", "decode"])
@pytest.mark.parametrize("kind,far", [("differential", 600), ("differential", 64), ("latent", 600), ("latent", 63)])
def test_a_key_that_stands_out_among_hundreds(kind, far, where):
    """One token is made so that a query ``far`` positions later scores it above all others, with a value many times larger; in
    decode the keys are walked in several ranges."""
    from quicknn_b200.cache import KVCache
    W, start = 48, 70
    if kind == "differential":
        mixer, w, m = differential_part(2, 1, 32, 48, 0.15, 0.4, 40.0, (0.2, 100), torch.float32, seed=20)
        w["k"] = w["q"][:64].copy()                                # the key head answers to the first query head's maps
        mixer.load({k: dev(v) for k, v in w.items()}, torch.float32, DEV)
        plain = lambda x: VP.differential_attention(x, f64(w), "", m, 1e-5)  # noqa: E731
    else:
        mixer, w, m = latent_part(3, 32, 16, 24, 32, 40, 2.0, 20000.0, torch.float32, seed=20)
        plain = lambda x: VP.latent_attention(x, f64(w), "", m, 1e-5)  # noqa: E731
    n = start + far + 3
    x = bf(rnd((n, W), 5, 0.3))
    row = start + far
    x[start] = x[row] * 12.0
    ref = plain(x.astype(np.float64))
    blind = x.copy()
    blind[start] = 0.0
    if kind == "differential":
        assert np.abs(ref[row] - plain(blind.astype(np.float64))[row]).max() > 0.05 * np.abs(ref[row]).max()
    cache = KVCache([mixer.cache_need()], [None], 4096, 2, 2048, torch.float32, DEV)
    slot = cache.allocate()
    tol = 4e-5 * np.abs(ref).max()
    if where == "prefill":
        step = part_step([n], [0], [slot], "prefill", torch.float32, cache, mixer)
        assert np.abs(host(mixer.forward(dev(x), step, cache.line(0))) - ref).max() < tol
    else:
        step = part_step([row - 1], [0], [slot], "prefill", torch.float32, cache, mixer)
        mixer.forward(dev(x[:row - 1]), step, cache.line(0))
        for p in range(row - 1, n):
            step = part_step([1], [p], [slot], "decode", torch.float32, cache, mixer)
            y = host(mixer.forward(dev(x[p:p + 1]), step, cache.line(0)))
            assert np.abs(y[0] - ref[p]).max() < tol, f"position {p}"


# ---- whole models ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name,dtype,peaky", [("A", "float32", True), ("A", "bfloat16", False), ("B", "bfloat16", True),
                                              ("B", "float32", True), ("C", "float32", True), ("C", "bfloat16", False)])
def test_every_cutting_gives_the_plain_logits(von, tmp_path, whole_model_tolerance, name, dtype, peaky):
    """Each request whole; its last 32 tokens one by one; batches of unequal lengths that shrink, one batch after another, so that
    slots, pages, rings and states are used again."""
    folder, plain = von(name, dtype, peaky)
    requests = prompts(name, LENGTHS_B if name == "B" else LENGTHS)
    ref = [plain.logits(t) for t in requests]
    replay = Replay(folder, dtype, tmp_path, max_tokens=576 if name == "B" else 384)
    try:
        worst = run_all_cuttings(replay, requests, ref, dtype)
    finally:
        replay.close()
    print(f"vonulorn {name} {dtype} peaky={peaky}: largest error {worst:.3g}")


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_stream_after_every_layer_and_what_a_left_out_part_would_change(von, name):
    from quicknn_b200.engine import Engine, Model
    folder, plain = von(name, "float32", True)
    model = Model.from_folder(folder, "float32", DEV)
    engine = Engine(model, max_tokens=512)
    streams = []
    for blk in model.blocks:
        def wrap(resid, step, line_, normed=None, next_norm=None, _inner=blk.forward):
            out = _inner(resid, step, line_, normed=normed, next_norm=next_norm)
            streams.append(host(out[0] if isinstance(out, tuple) else out))
            return out
        blk.forward = wrap
    toks = prompts(name, [75])[0]
    engine.step([(engine.new_sequence(), toks)], [[len(toks) - 1]])
    want = plain.layers(toks)
    assert len(streams) == want.shape[0] == len(model.spec.schedule)
    for i, (got, ref) in enumerate(zip(streams, want)):
        assert np.abs(got - ref).max() < 3e-5 * np.abs(ref).max(), f"after layer {i}"
    # the weights are such that a part that is left out shows far beyond the tolerance
    ref = plain.logits(toks)
    for suffix, change in ((".sink", lambda t: t - 40.0), (".A_log", lambda t: t + 1.0), (".dt_bias", lambda t: t + 1.0),
                           (".mix.b", lambda t: t * 0.0), (".lq2", lambda t: t * 0.0), (".norm2", lambda t: t - 0.2)):
        w = {k: change(v) if k.endswith(suffix) else v for k, v in plain.w.items()}
        assert np.abs(VP.forward(plain.cfg, w, toks) - ref).max() > 50e-4 * np.abs(ref).max(), suffix


@pytest.mark.parametrize("name,dtype,peaky", [("A", "float32", True), ("B", "float32", True), ("B", "bfloat16", True),
                                              ("C", "float32", True)])
def test_prompts_in_portions_down_to_two_tokens(von, tmp_path, name, dtype, peaky):
    """Steps that continue sequences by several tokens, beside requests that join or sit out."""
    folder, plain = von(name, dtype, peaky)
    big = name == "B"
    requests = prompts(name, [257, 170, 45] if big else [129, 70, 45], seed=7)
    ref = [plain.logits(t) for t in requests]
    replay = Replay(folder, dtype, tmp_path, max_tokens=576 if big else 384)
    pos = [0, 0, 0]

    def step(*parts, end=()):
        entries = [(f"r{i}", requests[i][pos[i]:pos[i] + n], range(n)) for i, n in parts]
        got = replay.step(entries, end=[f"r{i}" for i in end])
        r = 0
        for i, n in parts:
            ok, err, tol = near(got[r:r + n], ref[i][pos[i]:pos[i] + n], dtype)
            assert ok, f"request {i} positions {pos[i]}..{pos[i] + n - 1}: error {err:.3g} > {tol:.3g}"
            pos[i] += n
            r += n
    try:
        a, b = len(requests[0]), len(requests[1])
        step((0, 2), (1, 62))
        step((0, 62))                            # request 1 sits out; request 0 reaches the page edge
        step((0, 2), (1, 2), (2, 40))            # portions of two across the edge; request 2 joins
        step((0, 1), (1, 1), (2, 1))
        step((0, a - 67 - 3), (2, 4), end=[2])
        step((0, 3), (1, b - 65), end=[0, 1])
        assert pos == [a, b, 45]
        got = replay.step([("again", requests[0], [a - 1])], end=["again"])      # what they held is free again
        ok, err, tol = near(got, ref[0][a - 1:a], dtype)
        assert ok, (err, tol)
    finally:
        replay.close()


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(von, name):
    """More requests than slots, so that slots, rings and states are handed out again; decode steps run from CUDA graphs, one step
    ahead of the host, with padding rows; the tokens are the plain implementation's."""
    from quicknn_b200.engine import LLM
    from quicknn_b200.sampling import GenerationOptions
    folder, plain = von(name, "float32", True)
    reqs = prompts(name, [5, 70, 1, 33, 12], seed=3)
    llm = LLM(folder, max_context=256, max_batch=2, dtype="float32")
    res = llm.generate(reqs, GenerationOptions.greedy(12), stop_ids=[])
    for r, p in zip(res, reqs):
        assert r.tokens == plain.greedy(p, 12), f"request {r.index}"
    folder, plain = von(name, "bfloat16", False)
    llm16 = LLM(folder, max_context=256, max_batch=4, dtype="bfloat16")
    for r, p in zip(llm16.generate(reqs, GenerationOptions.greedy(6), stop_ids=[]), reqs):
        seq = list(p)
        for t in r.tokens:                      # bfloat16: every token is at least a near-best one of the plain logits
            row = plain.logits(seq)[-1]
            assert row[t] >= row.max() - 0.15 * (row.max() - row.min())
            seq.append(t)


def test_long_decoding_keeps_states_and_rings(von):
    """150 tokens generated one by one after a short prompt: temperatures step many times, pages fill, states are carried on."""
    from quicknn_b200.engine import LLM
    from quicknn_b200.sampling import GenerationOptions
    folder, plain = von("A", "float32", True)
    p = prompts("A", [3], seed=9)[0]
    llm = LLM(folder, max_context=256, max_batch=1, dtype="float32")
    got = llm.generate([p], GenerationOptions.greedy(150), stop_ids=[])[0].tokens
    seq = p + got
    ref = plain.logits(seq[:-1])
    for i, t in enumerate(got):                 # every generated token is the best one at its place
        row = ref[len(p) - 1 + i]
        assert row[t] >= row.max() - 1e-4 * max(1.0, np.abs(row).max()), f"token {i}"


def test_the_first_tokens_of_a_sequence(von):
    """One to five tokens as prompts, whole and one by one (shorter than the filters, nothing but the sink beside the first key)."""
    from quicknn_b200.engine import Engine, Model
    for name in ("A", "B", "C"):
        folder, plain = von(name, "float32", True)
        engine = Engine(Model.from_folder(folder, "float32", DEV), max_tokens=512)
        toks = prompts(name, [5], seed=4)[0]
        ref = plain.logits(toks)
        for n in range(1, 6):
            s = engine.new_sequence()
            got = host(engine.step([(s, toks[:n])], "all"))
            assert near(got, ref[:n], "float32")[0], (name, n)
            for p in range(n, 5):
                assert near(host(engine.step([(s, [toks[p]])])), ref[p:p + 1], "float32")[0], (name, n, p)
            engine.release(s)


def test_the_command_line_serves_the_design(von, tmp_path):
    import subprocess
    import sys
    from conftest import ROOT

    def run(*argv):
        return subprocess.run([sys.executable, "-m", "quicknn_b200", *argv], cwd=ROOT, capture_output=True, text=True)
    folder, plain = von("A", "float32", True)
    r = run("info", "--model", folder)
    assert r.returncode == 0, r.stderr
    info = json.loads(r.stdout)
    assert info["architecture"] == "Vonulorn" and info["layers"] == len(VON_A["layers"])
    p = prompts("A", [9, 4], seed=5)
    r = run("generate", "--model", folder, "--prompt-ids", ";".join(",".join(map(str, q)) for q in p), "--max-new-tokens", "8",
            "--temperature", "0", "--dtype", "float32", "--max-context", "64", "--stop-ids", "")
    assert r.returncode == 0, r.stderr
    got = [json.loads(l) for l in r.stdout.splitlines() if l.strip()]
    assert [g["tokens"] for g in got] == [plain.greedy(q, 8) for q in p]
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(VON_C))
    out = tmp_path / "random_c"
    r = run("random", "--config", str(cfg), "--seed", "3", "--out", str(out), "--dtype", "bfloat16")
    assert r.returncode == 0, r.stderr
    ref = VP.PlainVonulorn(str(out))
    toks = prompts("C", [21], seed=6)[0]
    replay = Replay(str(out), "float32", tmp_path / "logits", max_tokens=64)       # bfloat16 weights, widened exactly
    try:
        got = replay.step([("x", toks, range(len(toks)))], end=["x"])
    finally:
        replay.close()
    ok, err, tol = near(got, ref.logits(toks), "float32")
    assert ok, (err, tol)


def test_a_model_at_tensor_core_layer_sizes(tmp_path):
    """Both maps in 128 columns, latent rows of 256, states of 128 x 128, prompts of 700 tokens: the products run on the tcgen05
    kernels, the prompt attention on pairs of blocks; a batch that continues by portions and single tokens."""
    from quicknn_b200.engine import Engine, Model
    raw = _model(1024, 512, 1e-5, 0.7, 0.04, [
        _delta(4, 2, 128, 128, 4, 1024), _att(4, 2, 64, 128, 0.12, 0.4, 40.0, (0.2, 256), 1024), _delta(3, 3, 64, 256, 3, 768),
        _lat(4, 64, 64, 64, 256, 192, 0.09, 100000.0, 1024)])
    CONFIGS["T"] = (raw, 11)
    folder = make_folder(tmp_path, "T", "bfloat16", False)
    plain = VP.PlainVonulorn(folder)
    model = Model.from_folder(folder, "bfloat16", DEV)
    engine = Engine(model, max_tokens=4096)
    reqs = prompts("T", [700, 300], seed=2)
    ref = [plain.logits(t) for t in reqs]
    slots = [engine.new_sequence() for _ in reqs]
    rows = [[0, 255, 256, 257, 511, 512, 599], [0, 100, 249]]
    got = host(engine.step([(slots[0], reqs[0][:600]), (slots[1], reqs[1][:250])], rows))
    want = np.concatenate([ref[0][rows[0]], ref[1][rows[1]]])
    ok, err, tol = near(got, want, "bfloat16")
    assert ok, (err, tol)
    got = host(engine.step([(slots[0], reqs[0][600:640]), (slots[1], reqs[1][250:252])], "all"))
    ok, err, tol = near(got, np.concatenate([ref[0][600:640], ref[1][250:252]]), "bfloat16")
    assert ok, (err, tol)
    for k in range(6):
        got = host(engine.step([(slots[0], [reqs[0][640 + k]]), (slots[1], [reqs[1][252 + k]])]))
        ok, err, tol = near(got, np.stack([ref[0][640 + k], ref[1][252 + k]]), "bfloat16")
        assert ok, (k, err, tol)


# ---- configurations drawn at random ---------------------------------------------------------------------------------

def random_config(seed):
    """Every size, the order of the layers and every constant drawn from a seed."""
    rng = np.random.default_rng(4000 + seed)
    pick = lambda xs: xs[int(rng.integers(len(xs)))]  # noqa: E731
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        ff, kind = pick([None, 24, 40, 52, 64, 96]), rng.random()
        kv, per = pick([1, 2, 3]), int(rng.integers(1, 4))
        if kind < 0.45:
            layers.append(_delta(kv * per, kv, pick([8, 12, 16, 21, 32, 40, 64, 128]), pick([8, 12, 16, 20, 33, 48, 64, 96]),
                                 pick([1, 2, 3, 4, 5]), ff))
        elif kind < 0.75:
            layers.append(_att(kv * per, kv, pick([8, 10, 16, 24, 32]), pick([8, 12, 24, 32, 64, 70]), float(rng.uniform(0.1, 0.5)),
                               float(rng.uniform(-0.3, 0.9)), pick([None, 3.0, 15.0, 50.0]),
                               pick([None, (float(rng.uniform(0.05, 1.0)), pick([1, 3, 17, 64, 100]))]), ff))
        else:
            layers.append(_lat(int(rng.integers(1, 6)), pick([8, 16, 20, 32]), pick([2, 6, 8, 16, 32]), pick([8, 20, 24, 32]),
                               pick([16, 24, 40, 64]), pick([16, 21, 40, 64, 100]), float(rng.uniform(0.1, 0.5)),
                               pick([100.0, 10000.0, 500000.0]), ff))
    return _model(int(rng.integers(100, 700)), pick([48, 64, 96, 100, 160, 352]), pick([1e-5, 1e-6]), float(pick([1.0, 0.4, 1.3])), 0.07,
                  layers)


@pytest.mark.parametrize("seed", range(24))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Prompts of unequal lengths in one step, then tokens one by one, against the plain logits: float32 sharply for every
    configuration, bfloat16 for every other one."""
    from quicknn_b200.engine import Engine, Model
    raw = random_config(seed)
    name = f"R{seed}"
    CONFIGS[name] = (raw, 50 + seed)
    lens, extra = [130, 7, 1, 70], 5
    reqs = prompts(name, [n + extra for n in lens], seed=seed)
    for dtype in (("float32", "bfloat16") if seed % 2 == 0 else ("float32",)):
        folder = make_folder(tmp_path, name, dtype, dtype == "float32")
        plain = VP.PlainVonulorn(folder)
        ref = [plain.logits(t) for t in reqs]
        model = Model.from_folder(folder, dtype, DEV)
        engine = Engine(model, max_tokens=1024)
        slots = [engine.new_sequence() for _ in reqs]
        got = host(engine.step([(s, t[:n]) for s, t, n in zip(slots, reqs, lens)], [list(range(n)) for n in lens]))
        ok, err, tol = near(got, np.concatenate([r[:n] for r, n in zip(ref, lens)]), dtype)
        assert ok, f"{dtype} prompts: {err:.3g} > {tol:.3g}   {raw}"
        for k in range(extra):
            got = host(engine.step([(s, [t[n + k]]) for s, t, n in zip(slots, reqs, lens)], [[0]] * len(reqs)))
            ok, err, tol = near(got, np.stack([r[n + k] for r, n in zip(ref, lens)]), dtype)
            assert ok, f"{dtype} token {k}: {err:.3g} > {tol:.3g}   {raw}"
