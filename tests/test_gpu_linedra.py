"""Linedra on the GPU against the plain implementation (tests/plain/linedra_plain.py): the small kernels (causal convolutions,
block-diagonal products, the closing of a layer with its average over depth, the gate per head, the rows of latent
attention); sinks in every attention kernel; the linear recurrence, both mixers and the pair of branches alone over caches of
their own (prompts, single tokens, portions, slots handed out again, keys that stand out just inside and just outside a window
and far back); then whole models through bin/trace_run under every cutting, in portions down to two tokens, through the entry
point's generation loop, the command line, and configurations drawn at random.  The configurations are small and differ from
one another in every size and constant."""
import json
import os

import numpy as np
import pytest
import torch

from plain import linedra_plain as LP
from test_gpu_fuposun import part_step
from test_gpu_replay import Replay, run_all_cuttings

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
BOTH = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module", autouse=True)
def _need_gpu():
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV).to(dtype).contiguous()


def i32(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def host(t):
    return t.detach().float().cpu().numpy().astype(np.float64)


def rnd(shape, seed, scale=1.0):
    return (np.random.default_rng(seed).normal(size=shape) * scale).astype(np.float32)


def bf(a):
    return torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16).float().numpy()


def f64(w):
    return {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}


ROUTED = [0]              # layers with routed experts in the model that is being compared


def routed_layers(raw):
    ROUTED[0] = sum(1 for layer in raw["layers"] if layer.get("mlp") is not None)


def near(got, ref, dtype, float32=1e-4):
    """How whole models are compared.  float32: the largest difference, 1e-4 of the largest logit: the sharp check, since a wrong
    mask, key, window edge, sink, state or expert moves these models' logits by 1e-2 and more.  bfloat16: a row by the root
    mean square of its difference (mean taken off) against that of the logits, at most a tenth; one row in thirty, and as many
    again per routing layer, may lie beyond: a router that sees the bfloat16 rounding of its input chooses another expert
    where two logits lie within rounding of each other."""
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
    over = int((e > 0.1).sum())
    allowed = max(1, len(e) * (1 + ROUTED[0]) // 30)
    return over <= allowed, float(np.sort(e)[-1 - min(over, allowed, len(e) - 1)]), 0.1


@pytest.fixture
def whole_model_tolerance(monkeypatch):
    import test_gpu_replay
    monkeypatch.setattr(test_gpu_replay, "close", near)


# ---- configurations -------------------------------------------------------------------------------------

def _left(heads, kv, dim, vdim, scale, window):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def _par(left, width, blocks, conv, ls, rs, mlp):
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv}, "left_scale": ls, "right_scale": rs}}


def _latent(heads, dim, rot, vdim, q_rank, kv_rank, scale, base, mlp):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot}}}


def _moe(ff, experts, top, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _model(vocab, width, scale, eps, taps, mult, cap, std, layers):
    return dict(architecture="Linedra", vocab=vocab, width=width, embedding={"scale": scale}, norm={"eps": eps},
                canon={"taps": taps}, residual_mult=mult, logit_softcap=cap, initializer_range=std, layers=layers)


# A: a latent layer first and last; grouped queries with values wider than keys; a window shorter than a page and one of a
#    single token; a layer without a feed-forward; taps of 3 and 2; a residual multiplier of 1
LIN_A = _model(300, 64, 2.5, 1e-6, 3, 1.0, 20.0, 0.08, [
    _latent(3, 16, 8, 24, 40, 24, 0.3, 1000.0, _moe(24, 5, 2, 0.9)),
    _par(_left(4, 2, 16, 24, 0.35, 9), 48, 3, 2, 0.7, 1.6, _moe(40, 6, 1, 1.7)),
    _par(_left(2, 1, 24, 16, 0.25, 1), 32, 1, 5, 1.3, 0.6, None),
    _latent(2, 8, 16, 8, 24, 40, 0.25, 20000.0, None)])
# B: head size 64 and latent rows of 64 for the tensor-core kernels, windows beyond a page, parts of 64, experts all chosen
LIN_B = _model(512, 128, 11.0, 1e-5, 4, 0.6, 35.0, 0.06, [
    _par(_left(4, 1, 64, 64, 0.13, 70), 128, 2, 4, 1.1, 0.8, _moe(64, 8, 3, 2.5)),
    _latent(4, 32, 16, 32, 64, 48, 0.17, 30000.0, _moe(32, 4, 4, 1.0)),
    _par(_left(2, 2, 64, 64, 0.11, 130), 64, 4, 3, 0.9, 1.2, _moe(96, 6, 2, 7.0)),
    _par(_left(4, 2, 32, 32, 0.2, None), 96, 3, 4, 1.0, 1.0, None)])
# C: a width, head sizes, ranks, parts and a vocabulary that are no multiple of 8; one tap (no state of the input convolution);
#    one head and one block; a window of exactly a page; no softcap
LIN_C = _model(301, 100, 0.7, 1e-4, 1, 1.4, None, 0.07, [
    _par(_left(5, 5, 12, 20, 0.3, 64), 60, 5, 1, 1.5, 0.5, _moe(36, 3, 3, 3.0)),
    _latent(1, 20, 6, 28, 30, 21, 0.25, 500.0, _moe(12, 9, 4, 0.5)),
    _par(_left(1, 1, 20, 12, 0.22, 33), 36, 1, 6, 0.4, 1.9, None)])
CONFIGS = {"A": (LIN_A, 3), "B": (LIN_B, 4), "C": (LIN_C, 5)}
LENGTHS = [70, 33, 129, 45, 100, 64]
LENGTHS_B = [170, 33, 257, 45, 100, 64]


def stand_out(tensors, peaky):
    """What random draws would leave trivial: sinks of the size of the scores, decays from nearly none to nearly all, filters and
    averages over depth with sizeable numbers of both signs; ``peaky``: scores and router logits scaled up."""
    for k in list(tensors):
        t = tensors[k]
        if k.endswith(".sink"):
            tensors[k] = t * 8.0
        elif k.endswith(".lam"):
            tensors[k] = torch.linspace(-6.0, 1.5, t.numel())
        elif k.endswith(".canon1") or k.endswith(".conv"):
            tensors[k] = t * 4.0 if k.endswith(".canon1") else t * 0.5
        elif k.endswith(".dwa"):
            tensors[k] = t + 0.4 * torch.cos(torch.arange(t.numel()) * 1.7)
        elif peaky and (k.endswith("mlp.router") or k.endswith("left.q") or k.endswith("mix.uq")):
            tensors[k] = t * 4.0
    return tensors


def make_folder(base, name, storage, peaky):
    from quicknn_b200.config import LINEDRA, LinedraConfig
    from quicknn_b200.weights import random_tensors, write_safetensors
    raw, seed = CONFIGS[name]
    cfg = LinedraConfig.from_dict(raw)
    d = os.path.join(str(base), f"line{name}_{storage}{'_peaky' if peaky else ''}")
    os.makedirs(d, exist_ok=True)
    tensors = stand_out(dict(random_tensors(LINEDRA, cfg, seed, torch.float32, 0.2)), peaky)
    dt = torch.float32 if storage == "float32" else torch.bfloat16
    with open(os.path.join(d, "config.json"), "w") as fh:
        json.dump(cfg.to_dict(), fh)
    write_safetensors(os.path.join(d, "model.safetensors"), {k: v.to(dt).contiguous() for k, v in tensors.items()})
    return d


@pytest.fixture(scope="module")
def line(tmp_path_factory):
    base = tmp_path_factory.mktemp("linedra")
    made = {}

    def get(name, storage="float32", peaky=False):
        key = (name, storage, peaky)
        if key not in made:
            folder = make_folder(base, name, storage, peaky)
            made[key] = (folder, LP.PlainLinedra(folder))
        return made[key]
    return get


def prompts(name, lengths, seed=0):
    rng = np.random.default_rng(100 + seed)
    return [rng.integers(1, CONFIGS[name][0]["vocab"], n).tolist() for n in lengths]


# ---- the small kernels ------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("C,taps", [(64, 4), (72, 3), (40, 2), (48, 1), (37, 4), (24, 7), (264, 4)])
def test_causal_convolution_over_prompts_portions_and_single_tokens(dtype, C, taps):
    """Sequences of 21, 1 and 40 rows, then portions of 2, 17 and 1, then single tokens; a slot that another sequence held keeps
    nothing of it; a row of no sequence stays zero.  Columns in the middle of wider rows, with and without biases and the input."""
    from quicknn_b200.kernels import ops
    w, xb, ob = bf(rnd((C, taps), 1, 0.5)), bf(rnd(C, 2, 0.5)), bf(rnd(C, 3, 0.5))
    total, col0 = 70, 8
    xs = [bf(rnd((total, C), 10 + i)) for i in range(3)]
    for biased, add in ((False, True), (True, False)):
        ref = []
        for x in xs:
            v = x.astype(np.float64) + (xb if biased else 0)
            ref.append(LP.causal_conv(v, w.astype(np.float64)) + (ob if biased else 0) + (v if add else 0))
        tol = (2e-6 if dtype == torch.float32 else 0.01) * max(np.abs(r).max() for r in ref)
        state = torch.full((5, taps + 1, C), 9.0, device=DEV)             # what other sequences left there
        slots = [3, 0, 4]
        pos = [0, 0, 0]

        def step(lens, decode=False):
            live = [i for i, n in enumerate(lens) if n]
            rows = np.concatenate([xs[i][pos[i]:pos[i] + lens[i]] for i in live])
            wide = np.zeros((len(rows) + int(decode), C + 16), np.float32)
            wide[:len(rows), col0:col0 + C] = rows
            tok_pos = np.concatenate([np.arange(pos[i], pos[i] + lens[i]) for i in live] + ([[0]] if decode else []))
            ns = [lens[i] for i in live]
            row0 = np.cumsum([0] + ns[:-1])
            sl = [slots[i] for i in live] + ([-1] if decode else [])
            kw = dict(x_bias=dev(xb, dtype), out_bias=dev(ob, dtype)) if biased else {}
            y = host(ops.causal_conv(dev(wide, dtype), dev(w, dtype), state, None if decode else i32(row0),
                                     None if decode else i32(ns), i32(tok_pos), i32(sl), len(sl), max(ns), col0=col0,
                                     add_input=add, **kw))
            if decode:
                assert np.abs(y[-1]).max() == 0.0
            r = 0
            for i in live:
                assert np.abs(y[r:r + lens[i]] - ref[i][pos[i]:pos[i] + lens[i]]).max() < tol, (i, pos[i], lens)
                pos[i] += lens[i]
                r += lens[i]
        step([21, 1, 40])
        step([2, 17, 1])
        for _ in range(taps + 3):
            step([1, 1, 1], decode=True)
        step([9, 0, 3])
        step([1, 1, 0], decode=True)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,B,N,K", [(5, 3, 40, 24), (70, 2, 64, 64), (300, 4, 130, 72), (33, 1, 24, 200), (17, 5, 12, 12),
                                     (40, 2, 7, 9), (16, 6, 96, 320), (1000, 8, 192, 96), (3600, 8, 256, 64)])
def test_block_diagonal_products(dtype, T, B, N, K):
    """Parts of rows times matrices of their own: float32 and rounded results, a gate per output, parts that lie further apart
    than they are wide."""
    from quicknn_b200.kernels import ops
    w = bf(rnd((B, N, K), 1, K ** -0.5))
    step, col0 = K + 8, 8
    x = bf(rnd((T, col0 + B * step), 2))
    g = bf(rnd((T, B * N + 3), 3))
    parts = np.stack([x[:, col0 + b * step:col0 + b * step + K] for b in range(B)], axis=1).astype(np.float64)
    ref = np.einsum("tbk,bnk->tbn", parts, w.astype(np.float64)).reshape(T, B * N)
    y = host(ops.block_linear(dev(x, dtype), dev(w, dtype), col0=col0, step=step, out_dtype=torch.float32))
    assert np.abs(y - ref).max() < 3e-6 * np.abs(ref).max()          # sums are float32 and stay so
    want = ref * LP.sigmoid(g[:, 3:].astype(np.float64))
    y = host(ops.block_linear(dev(x, dtype), dev(w, dtype), col0=col0, step=step, gate=dev(g, dtype), gate_col0=3))
    assert np.abs(y - want).max() < (3e-6 if dtype == torch.float32 else 0.005) * np.abs(want).max()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H", [64, 100, 1024, 2312, 37, 9000])
def test_closing_a_layer_with_an_average_over_depth(dtype, H):
    """X = x + m norm(y); the average over earlier results; the next norm; y in one row or as the sum of several."""
    from quicknn_b200.kernels import ops
    T, mult, eps = 5, 0.7, 1e-5
    wp, wn = bf(rnd(H, 1, 0.3)), bf(rnd(H, 2, 0.3))
    x = rnd((T, H), 3, 2.0)
    for terms in (1, 3):
        y = bf(rnd((T * terms, H), 4))
        X = x + mult * LP.norm_about_zero(y.astype(np.float64).reshape(T, terms, H).sum(1), wp.astype(np.float64), eps)
        for n in (None, 1, 2, 6):
            hist = None if n is None else rnd((n, T, H), 5)
            num = None if n is None else bf(rnd(n + 1, 6))
            Z = X if n is None else (num[:n, None, None] * hist).sum(0) + num[n] * X
            want = LP.norm_about_zero(Z, wn.astype(np.float64), eps)
            resid, out, avg = dev(x), torch.zeros((T, H), device=DEV), torch.zeros((T, H), device=DEV)
            kw = {} if n is None else dict(hist=dev(hist), numbers=dev(num, dtype), avg_out=avg)
            got = ops.stream_update(resid, dev(y, dtype), mult, dev(wp, dtype), eps, True, out, terms=terms,
                                    w_next=dev(wn, dtype), eps_next=eps, unit_next=True, out_dtype=dtype, **kw)
            assert np.abs(host(resid) - x).max() == 0.0                  # a place of its own: what came in is not touched
            assert np.abs(host(out) - X).max() < 3e-6 * np.abs(X).max()
            if n is not None:
                assert np.abs(host(avg) - Z).max() < 3e-6 * np.abs(Z).max()
            assert np.abs(host(got) - want).max() < (4e-6 if dtype == torch.float32 else 0.006) * np.abs(want).max()
        r = dev(x)
        assert ops.stream_update(r, dev(y, dtype), mult, dev(wp, dtype), eps, True, terms=terms) is None     # in place, no norm
        assert np.abs(host(r) - X).max() < 3e-6 * np.abs(X).max()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,taps", [(64, 4), (72, 3), (128, 2), (64, 1), (100, 4), (64, 6), (4608, 4)])
def test_the_convolution_inside_the_kernel_that_closes_a_layer(dtype, H, taps):
    """Decode steps: n = norm(x + norm(y)) and n + conv(n) with the sequence's last rows, beside a row of no sequence; sizes that
    the fused kernel does not take give the same."""
    from quicknn_b200.kernels import ops
    B, n = 3, taps + 4
    wp, wn, cw = bf(rnd(H, 1, 0.3)), bf(rnd(H, 2, 0.3)), bf(rnd((H, taps), 3, 0.4))
    xs, ys = rnd((B, n, H), 4), bf(rnd((B, n, H), 5))
    ref = []
    for b in range(B):
        h = LP.norm_about_zero(xs[b] + 0.5 * LP.norm_about_zero(ys[b].astype(np.float64), wp.astype(np.float64), 1e-5),
                               wn.astype(np.float64), 1e-5)
        ref.append(h + LP.causal_conv(h, cw.astype(np.float64)))
    tol = (4e-6 if dtype == torch.float32 else 0.012) * np.abs(ref).max()
    state = torch.full((B + 1, taps, H), 7.0, device=DEV)
    slots = i32([2, 0, -1, 3])
    for t in range(n):
        pos = i32([t, t, 0, t])
        rows = lambda a: np.insert(a[:, t], 2, 0.0, axis=0)  # noqa: E731
        got = host(ops.stream_update(dev(rows(xs)), dev(rows(ys), dtype), 0.5, dev(wp, dtype), 1e-5, True, w_next=dev(wn, dtype),
                                     eps_next=1e-5, unit_next=True, out_dtype=dtype, conv=(dev(cw, dtype), state, pos, slots)))
        assert np.abs(got[[0, 1, 3]] - np.stack([r[t] for r in ref])).max() < tol, f"token {t}"
    assert float((state[1] - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", BOTH)
def test_a_gate_per_head_from_logits_or_from_a_matrix_scaled_into_wider_rows(dtype):
    from quicknn_b200.kernels import ops
    for T, H, D, W in ((3, 4, 16, 48), (9, 5, 12, 40), (2, 1, 128, 64)):
        o, x, w = bf(rnd((T, H * D), 1)), bf(rnd((T, W), 2)), bf(rnd((H, W), 3, 0.3))
        z = x.astype(np.float64) @ w.T.astype(np.float64)
        ref = (o.reshape(T, H, D) * 1.25 * LP.sigmoid(z)[:, :, None]).reshape(T, H * D)
        tol = (2e-6 if dtype == torch.float32 else 0.006) * np.abs(ref).max()
        out = torch.zeros((T, H * D + 24), dtype=dtype, device=DEV)
        ops.gate_heads(dev(o, dtype), dev(x, dtype), dev(w, dtype), H, 1.25, out, 8)
        assert np.abs(host(out)[:, 8:8 + H * D] - ref).max() < tol and float(out[:, :8].abs().max()) == 0.0
        zz = bf(z)
        ref = (o.reshape(T, H, D) * LP.sigmoid(zz.astype(np.float64))[:, :, None]).reshape(T, H * D)
        rows = np.concatenate([rnd((T, 5), 4), zz, rnd((T, 2), 5)], axis=1)
        got = host(ops.gate_heads(dev(o, dtype), dev(rows, dtype), None, H, x_col0=5))
        assert np.abs(got - ref).max() < tol


# ---- sinks in the attention kernels ------------------------------------------------------------------------------

def plain_heads(qkv, H, G, D, scale, window, sinks, slopes=None, cap=None):
    n = qkv.shape[0]
    q, k, v = qkv[:, :H * D].reshape(n, H, D), qkv[:, H * D:(H + G) * D].reshape(n, G, D), qkv[:, (H + G) * D:].reshape(n, G, D)
    i = np.arange(n)
    out = np.zeros((n, H, D))
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        if cap:
            s = cap * np.tanh(s / cap)
        if slopes is not None:
            s = s - slopes[h] * (i[:, None] - i[None, :])
        out[:, h] = LP.softmax_with_sink(s, LP.causal(n, window), sinks[h]) @ v[:, h // (H // G)]
    return out.reshape(n, H * D)


@pytest.mark.parametrize("dtype,D,tcgen05", [(torch.float32, 40, True), (torch.bfloat16, 40, True), (torch.bfloat16, 64, True),
                                             (torch.bfloat16, 128, True), (torch.bfloat16, 256, True), (torch.bfloat16, 64, False),
                                             (torch.bfloat16, 256, False)])
@pytest.mark.parametrize("cap,window,biased", [(None, None, True), (None, 70, False), (8.0, None, False)])
def test_sinks_in_prompts(monkeypatch, dtype, D, tcgen05, cap, window, biased):
    """The plain, mma.sync and tcgen05 prompt kernels (with a softcap the last one's other form; one long prompt for its pairs of
    blocks), rows packed in wider rows.  Sinks far below, among and far above the scores: the last leave almost nothing."""
    from quicknn_b200.kernels import ops
    monkeypatch.setattr(ops, "ATTN_TCGEN05", tcgen05)
    H, G, scale = 4, 2, D ** -0.5
    sinks = np.array([-30.0, 0.5, 3.0, 120.0])
    slopes = LP.distance_slopes(H) if biased else None
    for lens in ([150, 1, 67], [1500]):
        rows = bf(rnd((sum(lens), (H + 2 * G) * D + 16), 1, 1.2))
        qkv = dev(rows, dtype)[:, :(H + 2 * G) * D]
        row0 = np.cumsum([0] + lens[:-1])
        pos = np.concatenate([np.arange(n) for n in lens])
        got = host(ops.attn_prefill(qkv, H, G, D, i32(pos), i32(np.repeat(row0, lens)), scale, cap, window, i32(row0), i32(lens),
                                    max(lens), slopes=None if slopes is None else dev(slopes), sinks=dev(sinks)))
        ops.raise_on_status(DEV)
        for r, n in zip(row0, lens):
            ref = plain_heads(rows[r:r + n, :(H + 2 * G) * D].astype(np.float64), H, G, D, scale, window, sinks, slopes, cap)
            tol = (2e-5 if dtype == torch.float32 else 0.02) * np.abs(ref).max()
            assert np.abs(got[r:r + n] - ref).max() < tol
            assert np.abs(ref[:, 3 * D:]).max() < 1e-9 and np.abs(ref[:, :3 * D]).max() > 0.1


def attention_part(H, G, D, V, scale, window, dtype, W=48, seed=0):
    from quicknn_b200.parts import MIXERS, PartSpec
    spec = PartSpec("attention", {
        "hidden_size": W, "n_heads": H, "n_kv_heads": G, "head_dim": D, "v_head_dim": V, "scale": scale, "softcap": None,
        "window": window, "position": PartSpec("none", {"head_dim": D}), "distance_slopes": tuple(LP.distance_slopes(H)),
        "sink": True, "head_gate": True})
    mixer = MIXERS.get(spec.kind)(spec)
    w = {"q": bf(rnd((H * D, W), seed + 1, 0.4)), "k": bf(rnd((G * D, W), seed + 2, 0.4)), "v": bf(rnd((G * V, W), seed + 3, 0.3)),
         "sink": bf(rnd(H, seed + 4, 2.0)), "g": bf(rnd((H, W), seed + 5, 0.3)), "o": bf(rnd((W, H * V), seed + 6, 0.2))}
    names = {"q": "q_proj", "k": "k_proj", "v": "v_proj", "sink": "sink", "g": "head_gate", "o": "o_proj"}
    mixer.load({names[k]: dev(v, dtype) for k, v in w.items()}, dtype, DEV)
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    return mixer, w, m


def latent_part(H, D, R, V, QR, KR, scale, base, dtype, W=48, seed=0):
    from quicknn_b200.parts import MIXERS, PartSpec
    spec = PartSpec("latent_attention", {
        "hidden_size": W, "n_heads": H, "dim": D, "vdim": V, "q_rank": QR, "kv_rank": KR, "scale": scale, "window": None,
        "eps": 1e-5, "sink": True, "gate": "element", "position": PartSpec("rotary", {"head_dim": R, "theta": base, "rotary_dim": R})})
    mixer = MIXERS.get(spec.kind)(spec)
    w = {"dq": bf(rnd((QR, W), seed + 1, 0.3)), "dq.norm": bf(rnd(QR, seed + 2, 0.2) + 1.0), "uq": bf(rnd((H * (D + R), QR), seed + 3, 0.3)),
         "dkv": bf(rnd((KR + R, W), seed + 4, 0.3)), "dkv.norm": bf(rnd(KR, seed + 5, 0.2) + 1.0), "uk": bf(rnd((H * D, KR), seed + 6, 0.3)),
         "uv": bf(rnd((H * V, KR), seed + 7, 0.3)), "sink": bf(rnd(H, seed + 8, 2.0)), "g": bf(rnd((H * V, W), seed + 9, 0.3)),
         "o": bf(rnd((W, H * V), seed + 10, 0.2))}
    names = {"dq": "dq", "dq.norm": "dq_norm", "uq": "uq", "dkv": "dkv", "dkv.norm": "dkv_norm", "uk": "uk", "uv": "uv", "sink": "sink",
             "g": "gate", "o": "o"}
    mixer.load({names[k]: dev(v, dtype) for k, v in w.items()}, dtype, DEV)
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "q_rank": QR, "kv_rank": KR, "scale": scale, "rot": {"base": base, "dims": R}}
    return mixer, w, m


def walk_a_mixer(mixer, plain, dtype, W, tol_of, lens=(200, 1, 67), extra=70, portion=30):
    """Prompts of unequal lengths, ``extra`` single tokens each, a portion onto the first beside a single token of the third, then
    a slot (with its pages and state) that the first sequence gives back; all against the plain whole sequences."""
    from quicknn_b200.cache import KVCache
    cache = KVCache([mixer.cache_need()], [mixer.state_need()], 2048, 4, 512, dtype, DEV)
    lens = list(lens)
    xs = [bf(rnd((n + extra + portion, W), 30 + i)) for i, n in enumerate(lens)]
    ref = [plain(x.astype(np.float64)) for x in xs]
    tol = tol_of(max(np.abs(r).max() for r in ref))
    slots = [cache.allocate() for _ in lens]

    def run(ns, starts, which, mode):
        step = part_step(ns, starts, [slots[i] for i in which], mode, dtype, cache, mixer)
        rows = np.concatenate([xs[i][s:s + n] for i, s, n in zip(which, starts, ns)])
        y = host(mixer.forward(dev(rows, dtype), step, cache.line(0)))
        want = np.concatenate([ref[i][s:s + n] for i, s, n in zip(which, starts, ns)])
        err = np.abs(y - want).max()
        assert err < tol, f"{mode} {ns} from {starts}: {err:.3g} > {tol:.3g}"
    run(lens, [0, 0, 0], [0, 1, 2], "prefill")
    for t in range(extra):
        run([1, 1, 1], [n + t for n in lens], [0, 1, 2], "decode")
    run([portion - 2, 1], [lens[0] + extra, lens[2] + extra], [0, 2], "extend")
    run([2], [lens[0] + extra + portion - 2], [0], "extend")
    cache.free(slots[0])
    again = cache.allocate()
    x2 = bf(rnd((90, W), 77))
    step = part_step([90], [0], [again], "prefill", dtype, cache, mixer)
    y = host(mixer.forward(dev(x2, dtype), step, cache.line(0)))
    assert np.abs(y - plain(x2.astype(np.float64))).max() < tol
    return xs, ref, tol


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,D,V,window", [(4, 2, 16, 16, 9), (2, 2, 24, 40, 1), (6, 1, 64, 64, 70), (3, 3, 12, 20, 64),
                                            (8, 4, 64, 32, 100), (2, 1, 128, 128, 130), (1, 1, 8, 8, 63), (10, 1, 32, 32, 65),
                                            (5, 5, 40, 40, None), (4, 1, 256, 256, 137)])
def test_window_attention_alone_and_a_window_sink_or_slope_that_is_off_would_show(dtype, H, G, D, V, window):
    W = 48
    mixer, w, m = attention_part(H, G, D, V, 1.2 / np.sqrt(D), window, dtype)
    w64 = f64(w)
    xs, ref, tol = walk_a_mixer(mixer, lambda x: LP.window_attention(x, w64, "", m), dtype, W,
                                lambda top: (3e-5 if dtype == torch.float32 else 4e-2) * top)
    if dtype == torch.float32:
        x = xs[0].astype(np.float64)
        for off in ([] if window is None else [-1, 1] if window > 1 else [1]):
            assert np.abs(LP.window_attention(x, w64, "", dict(m, mask={"size": window + off})) - ref[0]).max() > 20 * tol
        assert np.abs(LP.window_attention(x, dict(w64, sink=w64["sink"] - 40.0), "", m) - ref[0]).max() > 20 * tol


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,D,R,V,QR,KR", [(3, 16, 8, 24, 40, 24), (2, 8, 16, 8, 24, 40), (1, 20, 6, 28, 30, 21), (4, 32, 16, 32, 64, 48),
                                           (9, 16, 32, 16, 32, 96), (2, 64, 64, 48, 48, 192), (2, 24, 2, 20, 16, 290)])
def test_latent_attention_alone_and_a_sink_or_a_rotation_that_is_left_out_would_show(dtype, H, D, R, V, QR, KR):
    W = 48
    mixer, w, m = latent_part(H, D, R, V, QR, KR, 0.9 / np.sqrt(D + R), 700.0, dtype)
    assert mixer.cache_need().head_dim == (64 if KR + R <= 64 else 128 if KR + R <= 128 else 256 if KR + R <= 256 else -(-(KR + R) // 8) * 8)
    w64 = f64(w)
    xs, ref, tol = walk_a_mixer(mixer, lambda x: LP.latent_attention(x, w64, "", m, 1e-5), dtype, W,
                                lambda top: (4e-5 if dtype == torch.float32 else 4e-2) * top)
    if dtype == torch.float32:
        x = xs[0].astype(np.float64)
        assert np.abs(LP.latent_attention(x, dict(w64, sink=w64["sink"] - 40.0), "", m, 1e-5) - ref[0]).max() > 20 * tol
        assert np.abs(LP.latent_attention(x, w64, "", dict(m, rot={"base": 500.0 if R > 2 else 1e30, "dims": R}), 1e-5) - ref[0]).max() \
            > (20 * tol if R > 2 else -1)


@pytest.mark.parametrize("where", ["prefill", "decode"])
@pytest.mark.parametrize("kind,window,far", [("window", 88, 87), ("window", 88, 88), ("window", 65, 64), ("window", 65, 65),
                                             ("window", None, 600), ("latent", None, 600), ("latent", None, 64)])
def test_a_key_that_stands_out_among_hundreds(kind, window, far, where):
    """One token is made so that a query ``far`` positions later scores it above all others, with a value many times larger:
    seen inside the window (its last position), not just outside; several key ranges in decode steps."""
    from quicknn_b200.cache import KVCache
    W, start = 48, 70
    if kind == "window":
        mixer, w, m = attention_part(4, 2, 32, 32, 0.4, window, torch.float32, seed=20)
        w["k"] = bf(np.concatenate([w["q"][:32], w["q"][64:96]]))          # a key head that answers to the first of its queries
        mixer.load({"q_proj": dev(w["q"]), "k_proj": dev(w["k"]), "v_proj": dev(w["v"]), "sink": dev(w["sink"]),
                    "head_gate": dev(w["g"]), "o_proj": dev(w["o"])}, torch.float32, DEV)
        m = dict(m)
        plain = lambda x: LP.window_attention(x, f64(w), "", m)  # noqa: E731
        mixer.slopes = dev(LP.distance_slopes(4))
    else:
        mixer, w, m = latent_part(3, 32, 16, 24, 32, 40, 2.0, 20000.0, torch.float32, seed=20)
        plain = lambda x: LP.latent_attention(x, f64(w), "", m, 1e-5)  # noqa: E731
    n = start + far + 3
    x = bf(rnd((n, W), 5, 0.3))
    row = start + far
    x[start] = x[row] * 12.0
    ref = plain(x.astype(np.float64))
    blind = x.copy()
    blind[start] = 0.0
    differs = np.abs(ref[row] - plain(blind.astype(np.float64))[row]).max()
    seen = window is None or far < window
    if kind == "window" and (far < 100 or not seen):                       # (the steepest slopes bury a key 600 positions back)
        assert (differs > 0.02 * np.abs(ref[row]).max()) == seen
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


# ---- the linear recurrence and the pair of branches alone ----------------------------------------------------------------

def recurrence_weights(width, blocks, conv, W, seed=0):
    d = width // blocks
    return {"y": bf(rnd((width, W), seed + 1, 0.3)), "y.b": bf(rnd(width, seed + 2, 0.3)), "x": bf(rnd((width, W), seed + 3, 0.3)),
            "x.b": bf(rnd(width, seed + 4, 0.3)), "conv": bf(rnd((width, conv), seed + 5, 0.5)), "conv.b": bf(rnd(width, seed + 6, 0.3)),
            "ra": bf(rnd((blocks, d, d), seed + 7, 1.5 / np.sqrt(d))), "ra.b": bf(rnd((blocks, d), seed + 8)),
            "ri": bf(rnd((blocks, d, d), seed + 9, 1.5 / np.sqrt(d))), "ri.b": bf(rnd((blocks, d), seed + 10)),
            "lam": bf(np.linspace(-7.0, 2.0, width)), "o": bf(rnd((W, width), seed + 11, 0.2))}


RECURRENCE_NAMES = {"y": "y", "y.b": "y_bias", "x": "x", "x.b": "x_bias", "conv": "conv", "conv.b": "conv_bias", "ra": "r", "ra.b": "r_bias",
                    "ri": "i", "ri.b": "i_bias", "lam": "lam", "o": "o"}


def recurrence_part(width, blocks, conv, dtype, W=48):
    from quicknn_b200.parts import MIXERS, PartSpec
    spec = PartSpec("rglru", {"hidden_size": W, "width": width, "blocks": blocks, "conv": conv})
    mixer = MIXERS.get("rglru")(spec)
    w = recurrence_weights(width, blocks, conv, W)
    mixer.load({RECURRENCE_NAMES[k]: dev(v, dtype) for k, v in w.items()}, dtype, DEV)
    return mixer, w


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("width,blocks,conv", [(64, 2, 4), (48, 3, 2), (32, 1, 1), (60, 5, 3), (36, 1, 6), (320, 4, 4), (96, 12, 9),
                                               (144, 2, 4)])
def test_the_recurrent_block_alone_and_a_lost_state_would_show(dtype, width, blocks, conv):
    mixer, w = recurrence_part(width, blocks, conv, dtype)
    w64 = f64(w)
    xs, ref, tol = walk_a_mixer(mixer, lambda x: LP.recurrent_block(x, w64, ""), dtype, 48,
                                lambda top: (3e-5 if dtype == torch.float32 else 4e-2) * top)
    fresh = LP.recurrent_block(xs[0][200:].astype(np.float64), w64, "")      # the same tokens without what came before them
    assert np.abs(fresh[:40] - ref[0][200:240]).max() > (20 if dtype == torch.float32 else 2) * tol


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("width,blocks", [(96, 2), (40, 5)])
def test_long_prompts_walk_the_recurrence_in_segments(dtype, width, blocks):
    """2500 rows (segments chained by a kernel of their own), 33, 32 and 5 rows beside one another; then 600 and 40
    rows onto states that are not empty; the plain walk, and for bfloat16 rows also the gates formed by kernels of their own."""
    from quicknn_b200.cache import KVCache
    from quicknn_b200.kernels import ops
    W = 48
    mixer, w = recurrence_part(width, blocks, 4, dtype)
    lens = [2500, 33, 32, 5]
    xs = [bf(rnd((n + 600, W), 40 + i)) for i, n in enumerate(lens)]
    ref = [LP.recurrent_block(x.astype(np.float64), f64(w), "") for x in xs]
    tol = (3e-5 if dtype == torch.float32 else 4e-2) * max(np.abs(r).max() for r in ref)
    for fused in ((True, False) if dtype == torch.bfloat16 else (True,)):
        ops.RECURRENCE_GATES_FUSED = fused
        try:
            cache = KVCache([None], [mixer.state_need()], 8192, 4, 4096, dtype, DEV)
            slots = [cache.allocate() for _ in lens]
            step = part_step(lens, [0] * 4, slots, "prefill", dtype, cache, mixer)
            y = host(mixer.forward(dev(np.concatenate([x[:n] for x, n in zip(xs, lens)]), dtype), step, cache.line(0)))
            assert np.abs(y - np.concatenate([r[:n] for r, n in zip(ref, lens)])).max() < tol
            step = part_step([600, 40], [2500, 5], [slots[0], slots[3]], "extend", dtype, cache, mixer)
            y = host(mixer.forward(dev(np.concatenate([xs[0][2500:3100], xs[3][5:45]]), dtype), step, cache.line(0)))
            assert np.abs(y - np.concatenate([ref[0][2500:3100], ref[3][5:45]])).max() < tol
            step = part_step([1, 1], [33, 32], [slots[1], slots[2]], "decode", dtype, cache, mixer)
            y = host(mixer.forward(dev(np.stack([xs[1][33], xs[2][32]]), dtype), step, cache.line(0)))
            assert np.abs(y - np.stack([ref[1][33], ref[2][32]])).max() < tol
        finally:
            ops.RECURRENCE_GATES_FUSED = True


@pytest.mark.parametrize("rows", [1, 8, 17, 40, 70])
def test_decode_batches_of_the_recurrent_block(rows):
    """One token for many sequences at unlike positions (tiles of 16 rows; beyond 64 rows the kernels one by one), with a row of no
    sequence among them."""
    from quicknn_b200.cache import KVCache
    W, dtype = 48, torch.bfloat16
    mixer, w = recurrence_part(96, 2, 4, dtype)
    cache = KVCache([None], [mixer.state_need()], 128 * 64, rows + 1, 64, dtype, DEV)
    slots = [cache.allocate() for _ in range(rows)]
    lens = [1 + (5 * i) % 7 for i in range(rows)]
    xs = [bf(rnd((n + 3, W), 200 + i)) for i, n in enumerate(lens)]
    ref = [LP.recurrent_block(x.astype(np.float64), f64(w), "") for x in xs]
    tol = 4e-2 * max(np.abs(r).max() for r in ref)
    step = part_step(lens, [0] * rows, slots, "prefill", dtype, cache, mixer)
    mixer.forward(dev(np.concatenate([x[:n] for x, n in zip(xs, lens)]), dtype), step, cache.line(0))
    for t in range(3):
        step = part_step([1] * rows, [n + t for n in lens], slots, "decode", dtype, cache, mixer)
        x = np.stack([x[n + t] for x, n in zip(xs, lens)])
        if rows == 17:                                   # a padding row at the end, as a padded decode step has it
            step.slots, step.tok_pos = i32(slots + [-1]), i32([n + t for n in lens] + [0])
            step.n_seqs += 1
            x = np.concatenate([x, np.ones((1, W), np.float32)])
        y = host(mixer.forward(dev(x, dtype), step, cache.line(0)))
        assert np.abs(y[:rows] - np.stack([r[n + t] for r, n in zip(ref, lens)])).max() < tol
        if rows == 17:
            assert np.abs(y[rows]).max() == 0.0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("H,G,D,V,window,width,blocks", [(4, 2, 16, 24, 9, 48, 3), (2, 1, 64, 64, 70, 128, 2), (5, 5, 12, 20, None, 36, 1)])
def test_the_two_branches_side_by_side(dtype, H, G, D, V, window, width, blocks):
    """One input product, one output product, the branches' numbers: prompts, single tokens, portions, a reused slot."""
    from quicknn_b200.parts import MIXERS, PartSpec
    W = 48
    left, wl, m = attention_part(H, G, D, V, 1.0 / np.sqrt(D), window, dtype)
    right = PartSpec("rglru", {"hidden_size": W, "width": width, "blocks": blocks, "conv": 3})
    mixer = MIXERS.get("parallel")(PartSpec("parallel", {"hidden_size": W, "eps": 1e-5, "branches": {"left": left.spec, "right": right},
                                                         "scales": {"left": 1.7, "right": -0.6}}))
    wr = recurrence_weights(width, blocks, 3, W, seed=50)
    tensors = {"left." + n: dev(wl[k], dtype) for k, n in (("q", "q_proj"), ("k", "k_proj"), ("v", "v_proj"), ("sink", "sink"),
                                                           ("g", "head_gate"), ("o", "o_proj"))}
    tensors.update({"right." + RECURRENCE_NAMES[k]: dev(v, dtype) for k, v in wr.items()})
    assert set(tensors) == set(MIXERS.get("parallel").param_shapes(mixer.spec))
    mixer.load(tensors, dtype, DEV)
    w = {**{"left." + k: v for k, v in f64(wl).items()}, **{"right." + k: v for k, v in f64(wr).items()}}
    raw = {"left": m, "right": {}, "left_scale": 1.7, "right_scale": -0.6}
    walk_a_mixer(mixer, lambda x: LP.parallel(x, w, "", raw), dtype, W, lambda top: (3e-5 if dtype == torch.float32 else 4e-2) * top)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("experts,top,W,ff,T", [(5, 2, 48, 24, 9), (1, 1, 64, 32, 4), (9, 4, 100, 12, 33), (8, 8, 64, 64, 70),
                                                (4, 2, 128, 96, 400), (33, 3, 64, 40, 50)])
def test_routed_experts_weighted_by_a_softmax_over_the_chosen_logits(dtype, experts, top, W, ff, T):
    from quicknn_b200.parts import FEED_FORWARDS, PartSpec
    ffn = FEED_FORWARDS.get("routed_experts")(PartSpec("routed_experts", {
        "hidden_size": W, "experts": experts, "top": top, "intermediate_size": ff, "limit": 0.8, "score": "softmax",
        "renormalize": True, "weight_on": "output"}))
    w = {"router": bf(rnd((experts, W), 1, 0.4))}
    names = {"router": "router"}
    for e in range(experts):
        for n, shape in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))):
            w[f"e{e}.{n}"] = bf(rnd(shape, 10 * e + len(n), 0.3))
            names[f"e{e}.{n}"] = f"experts.{e}.{n}_proj"
    ffn.load({names[k]: dev(v, dtype) for k, v in w.items()}, dtype, DEV)
    x = bf(rnd((T, W), 7))
    w64 = f64(w)
    ref = LP.routed(x.astype(np.float64), w64, "", {"router": {"experts": experts, "top": top}, "expert": {"limit": 0.8}})
    z = np.sort(x.astype(np.float64) @ w64["router"].T, axis=1)[:, ::-1]
    clear = np.ones(T, bool) if top == experts else (z[:, top - 1] - z[:, top]) > 1e-4       # the choice itself is clear
    got = host(ffn.forward(dev(x, dtype), None))
    tol = (1e-5 if dtype == torch.float32 else 0.02) * np.abs(ref).max()
    assert clear.mean() > 0.9 and np.abs(got - ref)[clear].max() < tol
    terms, n = ffn.forward_terms(dev(x, dtype), None)
    assert n == top and np.abs(host(terms).reshape(T, top, W).sum(1) - ref)[clear].max() < tol


# ---- whole models ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name,dtype,peaky", [("A", "float32", True), ("A", "bfloat16", False), ("B", "bfloat16", True),
                                              ("B", "float32", True), ("C", "float32", True), ("C", "bfloat16", False)])
def test_every_cutting_gives_the_plain_logits(line, tmp_path, whole_model_tolerance, name, dtype, peaky):
    """Each request whole; its last 32 tokens one by one; batches of unequal lengths that shrink, one batch after another, so that
    slots, pages, rings and states are used again."""
    folder, plain = line(name, dtype, peaky)
    routed_layers(CONFIGS[name][0])
    requests = prompts(name, LENGTHS_B if name == "B" else LENGTHS)
    ref = [plain.logits(t) for t in requests]
    replay = Replay(folder, dtype, tmp_path, max_tokens=576 if name == "B" else 384)
    try:
        worst = run_all_cuttings(replay, requests, ref, dtype)
    finally:
        replay.close()
    print(f"linedra {name} {dtype} peaky={peaky}: largest error {worst:.3g}")


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_the_stream_after_every_layer_and_what_a_left_out_part_would_change(line, name):
    from quicknn_b200.engine import Engine, Model
    folder, plain = line(name, "float32", True)
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
    for suffix, change in ((".canon1", lambda t: t * 0.0), (".sink", lambda t: t - 40.0), (".lam", lambda t: t + 1.0),
                           (".norm1b", lambda t: t - 0.1), (".dwa", lambda t: np.eye(1, len(t), len(t) - 1)[0])):
        w = {k: change(v) if k.endswith(suffix) else v for k, v in plain.w.items()}
        assert np.abs(LP.forward(plain.cfg, w, toks) - ref).max() > 50e-4 * np.abs(ref).max(), suffix


@pytest.mark.parametrize("name,dtype,peaky", [("A", "float32", True), ("B", "float32", True), ("B", "bfloat16", True),
                                              ("C", "float32", True)])
def test_prompts_in_portions_down_to_two_tokens(line, tmp_path, name, dtype, peaky):
    """Steps that continue sequences by several tokens, beside requests that join or sit out."""
    folder, plain = line(name, dtype, peaky)
    routed_layers(CONFIGS[name][0])
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
        step((0, a - 67 - 3), (2, 4), end=[2])   # a portion longer than the windows
        step((0, 3), (1, b - 65), end=[0, 1])
        assert pos == [a, b, 45]
        got = replay.step([("again", requests[0], [a - 1])], end=["again"])      # what they held is free again
        ok, err, tol = near(got, ref[0][a - 1:a], dtype)
        assert ok, (err, tol)
    finally:
        replay.close()


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_through_the_entry_point(line, name):
    """More requests than slots, so that slots, rings and recurrent states are handed out again; decode steps run from CUDA graphs,
    one step ahead of the host, with padding rows; the tokens are the plain implementation's."""
    from quicknn_b200.engine import LLM
    from quicknn_b200.sampling import GenerationOptions
    folder, plain = line(name, "float32", True)
    reqs = prompts(name, [5, 70, 1, 33, 12], seed=3)
    llm = LLM(folder, max_context=256, max_batch=2, dtype="float32")
    res = llm.generate(reqs, GenerationOptions.greedy(12), stop_ids=[])
    for r, p in zip(res, reqs):
        assert r.tokens == plain.greedy(p, 12), f"request {r.index}"
    folder, plain = line(name, "bfloat16", False)
    llm16 = LLM(folder, max_context=256, max_batch=4, dtype="bfloat16")
    for r, p in zip(llm16.generate(reqs, GenerationOptions.greedy(6), stop_ids=[]), reqs):
        seq = list(p)
        for t in r.tokens:                      # bfloat16: every token is at least a near-best one of the plain logits
            row = plain.logits(seq)[-1]
            assert row[t] >= row.max() - 0.15 * (row.max() - row.min())
            seq.append(t)


def test_long_decoding_keeps_states_rings_and_windows(line):
    """150 tokens generated one by one after a short prompt: the windows of 9 and of 1 token and the ring of a page pass over decoded
    tokens, states are carried all the way."""
    from quicknn_b200.engine import LLM
    from quicknn_b200.sampling import GenerationOptions
    folder, plain = line("A", "float32", True)
    p = prompts("A", [3], seed=9)[0]
    llm = LLM(folder, max_context=256, max_batch=1, dtype="float32")
    got = llm.generate([p], GenerationOptions.greedy(150), stop_ids=[])[0].tokens
    seq = p + got
    ref = plain.logits(seq[:-1])
    for i, t in enumerate(got):                 # every generated token is the best one at its place
        row = ref[len(p) - 1 + i]
        assert row[t] >= row.max() - 1e-4 * max(1.0, np.abs(row).max()), f"token {i}"


def test_the_first_tokens_of_a_sequence(line):
    """One to five tokens as prompts, whole and one by one (shorter than the filters, nothing but the sink beside the first key)."""
    from quicknn_b200.engine import Engine, Model
    for name in ("A", "B", "C"):
        folder, plain = line(name, "float32", True)
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


def test_the_command_line_serves_the_design(line, tmp_path):
    import subprocess
    import sys
    from conftest import ROOT

    def run(*argv):
        return subprocess.run([sys.executable, "-m", "quicknn_b200", *argv], cwd=ROOT, capture_output=True, text=True)
    folder, plain = line("A", "float32", True)
    r = run("info", "--model", folder)
    assert r.returncode == 0, r.stderr
    info = json.loads(r.stdout)
    assert info["architecture"] == "Linedra" and info["layers"] == len(LIN_A["layers"])
    p = prompts("A", [9, 4], seed=5)
    r = run("generate", "--model", folder, "--prompt-ids", ";".join(",".join(map(str, q)) for q in p), "--max-new-tokens", "8",
            "--temperature", "0", "--dtype", "float32", "--max-context", "64", "--stop-ids", "")
    assert r.returncode == 0, r.stderr
    got = [json.loads(l) for l in r.stdout.splitlines() if l.strip()]
    assert [g["tokens"] for g in got] == [plain.greedy(q, 8) for q in p]
    cfg = tmp_path / "cfg.json"
    cfg.write_text(json.dumps(LIN_C))
    out = tmp_path / "random_c"
    r = run("random", "--config", str(cfg), "--seed", "3", "--out", str(out), "--dtype", "bfloat16")
    assert r.returncode == 0, r.stderr
    ref = LP.PlainLinedra(str(out))
    toks = prompts("C", [21], seed=6)[0]
    replay = Replay(str(out), "float32", tmp_path / "logits", max_tokens=64)       # bfloat16 weights, widened exactly
    try:
        got = replay.step([("x", toks, range(len(toks)))], end=["x"])
    finally:
        replay.close()
    ok, err, tol = near(got, ref.logits(toks), "float32")
    assert ok, (err, tol)


def test_a_model_at_tensor_core_layer_sizes(tmp_path):
    """Head size 128, latent rows of 256, parts of 128, prompts of 700 tokens over windows of 256: the products run on the tcgen05
    kernels, the routed experts on the grouped product, a batch that continues by portions and single tokens."""
    from quicknn_b200.engine import Engine, Model
    raw = _model(1024, 512, 8.0, 1e-5, 4, 0.7, 30.0, 0.04, [
        _par(_left(4, 2, 128, 128, 0.09, 256), 512, 4, 4, 1.2, 0.9, _moe(256, 8, 2, 3.0)),
        _latent(4, 64, 64, 64, 256, 192, 0.09, 100000.0, _moe(256, 8, 2, 3.0))])
    CONFIGS["T"] = (raw, 11)
    routed_layers(raw)
    folder = make_folder(tmp_path, "T", "bfloat16", False)
    plain = LP.PlainLinedra(folder)
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
    rng = np.random.default_rng(3000 + seed)
    pick = lambda xs: xs[int(rng.integers(len(xs)))]  # noqa: E731
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        experts = int(rng.integers(1, 10))
        mlp = None if rng.random() < 0.25 else _moe(pick([16, 40, 64, 96]), experts, int(rng.integers(1, min(4, experts) + 1)), pick([0.5, 1.5, 7.0]))
        if rng.random() < 0.6:
            kv, blocks = pick([1, 2, 3]), pick([1, 2, 3, 4])
            dim, vdim = pick([8, 16, 20, 24, 32, 64]), pick([8, 16, 24, 32, 64])
            layers.append(_par(_left(kv * int(rng.integers(1, 4)), kv, dim, vdim, float(rng.uniform(0.1, 0.5)),
                                     pick([None, 1, 3, 17, 63, 64, 65, 80, 100])),
                               blocks * pick([8, 12, 16, 40]), blocks, pick([1, 2, 3, 4, 5]), float(rng.uniform(0.3, 1.8)),
                               float(rng.uniform(0.3, 1.8)), mlp))
        else:
            layers.append(_latent(int(rng.integers(1, 6)), pick([8, 16, 20, 32]), pick([2, 6, 8, 16, 32]), pick([8, 20, 24, 32]),
                                  pick([16, 24, 40, 64]), pick([16, 21, 40, 64, 100]), float(rng.uniform(0.1, 0.5)),
                                  pick([100.0, 10000.0, 500000.0]), mlp))
    return _model(int(rng.integers(100, 700)), pick([48, 64, 96, 100, 160, 352]), pick([1.0, 0.5, 9.0]), pick([1e-5, 1e-6]),
                  pick([1, 2, 3, 4, 5]), float(pick([1.0, 0.4, 1.3])), pick([None, 15.0, 50.0]), 0.07, layers)


@pytest.mark.parametrize("seed", range(24))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Prompts of unequal lengths in one step, then tokens one by one, against the plain logits: float32 sharply for every
    configuration, bfloat16 for every other one."""
    from quicknn_b200.engine import Engine, Model
    raw = random_config(seed)
    name = f"R{seed}"
    CONFIGS[name] = (raw, 50 + seed)
    routed_layers(raw)
    lens, extra = [130, 7, 1, 70], 5
    reqs = prompts(name, [n + extra for n in lens], seed=seed)
    for dtype in (("float32", "bfloat16") if seed % 2 == 0 else ("float32",)):
        folder = make_folder(tmp_path, name, dtype, dtype == "float32")
        plain = LP.PlainLinedra(folder)
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
