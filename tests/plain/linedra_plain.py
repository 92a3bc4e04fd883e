"""Plain, slow Linedra: whole sequences, no cache, one function per mechanism, NumPy only, float64.

A decoder whose ``config.json`` lists its layers.  With X_0 the embedded tokens times a constant and x_0 = X_0, layer i does

    y       = x_i + m N1b(mixer(c(N1(x_i))))        c(h)_t = h_t + sum_j w_j h_(t - taps + 1 + j), per channel
    X_(i+1) = y   + m N2b(ff(N2(y)))                 (a layer without a feed-forward: X_(i+1) = y)
    x_(i+1) = sum_(j <= i+1) a_ij X_j                learned numbers a_i, one per earlier result and the embedding

and the logits are cap tanh(E N(x_L) / cap) with E the embedding table.  Norms are RMS norms whose weights are stored around 0.

* mixer ``parallel``: left_scale * left + right_scale * right, both reading the same rows.
  left: grouped-query softmax attention without rotation; scale q.k minus slope_h (i - j); the last ``mask.size`` positions;
  a learned number per head joins the denominator as exp(sink_h); every head times sigmoid((W_g h)_h).
  right: y = gelu(W_y h + b), u = conv(W_x h + b); r and z are sigmoids of block-diagonal products of u;
  a = exp(-8 r softplus(lam)), S_t = a S_(t-1) + sqrt(1 - a^2) z u; out = W_o (S * y).
* mixer ``latent_attention``: queries through a normed latent, keys and values of all heads out of one normed latent row, a
  rotated key part shared by the heads, a sink, a gate per output element.
* feed-forward: routed experts, softmax over the chosen logits, experts with a clamped gate.

It shares no code with the library: its own safetensors reader, its own reading of ``config.json``.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import numpy as np

F = np.float64


def read_safetensors(path: str) -> Dict[str, np.ndarray]:
    with open(path, "rb") as fh:
        (n,) = struct.unpack("<Q", fh.read(8))
        header = json.loads(fh.read(n).decode("utf-8"))
        data = fh.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        b, e = info["data_offsets"]
        raw = data[b:e]
        if info["dtype"] == "BF16":
            arr = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        elif info["dtype"] == "F32":
            arr = np.frombuffer(raw, dtype="<f4")
        elif info["dtype"] == "I32":
            arr = np.frombuffer(raw, dtype="<i4")
        else:
            raise ValueError(f"plain reader: dtype {info['dtype']} of {name}")
        out[name] = arr.reshape(info["shape"]).astype(F)
    return out


# ---- small pieces --------------------------------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(x: np.ndarray, eps: float) -> np.ndarray:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def norm_about_zero(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return rms_unit(x, eps) * (1.0 + weight)


def causal_conv(x: np.ndarray, weight: np.ndarray) -> np.ndarray:
    """Per channel: out_t = sum_j weight[:, j] x_(t - taps + 1 + j), zeros before the first row."""
    n, taps = x.shape[0], weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1]), dtype=F), x], axis=0)
    return sum(padded[j:j + n] * weight[:, j] for j in range(taps))


def depth_average(results: List[np.ndarray], numbers: np.ndarray) -> np.ndarray:
    return sum(float(a) * X for a, X in zip(numbers, results))


# ---- attention ---------------------------------------------------------------------------------------------------

def distance_slopes(heads: int) -> np.ndarray:
    return 2.0 ** (-8.0 * (np.arange(heads, dtype=F) + 1.0) / heads)


def softmax_with_sink(scores: np.ndarray, see: np.ndarray, sink: float) -> np.ndarray:
    """Weights [n, n]: exp(score) over the visible keys' exp(score) plus exp(sink)."""
    s = np.where(see, scores, -np.inf)
    top = np.maximum(s.max(axis=1, keepdims=True), sink)
    e = np.exp(s - top)
    return e / (e.sum(axis=1, keepdims=True) + np.exp(sink - top))


def causal(n: int, window: Optional[int] = None) -> np.ndarray:
    i = np.arange(n)
    d = i[:, None] - i[None, :]
    return (d >= 0) if window is None else (d >= 0) & (d < window)


def window_attention(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict) -> np.ndarray:
    n = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[pre + "q"].T).reshape(n, H, D)
    k = (h @ w[pre + "k"].T).reshape(n, G, D)
    v = (h @ w[pre + "v"].T).reshape(n, G, V)
    see = causal(n, int(m["mask"]["size"]) if m.get("mask") else None)
    i = np.arange(n, dtype=F)
    distance = i[:, None] - i[None, :]
    gate = sigmoid(h @ w[pre + "g"].T)
    heads, slopes = [], distance_slopes(H)
    for hh in range(H):
        g = hh // (H // G)
        score = (q[:, hh] @ k[:, g].T) * float(m["scale"]) - slopes[hh] * distance
        heads.append(softmax_with_sink(score, see, float(w[pre + "sink"][hh])) @ v[:, g] * gate[:, hh:hh + 1])
    return np.concatenate(heads, axis=1) @ w[pre + "o"].T


def rotate_half(x: np.ndarray, base: float, dims: int) -> np.ndarray:
    """x: [tokens, ..., dim]; column i pairs with column i + dims/2 and turns by position * base^(-2i/dims)."""
    half = dims // 2
    f = float(base) ** (-2.0 * np.arange(half, dtype=F) / dims)
    a = np.arange(x.shape[0], dtype=F).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., dims:]], axis=-1)


def latent_attention(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict, eps: float) -> np.ndarray:
    n = h.shape[0]
    H, D, R, V, K = (int(m[x]) for x in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    cq = rms_unit(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]
    q = (cq @ w[pre + "uq"].T).reshape(n, H, D + R)
    kv = h @ w[pre + "dkv"].T
    c = rms_unit(kv[:, :K], eps) * w[pre + "dkv.norm"]
    kr = rotate_half(kv[:, K:], base, dims)
    qr = rotate_half(q[:, :, D:], base, dims)
    k = (c @ w[pre + "uk"].T).reshape(n, H, D)
    v = (c @ w[pre + "uv"].T).reshape(n, H, V)
    see = causal(n)
    heads = []
    for hh in range(H):
        score = (q[:, hh, :D] @ k[:, hh].T + qr[:, hh] @ kr.T) * float(m["scale"])
        heads.append(softmax_with_sink(score, see, float(w[pre + "sink"][hh])) @ v[:, hh])
    return (np.concatenate(heads, axis=1) * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---- the gated linear recurrence ------------------------------------------------------------------------------------

def block_product(u: np.ndarray, weight: np.ndarray, bias: np.ndarray) -> np.ndarray:
    """u cut into equal parts, part b times weight[b] ([out, in]) plus bias[b]."""
    n, B = u.shape[0], weight.shape[0]
    return (np.einsum("nbi,boi->nbo", u.reshape(n, B, -1), weight) + bias).reshape(n, -1)


def recurrence_inputs(u: np.ndarray, w: Dict[str, np.ndarray], pre: str):
    """(a, what is added to the state) per row and channel."""
    r = sigmoid(block_product(u, w[pre + "ra"], w[pre + "ra.b"]))
    z = sigmoid(block_product(u, w[pre + "ri"], w[pre + "ri.b"]))
    log_a = -8.0 * r * softplus(w[pre + "lam"])
    return np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a)) * z * u


def linear_recurrence(a: np.ndarray, b: np.ndarray) -> np.ndarray:
    S, out = np.zeros(a.shape[1], dtype=F), np.zeros_like(a)
    for t in range(a.shape[0]):
        S = a[t] * S + b[t]
        out[t] = S
    return out


def recurrent_block(h: np.ndarray, w: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    y = gelu_tanh(h @ w[pre + "y"].T + w[pre + "y.b"])
    u = causal_conv(h @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"]) + w[pre + "conv.b"]
    a, b = recurrence_inputs(u, w, pre)
    return (linear_recurrence(a, b) * y) @ w[pre + "o"].T


def parallel(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict) -> np.ndarray:
    return (float(m["left_scale"]) * window_attention(h, w, pre + "left.", m["left"])
            + float(m["right_scale"]) * recurrent_block(h, w, pre + "right."))


# ---- routed experts ---------------------------------------------------------------------------------------------

def clamped_expert(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, limit: float) -> np.ndarray:
    g = np.minimum(h @ w[pre + "gate"].T, limit)
    u = np.clip(h @ w[pre + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def route(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, top: int):
    """(chosen experts [n, top], their weights [n, top]): a softmax over the chosen logits alone."""
    z = h @ w[pre + "router"].T
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, chosen, axis=1)
    e = np.exp(zc - zc.max(axis=1, keepdims=True))
    return chosen, e / e.sum(axis=1, keepdims=True)


def routed(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, mlp: dict) -> np.ndarray:
    chosen, weights = route(h, w, pre, int(mlp["router"]["top"]))
    out = np.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        rows, place = np.nonzero(chosen == e)
        if rows.size:
            y = clamped_expert(h[rows], w, f"{pre}e{e}.", float(mlp["expert"]["limit"]))
            out[rows] += weights[rows, place][:, None] * y
    return out


# ---- the model ------------------------------------------------------------------------------------------------

def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, return_layers: bool = False):
    """Logits [tokens, vocab] of one whole sequence; with ``return_layers`` also the stream after every layer."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = w["embed"][np.asarray(tokens, dtype=np.int64)] * float(cfg["embedding"]["scale"])
    results, streams = [x], []
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        h = norm_about_zero(x, w[pre + "norm1"], eps)
        h = h + causal_conv(h, w[pre + "canon1"])
        if layer["type"] == "parallel":
            y = parallel(h, w, pre + "mix.", layer["mixer"])
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, pre + "mix.", layer["mixer"], eps)
        else:
            raise ValueError(f"layer type {layer['type']!r}")
        x = x + mult * norm_about_zero(y, w[pre + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = routed(norm_about_zero(x, w[pre + "norm2"], eps), w, pre + "mlp.", layer["mlp"])
            x = x + mult * norm_about_zero(y, w[pre + "norm2b"], eps)
        results.append(x)
        x = depth_average(results, w[pre + "dwa"])
        streams.append(x.copy())
    logits = norm_about_zero(x, w["final.norm"], eps) @ w["embed"].T
    cap = cfg.get("logit_softcap")
    if cap is not None:
        logits = float(cap) * np.tanh(logits / float(cap))
    return (logits, np.stack(streams)) if return_layers else logits


def load_folder(path: str):
    with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as fh:
        cfg = json.load(fh)
    return cfg, read_safetensors(os.path.join(path, "model.safetensors"))


class PlainLinedra:
    """A model folder read once; whole sequences through ``forward``."""

    def __init__(self, folder: str):
        self.cfg, self.w = load_folder(folder)

    def logits(self, tokens) -> np.ndarray:
        return forward(self.cfg, self.w, tokens)

    def layers(self, tokens) -> np.ndarray:
        return forward(self.cfg, self.w, tokens, return_layers=True)[1]

    def greedy(self, prompt, n: int) -> List[int]:
        seq, out = list(prompt), []
        for _ in range(n):
            t = int(np.argmax(self.logits(seq)[-1]))
            out.append(t)
            seq.append(t)
        return out
