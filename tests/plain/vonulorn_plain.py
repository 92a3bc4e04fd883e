"""Plain, slow Vonulorn: whole sequences, no cache, one function per mechanism, NumPy only, float64.

A decoder whose ``config.json`` lists its layers.  With x the embedded tokens, layer i does

    x = x + m mixer(N1(x));   x = x + m ff(N2(x))          (a layer without a feed-forward stops after the first)

and the logits are W_head N(x).  Norms are RMS norms with plain weights, m is one constant.

* mixer ``delta``: q, k, v pass a causal convolution per channel and silu; q and k become unit vectors; with a decay g and a
  step size b per head the state S [dim, vdim] follows the gated delta rule (Yang, Kautz, Hatamizadeh, "Gated Delta Networks:
  Improving Mamba2 with Delta Rule"): decay, read what the key finds, write the difference to the value, read with the query.
* mixer ``attention``: differential attention (Ye et al., "Differential Transformer"): two softmax maps per head over the same
  values, one subtracted from the other; queries grow with the logarithm of the position; scores are soft-capped.
* mixer ``latent_attention``: queries through a normed latent, keys and values of all heads out of one normed latent row, a
  rotated key part shared by the heads (neighbouring columns turn together), a sink.
* feed-forward: down(gelu(gate) * up).

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
        else:
            raise ValueError(f"plain reader: dtype {info['dtype']} of {name}")
        out[name] = arr.reshape(info["shape"]).astype(F)
    return out


# ---- small pieces --------------------------------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(x: np.ndarray, eps: float) -> np.ndarray:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def unit_vectors(x: np.ndarray) -> np.ndarray:
    """x / sqrt(sum(x^2) + 1e-6) over the last axis."""
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def causal_conv(x: np.ndarray, weight: np.ndarray) -> np.ndarray:
    """Per channel: out_t = sum_j weight[:, j] x_(t - taps + 1 + j), zeros before the first row."""
    n, taps = x.shape[0], weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1]), dtype=F), x], axis=0)
    return sum(padded[j:j + n] * weight[:, j] for j in range(taps))


def causal(n: int) -> np.ndarray:
    return np.tril(np.ones((n, n), dtype=bool))


def softmax_rows(scores: np.ndarray, see: np.ndarray, sink: Optional[float] = None) -> np.ndarray:
    """exp(score) of the visible keys over their sum (plus exp(sink))."""
    s = np.where(see, scores, -np.inf)
    top = s.max(axis=1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    den = e.sum(axis=1, keepdims=True)
    return e / (den if sink is None else den + np.exp(sink - top))


# ---- the gated delta rule --------------------------------------------------------------------------------------

def delta_rule(q: np.ndarray, k: np.ndarray, v: np.ndarray, beta: np.ndarray, g: np.ndarray, S: Optional[np.ndarray] = None):
    """One head.  q, k: [n, dim], v: [n, vdim], beta, g: [n].  Returns (read-outs [n, vdim], the state at the end)."""
    S = np.zeros((q.shape[1], v.shape[1]), dtype=F) if S is None else S.copy()
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out, S


def delta_inputs(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict):
    """(q, k: [n, kv_heads, dim], v: [n, heads, vdim], beta, g: [n, heads])."""
    n = h.shape[0]
    H, G, D, V = (int(m[x]) for x in ("heads", "kv_heads", "dim", "vdim"))
    q, k, v = (silu(causal_conv(h @ w[pre + t].T, w[pre + t + ".conv"])) for t in ("q", "k", "v"))
    q = unit_vectors(q.reshape(n, G, D)) / math.sqrt(D)
    k = unit_vectors(k.reshape(n, G, D))
    beta = sigmoid(h @ w[pre + "b"].T)
    g = np.exp(-np.exp(w[pre + "A_log"]) * softplus(h @ w[pre + "a"].T + w[pre + "dt_bias"]))
    return q, k, v.reshape(n, H, V), beta, g


def delta(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict, eps: float) -> np.ndarray:
    H, G = int(m["heads"]), int(m["kv_heads"])
    q, k, v, beta, g = delta_inputs(h, w, pre, m)
    heads = [delta_rule(q[:, hh // (H // G)], k[:, hh // (H // G)], v[:, hh], beta[:, hh], g[:, hh])[0] for hh in range(H)]
    o = np.concatenate([rms_unit(o, eps) * w[pre + "norm"] for o in heads], axis=1)
    return (o * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---- differential attention -------------------------------------------------------------------------------------

def query_temperature(n: int, t: Optional[dict]) -> np.ndarray:
    """One factor per position: 1 + coef ln(floor((p + 1) / every) + 1)."""
    p = np.arange(n, dtype=F)
    if t is None:
        return np.ones(n)
    return 1.0 + float(t["coef"]) * np.log(np.floor((p + 1.0) / float(t["every"])) + 1.0)


def differential_lambda(w: Dict[str, np.ndarray], pre: str, diff: float) -> float:
    return float(np.exp((w[pre + "lq1"] * w[pre + "lk1"]).sum()) - np.exp((w[pre + "lq2"] * w[pre + "lk2"]).sum()) + diff)


def softmax_map(q: np.ndarray, k: np.ndarray, scale: float, cap: Optional[float]) -> np.ndarray:
    """Attention weights [n, n] of one head and one map."""
    score = (q @ k.T) * scale
    if cap is not None:
        score = cap * np.tanh(score / cap)
    return softmax_rows(score, causal(q.shape[0]))


def differential_attention(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict, eps: float) -> np.ndarray:
    n = h.shape[0]
    H, G, D, V = (int(m[x]) for x in ("heads", "kv_heads", "dim", "vdim"))
    diff, scale = float(m["diff"]), float(m["scale"])
    cap = None if m.get("softcap") is None else float(m["softcap"])
    q = (h @ w[pre + "q"].T).reshape(n, H, 2, D) * query_temperature(n, m.get("q_temp"))[:, None, None, None]
    k = (h @ w[pre + "k"].T).reshape(n, G, 2, D)
    v = (h @ w[pre + "v"].T).reshape(n, G, V)
    lam = differential_lambda(w, pre, diff)
    heads = []
    for hh in range(H):
        g = hh // (H // G)
        a1, a2 = (softmax_map(q[:, hh, j], k[:, g, j], scale, cap) @ v[:, g] for j in range(2))
        heads.append(rms_unit(a1 - lam * a2, eps) * (1.0 - diff))
    return np.concatenate(heads, axis=1) @ w[pre + "o"].T


# ---- latent attention -------------------------------------------------------------------------------------------

def rotate_neighbours(x: np.ndarray, base: float, dims: int) -> np.ndarray:
    """x: [tokens, ..., dim]; columns 2i and 2i + 1 turn together by position * base^(-2i/dims)."""
    f = float(base) ** (-2.0 * np.arange(dims // 2, dtype=F) / dims)
    a = np.arange(x.shape[0], dtype=F).reshape((-1,) + (1,) * (x.ndim - 1)) * f
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return out


def latent_attention(h: np.ndarray, w: Dict[str, np.ndarray], pre: str, m: dict, eps: float) -> np.ndarray:
    n = h.shape[0]
    H, D, R, V, K = (int(m[x]) for x in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    cq = rms_unit(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]
    q = (cq @ w[pre + "uq"].T).reshape(n, H, D + R)
    kv = h @ w[pre + "dkv"].T
    c = rms_unit(kv[:, :K], eps) * w[pre + "dkv.norm"]
    kr = rotate_neighbours(kv[:, K:], base, dims)
    qr = rotate_neighbours(q[:, :, D:], base, dims)
    k = (c @ w[pre + "uk"].T).reshape(n, H, D)
    v = (c @ w[pre + "uv"].T).reshape(n, H, V)
    heads = []
    for hh in range(H):
        score = (q[:, hh, :D] @ k[:, hh].T + qr[:, hh] @ kr.T) * float(m["scale"])
        heads.append(softmax_rows(score, causal(n), float(w[pre + "sink"][hh])) @ v[:, hh])
    return np.concatenate(heads, axis=1) @ w[pre + "o"].T


# ---- the model ------------------------------------------------------------------------------------------------

MIXERS = {"delta": delta, "attention": differential_attention, "latent_attention": latent_attention}


def gated_mlp(h: np.ndarray, w: Dict[str, np.ndarray], pre: str) -> np.ndarray:
    return (gelu_tanh(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, return_layers: bool = False):
    """Logits [tokens, vocab] of one whole sequence; with ``return_layers`` also the stream after every layer."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = w["embed"][np.asarray(tokens, dtype=np.int64)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        h = rms_unit(x, eps) * w[pre + "norm1"]
        x = x + mult * MIXERS[layer["type"]](h, w, pre + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + mult * gated_mlp(rms_unit(x, eps) * w[pre + "norm2"], w, pre + "mlp.")
        streams.append(x.copy())
    logits = (rms_unit(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, np.stack(streams)) if return_layers else logits


def load_folder(path: str):
    with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as fh:
        cfg = json.load(fh)
    return cfg, read_safetensors(os.path.join(path, "model.safetensors"))


class PlainVonulorn:
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
