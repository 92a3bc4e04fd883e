"""The gated delta rule (``delta_rule``; Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"): a
matrix state per value head that decays and is corrected towards the value at the current key.

    q = silu(conv(W_q x)),  k = silu(conv(W_k x))   (kv_heads x dim),    v = silu(conv(W_v x))   (heads x vdim)
    q, k per head / sqrt(sum of squares + 1e-6);    q also * dim^(-1/2)
    beta = sigmoid(W_b x),   g = exp(-exp(A) softplus(W_a x + dt))       one of each per value head
    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q      S: [dim, vdim]
    y = W_o ( rmsnorm_per_head(o) * silu(W_g x) )

conv is a causal convolution over time per channel with ``conv`` taps.  Value head h reads query/key head h // (heads / kv_heads).
A slot's state is float32: a ring of the convolution's last inputs [taps, 2 kv_heads dim + heads vdim], then S
[heads, dim, vdim].  q, k, v and the gate are one stacked product; beta's and g's logits are float32 products.  Unit vectors, gates,
the state and the norm are float32: what the convolution leaves is stored in the activations' type, with the factors that make
unit vectors of it beside it, applied where the rows are read.  Prompts and portions walk in chunks of 16 rows
(``ops.delta_scan``); a decode step is one kernel between the two products (``ops.delta_step``).
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..kernels import ops
from .base import MIXERS, CacheNeed, Mixer, StateNeed
from .linear import project, stack_rows
from .spec import PartSpec

UNIT_EPS = 1e-6


@MIXERS.register("delta_rule")
class GatedDeltaRule(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.n_heads = int(p["n_heads"])
        self.n_kv = int(p["n_kv_heads"])
        self.dim = int(p["dim"])
        self.vdim = int(p["vdim"])
        self.taps = int(p["conv"])
        self.eps = float(p["eps"])
        if self.n_kv < 1 or self.n_heads % self.n_kv:
            raise ValueError(f"delta_rule: {self.n_kv} query/key heads do not divide {self.n_heads} heads")
        if self.dim > 256:
            raise ValueError(f"delta_rule: at most 256 key channels per head (got {self.dim})")
        if self.taps < 1:
            raise ValueError(f"delta_rule: at least one tap (got {self.taps})")
        self.channels = 2 * self.n_kv * self.dim + self.n_heads * self.vdim
        self.w_in: Optional[torch.Tensor] = None         # q | k | v | gate rows
        self.w_ba: Optional[torch.Tensor] = None         # beta's rows, then g's
        self.w_o: Optional[torch.Tensor] = None

    @classmethod
    def param_shapes(cls, spec: PartSpec) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        p = spec.params
        W, H, G, d, vd, taps = (int(p[n]) for n in ("hidden_size", "n_heads", "n_kv_heads", "dim", "vdim", "conv"))
        M, N, S = cls.PARAM_ROLE_MATRIX, cls.PARAM_ROLE_NORM, cls.PARAM_ROLE_SCALE
        return {"q": ((G * d, W), M), "q_conv": ((G * d, taps), S), "k": ((G * d, W), M), "k_conv": ((G * d, taps), S),
                "v": ((H * vd, W), M), "v_conv": ((H * vd, taps), S), "b": ((H, W), M), "a": ((H, W), M), "A_log": ((H,), N),
                "dt_bias": ((H,), N), "norm": ((vd,), S), "gate": ((H * vd, W), M), "o": ((W, H * vd), M)}

    def load(self, tensors, compute_dtype, device) -> None:
        self.w_in = stack_rows([tensors["q"], tensors["k"], tensors["v"], tensors["gate"]])
        self.conv = stack_rows([tensors["q_conv"], tensors["k_conv"], tensors["v_conv"]])
        self.w_ba = stack_rows([tensors["b"], tensors["a"]])
        self.rate = torch.exp(tensors["A_log"].to(torch.float64)).to(torch.float32).contiguous()
        self.bias = tensors["dt_bias"].to(torch.float32).contiguous()
        self.norm = tensors["norm"].contiguous()
        self.w_o = tensors["o"].contiguous()

    def weight_bytes(self) -> int:
        ws = (self.w_in, self.conv, self.w_ba, self.rate, self.bias, self.norm, self.w_o)
        return sum(w.numel() * w.element_size() for w in ws)

    def cache_need(self) -> Optional[CacheNeed]:
        return None

    def state_need(self) -> Optional[StateNeed]:
        ring = (self.taps * self.channels + 3) // 4 * 4          # S starts on 16 bytes
        return StateNeed((ring + self.n_heads * self.dim * self.vdim,), "float32")

    @property
    def _s_offset(self) -> int:
        return (self.taps * self.channels + 3) // 4 * 4

    def _gates(self, x: torch.Tensor) -> torch.Tensor:
        """Logits of beta | g, float32."""
        w = self.w_ba
        return ops.block_linear(x if x.dtype == w.dtype else ops.cast(x, w.dtype), w.unsqueeze(0), out_dtype=torch.float32)

    def forward(self, x: torch.Tensor, step, line) -> torch.Tensor:
        H, G, d, vd, C = self.n_heads, self.n_kv, self.dim, self.vdim, self.channels
        scale = float(d) ** -0.5
        p = project(x, self.w_in)                                         # q | k | v | gate
        decode = step.mode == "decode"
        if decode:
            y = ops.delta_step(p, x, self.w_ba, self.conv, self.rate, self.bias, self.norm, self.eps, UNIT_EPS, scale, line.state,
                               self._s_offset, step.tok_pos, step.slots, H, G, d, vd)
            if y is not None:
                return project(y, self.w_o)
        row0, lens = (None, None) if decode else (step.seq_row0, step.seq_len)
        longest = 1 if decode else step.max_q_len
        rows, inv = ops.causal_conv(p, self.conv, line.state, row0, lens, step.tok_pos, step.slots, step.n_seqs, longest,
                                    activation="silu", unit_heads=(2 * G, d, UNIT_EPS))
        o = ops.delta_scan(rows, inv, self._gates(x), self.rate, self.bias, scale, line.state, self._s_offset, row0, lens, step.slots,
                           step.n_seqs, longest, H, G, d, vd)
        y = ops.head_norm_gate(o, vd, H, vd, self.eps, p, C, "silu", weight=self.norm)
        return project(y, self.w_o)
