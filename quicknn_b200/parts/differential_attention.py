"""Differential attention (``differential_attention``; Ye et al., "Differential Transformer"): two softmax maps per head over the
same values, one subtracted from the other.

    q = W_q x  (heads x 2 x dim),   k = W_k x  (kv_heads x 2 x dim),   v = W_v x  (kv_heads x vdim)
    a_j = softmax(cap tanh(scale q_j K_j^T / cap)) V                    j = 1, 2
    o = a_1 - lambda a_2,   o / rms(o) * (1 - diff),   y = W_o [o_1 .. o_H]
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff                     one number per layer

The attention itself is the library's grouped-query attention: a key head keeps both maps' keys side by side (2 dim columns) and
map j of a head is a query head of its own with zeros in the other map's columns, so its score meets its own map's keys only and
keys and values are cached once (``ops.map_prep``).  Heads are carried at a size that the tensor-core kernels take (64, 128, 256)
where 2 dim and vdim fit one.  One kernel subtracts, norms and scales (``ops.map_difference``).

Options: ``softcap`` (None: none), ``window``, ``query_temperature`` = {"coef", "every"}: queries at position p are multiplied by
1 + coef ln(floor((p + 1) / every) + 1).  There is no rotation.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..kernels import ops
from .attention import AttentionMixer
from .base import MIXERS
from .latent_attention import carried_size
from .linear import project, stack_rows
from .spec import PartSpec

MAPS = 2


@MIXERS.register("differential_attention")
class DifferentialAttention(AttentionMixer):
    def __init__(self, spec: PartSpec):
        p = spec.params
        self.real_heads = int(p["n_heads"])
        self.dim = int(p["dim"])
        self.vdim = int(p["vdim"])
        self.diff = float(p["diff"])
        self.eps = float(p["eps"])
        t = p.get("query_temperature")
        self.temp = (0.0, 1.0) if t is None else (float(t["coef"]), float(t["every"]))
        D = carried_size(max(MAPS * self.dim, self.vdim))
        super().__init__(PartSpec("attention", {
            "hidden_size": int(p["hidden_size"]), "n_heads": MAPS * self.real_heads, "n_kv_heads": int(p["n_kv_heads"]),
            "head_dim": D, "scale": float(p["scale"]), "softcap": p.get("softcap"), "window": p.get("window"),
            "position": PartSpec("none", {"head_dim": D})}))
        self.spec = spec
        if self.real_heads % self.n_kv:
            raise ValueError(f"{self.n_kv} kv heads do not divide {self.real_heads} heads")
        self.lam = 0.0

    @classmethod
    def param_shapes(cls, spec: PartSpec) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        p = spec.params
        W, H, G, d, vd = (int(p[n]) for n in ("hidden_size", "n_heads", "n_kv_heads", "dim", "vdim"))
        M, N = cls.PARAM_ROLE_MATRIX, cls.PARAM_ROLE_NORM
        out = {"q": ((H * MAPS * d, W), M), "k": ((G * MAPS * d, W), M), "v": ((G * vd, W), M), "o": ((W, H * vd), M)}
        out.update({n: ((d,), N) for n in ("lq1", "lk1", "lq2", "lk2")})
        return out

    def load(self, tensors, compute_dtype, device) -> None:
        self.w_qkv = stack_rows([tensors["q"], tensors["k"], tensors["v"]])
        self.w_o = tensors["o"].contiguous()
        # one number per layer: float64 on the host, rounded once
        l = {n: tensors[n].detach().to("cpu", torch.float64) for n in ("lq1", "lk1", "lq2", "lk2")}
        self.lam = float(torch.exp((l["lq1"] * l["lk1"]).sum()) - torch.exp((l["lq2"] * l["lk2"]).sum()) + self.diff)
        why = (ops.attention_refusal(compute_dtype, self.n_heads, self.n_kv, self.head_dim)
               or ops.linear_refusal(self.w_qkv.dtype, self.hidden))
        if why:
            raise ValueError(f"differential attention mixer: {why}")
        dev = torch.device(device)
        sms = torch.cuda.get_device_properties(dev).multi_processor_count if dev.type == "cuda" else 148
        self._resident = sms * max(1, min(8, 512 // max(1, self.head_dim)))

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_qkv, self.w_o))

    def forward(self, x: torch.Tensor, step, line) -> torch.Tensor:
        decode = step.mode == "decode"
        p = project(x, self.w_qkv)
        # packed with keys and values for every step but a decode step, whose attention reads the cache; a step that continues
        # sequences appends after its attention (``attend``)
        rows = ops.map_prep(p, self.real_heads, self.n_kv, MAPS, self.dim, self.vdim, self.head_dim, step.tok_pos, step.tok_slot, line,
                            bool(line.writes and step.mode != "extend"), not decode, self.temp[0], self.temp[1])
        a = self.attend(rows, step, line)                                 # [T, heads * 2 * carried size]
        return project(ops.map_difference(a, self.real_heads, self.vdim, self.lam, self.eps, 1.0 - self.diff), self.w_o)
