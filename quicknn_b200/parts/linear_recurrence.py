"""The recurrent block around a real-gated linear recurrence (``rglru``; De et al., "Griffin: Mixing Gated Linear Recurrences
with Local Attention for Efficient Language Models"): one number of state per channel.

    y = gelu(W_y x + b_y)                     u = conv(W_x x + b_x) + b_c      a causal convolution per channel, ``conv`` taps
    r = sigmoid(R_b u_b + r_b),  i = sigmoid(I_b u_b + i_b)                    u cut into ``blocks`` equal parts u_b
    log a = -8 r softplus(lam),  a = exp(log a)
    S_t = a S_(t-1) + sqrt(1 - a^2) i u       out = W_o (S * y)

A slot's state is float32 [conv + 1, width]: a ring of the convolution's last inputs, then S.  The decay 8 softplus(lam) is
formed once, when the model is loaded (float64, rounded to float32); the gates' products have float32 results; from
there to S everything is float32.  y and u are one stacked product, r and i of a part are one matrix.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..kernels import ops
from .base import MIXERS, CacheNeed, Mixer, StateNeed
from .linear import project, stack_rows
from .spec import PartSpec

DECAY = 8.0
STEP_MAX_ROWS = 64             # decode rows up to which the whole step is one kernel (it forms u once per 32 channels of a part)


@MIXERS.register("rglru")
class RealGatedRecurrence(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.width = int(p["width"])
        self.blocks = int(p["blocks"])
        self.taps = int(p["conv"])
        if self.blocks < 1 or self.width % self.blocks:
            raise ValueError(f"rglru: {self.blocks} parts do not divide {self.width} channels")
        if self.taps < 1:
            raise ValueError(f"rglru: at least one tap (got {self.taps})")
        self.part = self.width // self.blocks
        self.out_width = self.width
        self.w_in: Optional[torch.Tensor] = None         # y | x rows
        self.w_gates: Optional[torch.Tensor] = None      # [blocks, 2 * part, part]: r rows, then i rows
        self.w_o: Optional[torch.Tensor] = None

    @classmethod
    def param_shapes(cls, spec: PartSpec) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        p = spec.params
        W, D, B = int(p["hidden_size"]), int(p["width"]), int(p["blocks"])
        d = D // B
        M, N = cls.PARAM_ROLE_MATRIX, cls.PARAM_ROLE_NORM
        return {"y": ((D, W), M), "y_bias": ((D,), N), "x": ((D, W), M), "x_bias": ((D,), N),
                "conv": ((D, int(p["conv"])), cls.PARAM_ROLE_SCALE), "conv_bias": ((D,), N),
                "r": ((B, d, d), M), "r_bias": ((B, d), N), "i": ((B, d, d), M), "i_bias": ((B, d), N),
                "lam": ((D,), N), "o": ((W, D), M)}

    def load(self, tensors, compute_dtype, device) -> None:
        self.w_in = stack_rows([tensors["y"], tensors["x"]])
        wide = torch.float32 if torch.float32 in (tensors["r"].dtype, tensors["i"].dtype) else tensors["r"].dtype
        self.w_gates = torch.cat([tensors["r"].to(wide), tensors["i"].to(wide)], dim=1).contiguous()
        self.y_bias, self.x_bias = tensors["y_bias"].contiguous(), tensors["x_bias"].contiguous()
        self.conv, self.conv_bias = tensors["conv"].contiguous(), tensors["conv_bias"].contiguous()
        self.r_bias = tensors["r_bias"].to(torch.float32).reshape(-1).contiguous()
        self.i_bias = tensors["i_bias"].to(torch.float32).reshape(-1).contiguous()
        self.decay = (DECAY * torch.nn.functional.softplus(tensors["lam"].to(torch.float64))).to(torch.float32).contiguous()
        self.w_o = tensors["o"].contiguous()

    def weight_bytes(self) -> int:
        ws = (self.w_in, self.w_gates, self.w_o, self.y_bias, self.x_bias, self.conv, self.conv_bias, self.r_bias, self.i_bias,
              self.decay)
        return sum(w.numel() * w.element_size() for w in ws if w is not None)

    def cache_need(self) -> Optional[CacheNeed]:
        return None

    def state_need(self) -> Optional[StateNeed]:
        return StateNeed((self.taps + 1, self.width), "float32")

    def input_matrix(self) -> torch.Tensor:
        """What multiplies the input, for a mixer that stacks it with its other branches'."""
        return self.w_in

    def release_inputs(self) -> None:
        """Forget the input matrix: it lives on in the stacked one."""
        self.w_in = None

    def before_output(self, p: torch.Tensor, col0: int, step, line, scale: float, out: torch.Tensor, out_col0: int) -> torch.Tensor:
        """scale * S * y: what the output matrix multiplies, into the columns ``out_col0 ..`` of ``out``.  p: rows whose columns
        from ``col0`` on are the input times ``input_matrix`` (y | x)."""
        D = self.width
        decode = step.mode == "decode"
        if decode and step.n_seqs <= STEP_MAX_ROWS and ops.recurrent_step(
                p, col0, col0 + D, self.x_bias, self.y_bias, self.conv, self.conv_bias, self.w_gates, self.r_bias, self.i_bias,
                self.decay, line.state, step.tok_pos, step.slots, scale, out, out_col0):
            return out
        row0, lens = (None, None) if decode else (step.seq_row0, step.seq_len)
        longest = 1 if decode else step.max_q_len
        u = ops.causal_conv(p, self.conv, line.state, row0, lens, step.tok_pos, step.slots, step.n_seqs, longest, col0=col0 + D,
                            x_bias=self.x_bias, out_bias=self.conv_bias)
        return ops.linear_recurrence(u, self.w_gates, self.r_bias, self.i_bias, self.decay, line.state, self.taps * D, row0, lens,
                                     step.slots, step.n_seqs, longest, y=p, y_col0=col0, y_bias=self.y_bias, scale=scale,
                                     out=out, out_col0=out_col0)

    def forward(self, x: torch.Tensor, step, line) -> torch.Tensor:
        out = torch.empty((x.shape[0], self.width), dtype=x.dtype, device=x.device)
        return project(self.before_output(project(x, self.w_in), 0, step, line, 1.0, out, 0), self.w_o)
