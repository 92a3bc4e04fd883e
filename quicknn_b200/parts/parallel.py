"""Mixers side by side: several mixers read the same input.  Either each output is RMS-normed over the model width with a
plain weight of its own and the mixer's output is their mean,

    y = (1/n) sum_b  rmsnorm(branch_b(x)) * w_b

or, with ``scales`` = {branch: number}, the outputs are summed with fixed numbers,

    y = sum_b  scale_b branch_b(x)

which is two products: the branches' input matrices are stacked (``input_matrix``), every branch works on its columns of the
product's rows, and the branches leave what their output matrices multiply, already scaled, side by side in one row
(``before_output``), the output matrices being stacked along their inner size.

``branches`` maps a name to the branch's ``PartSpec`` (any registered mixer); the branch's parameters are this mixer's
``<name>.<parameter>`` and its weight ``<name>.out``.  The branches share one cache line: at most one of them may keep
keys and values and at most one a fixed-size state, and each sees what it asked for.  The mean is not formed here when
the block that holds the mixer can form it inside its own kernel (``forward_branches``).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..kernels import ops
from .base import MIXERS, CacheNeed, Mixer, StateNeed
from .linear import project, stack_rows
from .spec import PartSpec


@MIXERS.register("parallel")
class ParallelMixer(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.eps = float(p["eps"])
        self.names: List[str] = list(p["branches"])
        if not (1 <= len(self.names) <= 4):
            raise ValueError(f"parallel: one to four branches (got {len(self.names)})")
        self.branches: List[Mixer] = [MIXERS.get(p["branches"][n].kind)(p["branches"][n]) for n in self.names]
        if sum(b.cache_need() is not None for b in self.branches) > 1:
            raise ValueError("parallel: at most one branch may keep keys and values")
        if sum(b.state_need() is not None for b in self.branches) > 1:
            raise ValueError("parallel: at most one branch may keep a state")
        self.out_weights: List[torch.Tensor] = []
        scales = p.get("scales")
        self.scales: Optional[List[float]] = None if scales is None else [float(scales[n]) for n in self.names]
        self.w_in: Optional[torch.Tensor] = None         # with scales: the branches' input matrices one below the other
        self.w_o: Optional[torch.Tensor] = None          # and their output matrices side by side
        self.in_cols: List[int] = []
        if self.scales is not None and not all(hasattr(b, "before_output") for b in self.branches):
            raise ValueError("parallel: branches with fixed scales offer their rows before the output product")

    @classmethod
    def param_shapes(cls, spec: PartSpec) -> Dict[str, Tuple[Tuple[int, ...], str]]:
        p = spec.params
        out: Dict[str, Tuple[Tuple[int, ...], str]] = {}
        for name, sub in p["branches"].items():
            for k, v in MIXERS.get(sub.kind).param_shapes(sub).items():
                out[f"{name}.{k}"] = v
            if p.get("scales") is None:
                out[f"{name}.out"] = ((int(p["hidden_size"]),), cls.PARAM_ROLE_SCALE)
        return out

    def load(self, tensors, compute_dtype, device) -> None:
        self.out_weights = []
        for name, b in zip(self.names, self.branches):
            pre = name + "."
            b.load({k[len(pre):]: v for k, v in tensors.items() if k.startswith(pre) and k != pre + "out"},
                   compute_dtype, device)
            if self.scales is None:
                self.out_weights.append(tensors[pre + "out"].contiguous())
        if self.scales is not None:
            ws = [b.w_o for b in self.branches]
            wide = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
            self.w_o = torch.cat([w.to(wide) for w in ws], dim=1).contiguous()
            ins = [b.input_matrix() for b in self.branches]
            self.in_cols = [sum(w.shape[0] for w in ins[:i]) for i in range(len(ins))]
            pad = torch.zeros(((-sum(w.shape[0] for w in ins)) % 8, self.hidden), dtype=ins[0].dtype, device=ins[0].device)
            self.w_in = stack_rows(ins + [pad])          # rows of whole 16-byte pieces
            for b in self.branches:                      # the branches' own matrices are ranges of these from here on
                b.w_o = None
                b.release_inputs()

    def weight_bytes(self) -> int:
        own = self.out_weights + ([self.w_in, self.w_o] if self.w_o is not None else [])
        return sum(b.weight_bytes() for b in self.branches) + sum(w.numel() * w.element_size() for w in own)

    def cache_need(self) -> Optional[CacheNeed]:
        for b in self.branches:
            if b.cache_need() is not None:
                return b.cache_need()
        return None

    def state_need(self) -> Optional[StateNeed]:
        for b in self.branches:
            if b.state_need() is not None:
                return b.state_need()
        return None

    def scratch_need(self, step) -> int:
        return max(b.scratch_need(step) for b in self.branches)

    def schedule(self, step) -> tuple:
        return tuple(b.schedule(step) for b in self.branches)

    def forward_branches(self, x: torch.Tensor, step, line) -> List[torch.Tensor]:
        """The branches' outputs, not yet normed."""
        return [b.forward(x, step, line) for b in self.branches]

    def forward(self, x: torch.Tensor, step, line) -> torch.Tensor:
        if self.scales is not None:
            p = project(x, self.w_in)
            rows = torch.empty((x.shape[0], self.w_o.shape[1]), dtype=x.dtype, device=x.device)
            col = 0
            for b, s, c in zip(self.branches, self.scales, self.in_cols):
                b.before_output(p, c, step, line, s, rows, col)
                col += b.out_width
            return project(rows, self.w_o)
        return ops.mean_rmsnorm(self.forward_branches(x, step, line), self.out_weights, self.eps, x.dtype)
