"""Small parts that run once per step outside the layers, or between two places of the schedule.

``add_row``   x[t, :] += table[row, :] for every token of the step: a learned vector added to the residual
              stream at a fixed place (the start of a pass through a repeated run of layers).  Options:
              ``rows`` and ``width`` (the table's shape), ``row``; ``add_embedding``: the residual as the first layer
              found it is added before the row, x[t, :] <- (x[t, :] + embedded[t, :]) + table[row, :].
``token_pairs``  the embedding of a token plus a row of a second table that its pair with the token before chooses: row
              (before * mul_prev + token * mul_cur) mod buckets, and the last row, number ``buckets``, for a sequence's first
              token.  The last token of a sequence is a state of it.  Options: ``buckets``, ``width``, ``mul_prev``, ``mul_cur``.
``scale``     logits *= factor.  Option: ``factor``.
``soft_cap``  logits <- cap tanh(logits / cap), in float32.  Option: ``cap``.
``rmsnorm``   x <- x / sqrt(mean(x^2) + eps) * (w + offset) over every row, in place and in float32: a norm of the
              embedded tokens before the first layer.  Options: ``width``, ``eps``, ``unit_offset`` (the stored weight
              is the gain minus one).
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import kernels
from ..config.spec import HookSpec
from .base import LayerIO, ParamDecl, Part, StateNeed, register_hook


class AddRow(Part):
    def __init__(self, spec: HookSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        self.row_index = int(spec.options["row"])
        if not 0 <= self.row_index < int(spec.options["rows"]):
            raise ValueError(f"add_row: row {self.row_index} is outside the table of {spec.options['rows']} rows")
        self.reads_kept = ("embedding",) if spec.options.get("add_embedding") else ()
        self.row: Optional[torch.Tensor] = None

    @classmethod
    def declare(cls, spec: HookSpec) -> Dict[str, ParamDecl]:
        return {"table": ParamDecl((int(spec.options["rows"]), int(spec.options["width"])))}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.row = tensors["table"][self.row_index].contiguous()

    def kernel_libraries(self) -> Tuple[str, ...]:
        return ("elementwise",)

    def forward(self, step, x: torch.Tensor) -> None:
        kernels.add_row(x, self.row, rows=step.kept["embedding"] if self.reads_kept else None)


class TokenPairs(Part):
    def __init__(self, spec: HookSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        o = spec.options
        self.mul_prev, self.mul_cur = int(o["mul_prev"]), int(o["mul_cur"])
        if int(o["buckets"]) < 1 or min(self.mul_prev, self.mul_cur) < 0:
            raise ValueError("token_pairs: at least one bucket and factors that are not negative are needed")
        self.table: Optional[torch.Tensor] = None

    @classmethod
    def declare(cls, spec: HookSpec) -> Dict[str, ParamDecl]:
        return {"table": ParamDecl((int(spec.options["buckets"]) + 1, int(spec.options["width"])))}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors["table"].contiguous()

    def kernel_libraries(self) -> Tuple[str, ...]:
        return ("elementwise",)

    def state_needs(self) -> StateNeed:
        return StateNeed((1,), torch.int32)

    def embed(self, step, io: LayerIO, table: torch.Tensor, scale: float, x: torch.Tensor,
              kept: Optional[torch.Tensor]) -> None:
        kernels.embed_pairs(table, self.table, io.state, self.mul_prev, self.mul_cur, step, x, kept, scale)


class Scale(Part):
    def __init__(self, spec: HookSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        self.factor = float(spec.options["factor"])

    def kernel_libraries(self) -> Tuple[str, ...]:
        return ("elementwise",)

    def forward(self, step, x: torch.Tensor) -> None:
        kernels.scale_(x, self.factor)


class SoftCap(Part):
    def __init__(self, spec: HookSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        self.cap = float(spec.options["cap"])
        if not self.cap > 0.0:
            raise ValueError(f"soft_cap: the cap must be positive, found {self.cap}")

    def kernel_libraries(self) -> Tuple[str, ...]:
        return ("elementwise",)

    def forward(self, step, x: torch.Tensor) -> None:
        kernels.soft_cap_(x, self.cap)


class NormRows(Part):
    def __init__(self, spec: HookSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        self.width = int(spec.options["width"])
        self.eps = float(spec.options["eps"])
        self.weight_offset = 1.0 if spec.options.get("unit_offset") else 0.0
        self.weight: Optional[torch.Tensor] = None

    @classmethod
    def declare(cls, spec: HookSpec) -> Dict[str, ParamDecl]:
        return {"weight": ParamDecl((int(spec.options["width"]),), init="zeros" if spec.options.get("unit_offset") else "ones")}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors["weight"].contiguous()

    def kernel_libraries(self) -> Tuple[str, ...]:
        return ("elementwise",)

    def forward(self, step, x: torch.Tensor) -> None:
        if x.shape[-1] != self.width:
            raise ValueError(f"rmsnorm hook: rows of {x.shape[-1]} elements, the norm is over {self.width}")
        # every element is read and written by the same thread, after the row's sum is known: in place is safe
        kernels.rmsnorm_rows(x, self.weight, x, self.eps, weight_offset=self.weight_offset)


register_hook("add_row", AddRow)
register_hook("token_pairs", TokenPairs)
register_hook("rmsnorm", NormRows)
register_hook("scale", Scale)
register_hook("soft_cap", SoftCap)
