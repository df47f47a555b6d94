"""Residual streams (hyper-connections): a token is carried by s copies of the residual instead of one.

Around a sublayer with learned numbers in [s], out [s] and mix [s, s] (indexed [from, to]):
    u = sum_a in[a] x_a;   y = sublayer(norm(u));   x_b <- sum_a mix[a, b] x_a + out[b] y     (all b from the old x)
which replaces norm, sublayer and residual sum.  ``StreamNorm`` is the norm of such a weighted sum (and, without learned
numbers, of the plain sum of the streams: the norm before the head); ``HyperBlock`` the arrangement of a layer.  The
residual rows are [T, s * width] float32; the kernel that spreads a sublayer's output over the streams also makes the rows
of the sublayer that follows, here or in the next block, so the streams are read and written once a sublayer.
A mixer that offers ``forward_branches`` (side-by-side mixers whose outputs are normed and summed) hands its outputs over
unsummed, and the same kernel norms and sums them.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import kernels
from ..config.spec import LayerSpec, NormSpec
from .base import (KVNeed, LayerIO, ParamDecl, Part, feed_forward_class, mixer_class, norm_class, register_block,
                   register_norm)


class StreamNorm(Part):
    """norm(sum_a in[a] x_a) * weight.  Options: ``streams``; ``learned`` (True: the tensor ``in``; False: every stream
    counts once)."""

    def __init__(self, spec: NormSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        self.width, self.eps = spec.width, float(spec.eps)
        self.streams = int(spec.options["streams"])
        self.learned = bool(spec.options.get("learned", True))
        self.weight: Optional[torch.Tensor] = None
        self.gather: Optional[torch.Tensor] = None

    @classmethod
    def declare(cls, spec: NormSpec) -> Dict[str, ParamDecl]:
        p = {"weight": ParamDecl((spec.width,), init="ones")}
        if spec.options.get("learned", True):
            p["in"] = ParamDecl((int(spec.options["streams"]),))
        return p

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors["weight"].float().contiguous()
        self.gather = tensors["in"].float().contiguous() if self.learned else None

    def kernel_libraries(self) -> Tuple[str, ...]:
        return ("streams",)

    def forward(self, step, x: torch.Tensor, out: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None, n_rows: Optional[int] = None,
                name: str = "norm_out") -> torch.Tensor:
        n = n_rows if n_rows is not None else (rows.numel() if rows is not None else x.shape[0])
        if out is None:
            out = step.ws.buf(name, (n, self.width), self.dtype)
        kernels.stream_norm(x, self.streams, self.gather, self.weight, self.eps, out, rows=rows)
        return out


class HyperBlock(Part):
    """A layer over residual streams.  ``LayerSpec.options``: ``streams``; ``mixer_norm`` and ``ffn_norm`` are norms of kind
    "stream_norm"; the tensors ``mixer_hc.out``, ``mixer_hc.mix`` (and ``ffn_hc.*``) spread a sublayer's output.  A layer
    whose spec has no feed-forward ends after the mixer."""

    def __init__(self, spec: LayerSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        self.streams = int(spec.options["streams"])
        self.parts: Dict[str, Part] = {prefix: klass(sub, dtype, device) for prefix, klass, sub in self._children(spec)}
        self.mixer_norm = self.parts["mixer_norm."]
        self.mixer = self.parts["mixer."]
        self.ffn_norm = self.parts.get("ffn_norm.")
        self.ffn = self.parts.get("ffn.")
        self.coef: Dict[str, torch.Tensor] = {}

    @classmethod
    def _children(cls, spec: LayerSpec):
        out = [("mixer_norm.", norm_class(spec.mixer_norm.kind), spec.mixer_norm),
               ("mixer.", mixer_class(spec.mixer.kind), spec.mixer)]
        if spec.ffn is not None:
            out += [("ffn_norm.", norm_class(spec.ffn_norm.kind), spec.ffn_norm),
                    ("ffn.", feed_forward_class(spec.ffn.kind), spec.ffn)]
        for _, klass, sub in out[0::2]:
            if klass is not StreamNorm or int(sub.options["streams"]) != int(spec.options["streams"]):
                raise ValueError("hyper: a sublayer's norm must be a stream_norm over the block's streams")
        return out

    @classmethod
    def declare(cls, spec: LayerSpec) -> Dict[str, ParamDecl]:
        out: Dict[str, ParamDecl] = {}
        for prefix, klass, sub in cls._children(spec):
            for name, decl in klass.declare(sub).items():
                out[prefix + name] = decl
        s = int(spec.options["streams"])
        for which in ("mixer_hc.",) + (("ffn_hc.",) if spec.ffn is not None else ()):
            out[which + "out"] = ParamDecl((s,))
            out[which + "mix"] = ParamDecl((s, s))
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        for prefix, part in self.parts.items():
            part.bind({k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)})
        for which in ("mixer_hc.",) + (("ffn_hc.",) if self.ffn is not None else ()):
            self.coef[which] = torch.cat([tensors[which + "mix"].float().reshape(-1), tensors[which + "out"].float()]).contiguous()

    def kernel_libraries(self) -> Tuple[str, ...]:
        libs: Tuple[str, ...] = ("streams",)
        for part in self.parts.values():
            libs += part.kernel_libraries()
        return libs

    def cache_needs(self) -> Optional[KVNeed]:
        return self.mixer.cache_needs()

    def state_needs(self):
        return self.mixer.state_needs()

    def accepts_normed_input(self) -> bool:
        """The block before may hand over the rows this block's mixer reads (``h_in``)."""
        return True

    def _spread(self, step, which: str, branches, norms, x: torch.Tensor, nxt, name: str) -> Optional[torch.Tensor]:
        """The new streams from the old ones and the sublayer's output; with ``nxt`` (the StreamNorm of the sublayer that
        follows) also its rows, which are returned."""
        h = None
        if nxt is not None:
            h = step.ws.buf(name, (x.shape[0], nxt.width), self.dtype)
        weights, eps, factor = norms if norms is not None else (None, 0.0, 1.0)
        kernels.stream_mix(x, self.streams, self.coef[which], branches, weights, eps, factor,
                           nxt=None if nxt is None else (nxt.gather, nxt.weight, nxt.eps, h))
        return h

    def _run(self, part, step, io, h: torch.Tensor) -> torch.Tensor:
        branch = step.ws.buf("branch", (h.shape[0], self.mixer_norm.width), torch.float32)
        args = (step, h, branch) if io is None else (step, io, h, branch)
        if part.can_overwrite:
            part.forward(*args, accumulate=False)
        else:
            branch.zero_()
            part.forward(*args)
        return branch

    def forward(self, step, io: LayerIO, x: torch.Tensor, h_in=None, next_norm=None):
        """``h_in``: the rows the mixer reads, left by the block before.  ``next_norm``: the first norm of the block after;
        if it is a StreamNorm over the same streams the result is its rows, else None."""
        h = h_in if isinstance(h_in, torch.Tensor) else self.mixer_norm.forward(step, x)
        feeds = next_norm if isinstance(next_norm, StreamNorm) and next_norm.learned else None
        if hasattr(self.mixer, "forward_branches") and self.mixer.norms is not None:
            branches, norms = self.mixer.forward_branches(step, io, h), self.mixer.norms
        else:
            branches, norms = [self._run(self.mixer, step, io, h)], None
        if self.ffn is None:
            return self._spread(step, "mixer_hc.", branches, norms, x, feeds, "norm_out_next")
        h = self._spread(step, "mixer_hc.", branches, norms, x, self.ffn_norm, "norm_out_ffn")
        branch = self._run(self.ffn, step, None, h)
        return self._spread(step, "ffn_hc.", [branch], None, x, feeds, "norm_out_next")


register_norm("stream_norm", StreamNorm)
register_block("hyper", HyperBlock)
