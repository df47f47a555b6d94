"""Several mixers side by side: all read the same rows and their outputs are summed.

``MixerSpec.options["parts"]`` lists (prefix, MixerSpec) pairs; a part's tensors are declared under its prefix, and a
factor on a part's output is that part's own option (it rides where the part rounds its heads before its output
projection, so the sum itself is plain).  With ``norm_eps`` every part's output is divided by its root mean square over
the model width and multiplied by a weight of the part's own (``<prefix>out_norm.weight``) before the sum, and the sum is
multiplied by ``factor``: ``forward_branches`` then leaves the outputs side by side for a block that norms and sums them
in a kernel of its own, ``forward`` does it here.  At most one part may keep keys and values: the place of the schedule
owns one set of pages, which goes to the part that asked.  States per sequence go to the parts that asked for them.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Dict, List, Optional, Tuple

import torch

from .. import kernels
from ..config.spec import MixerSpec
from .base import KVNeed, LayerIO, ParamDecl, Part, StateNeed, mixer_class, register_mixer


class SideBySide(Part):
    can_overwrite = True

    def __init__(self, spec: MixerSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        parts = spec.options.get("parts")
        if not parts:
            raise ValueError("side_by_side: the spec must list the mixers that run side by side")
        self.parts: List[Tuple[str, Part]] = [(prefix, mixer_class(sub.kind)(sub, dtype, device)) for prefix, sub in parts]
        if sum(1 for _, p in self.parts if p.cache_needs() is not None) > 1:
            raise ValueError("side_by_side: only one of the mixers may keep keys and values")
        # per part: which of the place's states are its own, and whether it finds them in a tuple
        self.state_of: List[Optional[Tuple[int, int, bool]]] = []
        self.all_states: Tuple[StateNeed, ...] = ()
        for _, p in self.parts:
            need = p.state_needs()
            if need is None:
                self.state_of.append(None)
                continue
            several = isinstance(need, tuple)
            need = need if several else (need,)
            self.state_of.append((len(self.all_states), len(need), several))
            self.all_states += need
        eps = spec.options.get("norm_eps")
        self.norm_eps = None if eps is None else float(eps)
        self.factor = float(spec.options.get("factor", 1.0))
        if self.norm_eps is None and self.factor != 1.0:
            raise ValueError("side_by_side: a factor on the sum goes with the norms of the outputs")
        if self.norm_eps is not None and len(self.parts) != 2:
            raise ValueError("side_by_side: normed outputs are summed in pairs")
        self.norms = None            # (weights, eps, factor), once the weights are bound

    @classmethod
    def declare(cls, spec: MixerSpec) -> Dict[str, ParamDecl]:
        out: Dict[str, ParamDecl] = {}
        for prefix, sub in spec.options["parts"]:
            for name, decl in mixer_class(sub.kind).declare(sub).items():
                out[prefix + name] = decl
            if spec.options.get("norm_eps") is not None:
                out[prefix + "out_norm.weight"] = ParamDecl((spec.width,), init="ones")
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        for prefix, part in self.parts:
            part.bind({k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)})
        if self.norm_eps is not None:
            self.norms = ([tensors[prefix + "out_norm.weight"].float().contiguous() for prefix, _ in self.parts],
                          self.norm_eps, self.factor)
            self._one_stream = torch.ones(2, dtype=torch.float32, device=self.norms[0][0].device)

    def kernel_libraries(self) -> Tuple[str, ...]:
        libs: Tuple[str, ...] = () if self.norm_eps is None else ("streams",)
        for _, part in self.parts:
            libs += part.kernel_libraries()
        return libs

    def cache_needs(self) -> Optional[KVNeed]:
        for _, part in self.parts:
            need = part.cache_needs()
            if need is not None:
                return need
        return None

    def state_needs(self):
        if len(self.all_states) == 1 and not any(o is not None and o[2] for o in self.state_of):
            return self.all_states[0]
        return self.all_states or None

    def _io(self, i: int, io: LayerIO) -> LayerIO:
        """The place's storage as part ``i`` sees it."""
        own = self.state_of[i]
        if own is None or not isinstance(io.state, tuple):
            return io
        at, n, several = own
        return replace(io, state=io.state[at:at + n] if several else io.state[at])

    def forward_branches(self, step, io: LayerIO, h: torch.Tensor) -> List[torch.Tensor]:
        """Every part's output in a float32 buffer of its own, not yet normed."""
        branches = []
        for i, (_, part) in enumerate(self.parts):
            branch = step.ws.buf(f"side_branch{i}", (h.shape[0], self.spec.width), torch.float32)
            if part.can_overwrite:
                part.forward(step, self._io(i, io), h, branch, accumulate=False)
            else:
                branch.zero_()
                part.forward(step, self._io(i, io), h, branch)
            branches.append(branch)
        return branches

    def forward(self, step, io: LayerIO, h: torch.Tensor, residual: torch.Tensor, accumulate: bool = True):
        if self.norms is not None:
            branches = self.forward_branches(step, io, h)
            if not accumulate:
                residual.zero_()
            # one stream, kept as it is, plus the normed sum
            kernels.stream_mix(residual, 1, self._one_stream, branches, *self.norms)
            return None
        for i, (_, part) in enumerate(self.parts):
            if i == 0 and not accumulate:
                if part.can_overwrite:
                    part.forward(step, self._io(i, io), h, residual, accumulate=False)
                    continue
                residual.zero_()
            part.forward(step, self._io(i, io), h, residual)
        return None


register_mixer("side_by_side", SideBySide)
