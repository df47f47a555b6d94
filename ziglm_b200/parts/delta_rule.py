"""The gated delta rule: a matrix-valued state per head that is decayed, corrected towards a value and read, token by
token, behind a short causal convolution.

For the rows h the mixer reads, H heads over G heads of q and k, query/key size D, value size V, a convolution of K taps:
    q, k, v <- silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))      per channel, zeros before the sequence's start
    q, k    <- q / |q| * D^(-1/2),  k / |k|                                 per head, |x| = sqrt(sum x^2 + 1e-6)
    beta    = sigmoid(W_b h)                                                one write strength a head
    g       = exp(-exp(A_log) softplus(a + dt_bias))                        ``decay`` "head": a = W_a h, one a head;
                                                                            "channel": a = W_a2 (W_a1 h), one a key channel
    S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q   S [D, V] per head, zero at the start; head
                                                                            h reads the q and k of head h // (H / G)
    out = W_o (o / rms(o) * w * act(gate))                                  per head over V, w shared by the heads;
                                                                            ``gate`` "silu": W_g h, "sigmoid": W_g2 (W_g1 h)
The rank of a product of low rank is an option (``decay_rank``, ``gate_rank``; None: the file's, any).  A sequence
carries the convolution's last inputs [K, C] and S, both float32 (two ``StateNeed``).  Decays, write strengths, unit
vectors, the state and the products that enter it are float32 in both precisions; in bfloat16 the projections are, but for
the last product before a decay or a write strength, whose sums stay float32.
A step of one token a sequence runs everything between the first product and W_o in one kernel (in steps of many sequences
the small products before a, b and the gate are taken before it).
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import kernels
from ..config.spec import MixerSpec
from .base import FreeDim, KVNeed, LayerIO, ParamDecl, Part, StateNeed, register_mixer
from .linear import Linear


# Sequences up to which a step of one token a sequence leaves the small products before decays, write strengths and the gate
# to the kernel of the recurrence: its blocks then read their head's rows of the weights once for every sequence.
FUSED_SEQUENCES = 16


def _up8(n: int) -> int:
    return -(-n // 8) * 8


def _stack_rows(ws, dtype: torch.dtype):
    """The matrices one below the other, each from a multiple of eight rows on (zero rows between), and where they start."""
    at, blocks, starts = 0, [], []
    for w in ws:
        starts.append(at)
        n = _up8(w.shape[0])
        blocks.append(torch.cat([w.to(dtype), w.new_zeros((n - w.shape[0],) + tuple(w.shape[1:]), dtype=dtype)], dim=0))
        at += n
    return torch.cat(blocks, dim=0), starts


class GatedDeltaRule(Part):
    can_overwrite = True

    def __init__(self, spec: MixerSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        o = spec.options
        self.n_heads, self.n_kv, self.dim = spec.n_heads, spec.n_kv_heads, spec.head_dim
        self.value_dim = int(o.get("value_dim", spec.head_dim))
        self.taps = int(o["taps"])
        if self.n_heads <= 0 or self.n_kv <= 0 or self.n_heads % self.n_kv:
            raise ValueError(f"gated_delta_rule: {self.n_heads} heads cannot share {self.n_kv} heads of q and k")
        if min(self.dim, self.value_dim, self.taps) <= 0:
            raise ValueError("gated_delta_rule: key size, value size and taps must be positive")
        if self.dim > 512:
            raise ValueError(f"gated_delta_rule: keys of {self.dim} elements are not supported (at most 512)")
        self.decay = o.get("decay", "head")
        if self.decay not in ("head", "channel"):
            raise ValueError(f"gated_delta_rule: decay {self.decay!r} is not known (head, channel)")
        self.gate = o.get("gate")
        if self.gate not in (None, "silu", "sigmoid"):
            raise ValueError(f"gated_delta_rule: output gate {self.gate!r} is not known (silu, sigmoid)")
        self.low_rank_gate = self.gate is not None and bool(o.get("gate_low_rank", self.gate == "sigmoid"))
        self.eps = float(o["norm_eps"])
        self.channels = 2 * self.n_kv * self.dim + self.n_heads * self.value_dim
        self.proj: Optional[Linear] = None      # [q; k; v; then g, or the first factors a1 and g1]
        self.rates: Optional[Linear] = None     # [b; a] with float32 sums
        self.a2: Optional[Linear] = None
        self.g2: Optional[Linear] = None
        self.o: Optional[Linear] = None
        self.a_at = self.g_at = self.a_rank = self.g_rank = 0
        self.conv_w = self.rate = self.dt_bias = self.norm_w = self.norm_rows = None

    @classmethod
    def declare(cls, spec: MixerSpec) -> Dict[str, ParamDecl]:
        H, G, D, d, o = spec.n_heads, spec.n_kv_heads, spec.head_dim, spec.width, spec.options
        V, K = int(o.get("value_dim", D)), int(o["taps"])
        p = {"q.weight": ParamDecl((G * D, d)), "k.weight": ParamDecl((G * D, d)), "v.weight": ParamDecl((H * V, d)),
             "q.conv": ParamDecl((G * D, K)), "k.conv": ParamDecl((G * D, K)), "v.conv": ParamDecl((H * V, K)),
             "b.weight": ParamDecl((H, d)), "A_log": ParamDecl((H,)), "norm.weight": ParamDecl((V,), init="ones"),
             "o.weight": ParamDecl((d, H * V))}

        def rank(key: str) -> int:
            return FreeDim(D) if o.get(key) is None else int(o[key])

        if o.get("decay", "head") == "head":
            p["a.weight"], p["dt_bias"] = ParamDecl((H, d)), ParamDecl((H,))
        else:
            r = rank("decay_rank")
            p["a1.weight"], p["a2.weight"], p["dt_bias"] = ParamDecl((r, d)), ParamDecl((H * D, r)), ParamDecl((H * D,))
        gate = o.get("gate")
        if gate is not None and o.get("gate_low_rank", gate == "sigmoid"):
            r = rank("gate_rank")
            p["g1.weight"], p["g2.weight"] = ParamDecl((r, d)), ParamDecl((H * V, r))
        elif gate is not None:
            p["g.weight"] = ParamDecl((H * V, d))
        return p

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        def wide(ws) -> torch.dtype:
            return torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype

        def second(name: str, rank: int) -> Linear:
            w = tensors[name]
            if w.shape[1] != rank:
                raise ValueError(f"gated_delta_rule: {name} takes {w.shape[1]} numbers, the product before it gives {rank}")
            return Linear(torch.cat([w, w.new_zeros(w.shape[0], _up8(rank) - rank)], dim=1))

        # q, k and v lie one behind the other: what the convolution runs over
        ws = [torch.cat([tensors[f"{n}.weight"].to(wide([tensors[f"{m}.weight"] for m in "qkv"])) for n in "qkv"], dim=0)]
        low = self.decay == "channel"
        if low:
            ws.append(tensors["a1.weight"])
        if self.gate is not None:
            ws.append(tensors["g1.weight"] if self.low_rank_gate else tensors["g.weight"])
        weight, starts = _stack_rows(ws, wide(ws))
        self.proj = Linear(weight)
        if low:
            self.a_at, self.a_rank = starts[1], int(tensors["a1.weight"].shape[0])
            self.a2 = second("a2.weight", self.a_rank)
        if self.gate is not None:
            self.g_at = starts[-1]
            if self.low_rank_gate:
                self.g_rank = int(tensors["g1.weight"].shape[0])
                self.g2 = second("g2.weight", self.g_rank)
        bs = [tensors["b.weight"]] + ([] if low else [tensors["a.weight"]])
        rates = torch.cat([b.to(wide(bs)) for b in bs], dim=0)
        self.rates = Linear(torch.cat([rates, rates.new_zeros(_up8(rates.shape[0]) - rates.shape[0], rates.shape[1])], dim=0))
        self.o = Linear(tensors["o.weight"])
        self.conv_w = torch.cat([tensors[f"{n}.conv"].float() for n in "qkv"], dim=0).t().contiguous()
        self.rate = torch.exp(tensors["A_log"].float()).contiguous()
        self.dt_bias = tensors["dt_bias"].float().contiguous()
        self.norm_w = tensors["norm.weight"].float().contiguous()
        self.norm_rows = self.norm_w.repeat(self.n_heads).contiguous()

    def kernel_libraries(self) -> Tuple[str, ...]:
        libs = ("delta_rule", "elementwise")
        for lin in (self.proj, self.rates, self.a2, self.g2, self.o):
            if lin is not None:
                libs += lin.libraries(self.dtype)
        return libs

    def cache_needs(self) -> Optional[KVNeed]:
        return None

    def state_needs(self) -> Tuple[StateNeed, ...]:
        return (StateNeed((self.taps, self.channels), torch.float32),
                StateNeed((self.n_heads, self.value_dim, kernels.delta_state_size(self.dim)), torch.float32))

    def forward(self, step, io: LayerIO, h: torch.Tensor, residual: torch.Tensor, accumulate: bool = True):
        T, H, V = residual.shape[0], self.n_heads, self.value_dim
        ring, state = io.state
        proj = step.ws.buf("delta_proj", (T, self.proj.out_features), self.dtype)
        self.proj(h, proj)
        out = step.ws.buf("delta_out", (T, H * V), self.dtype)
        a_cols = slice(self.a_at, self.a_at + _up8(self.a_rank))
        g_cols = slice(self.g_at, self.g_at + _up8(self.g_rank))
        fused = (step.single_token and T <= FUSED_SEQUENCES and h.shape[1] % 8 == 0 and h.stride(0) % 8 == 0
                 and all(lin is None or lin.weight.dtype == self.dtype for lin in (self.rates, self.a2, self.g2)))
        args = (proj, self.conv_w, ring, H, self.n_kv, self.dim, V)
        if fused:
            low_gate = (self.g2.weight, self.g_at) if self.low_rank_gate else None
            gate = proj[:, self.g_at:self.g_at + H * V] if self.gate is not None and not self.low_rank_gate else None
            kernels.delta_rule_decode(
                *args, None, None, self.rate, self.dt_bias, state, step, self.norm_w, self.eps, gate, self.gate, out, h=h,
                w_b=self.rates.weight[:H], w_a=self.rates.weight[H:2 * H] if self.decay == "head" else None,
                a2=(self.a2.weight, self.a_at) if self.decay == "channel" else None, g2=low_gate)
            self.o(out, residual, accumulate=accumulate)
            return None
        rates = step.ws.buf("delta_rates", (T, self.rates.out_features), torch.float32)
        self.rates(h, rates)
        if self.decay == "head":
            a = rates[:, H:2 * H]
        else:
            a = step.ws.buf("delta_a", (T, H * self.dim), torch.float32)
            self.a2(proj[:, a_cols], a)
        gate = None
        if self.low_rank_gate:
            gate = step.ws.buf("delta_gate", (T, H * V), self.dtype)
            self.g2(proj[:, g_cols], gate)
        elif self.gate is not None:
            gate = proj[:, self.g_at:self.g_at + H * V]
        args += (a, rates[:, :H], self.rate, self.dt_bias, state, step)
        if step.single_token:
            kernels.delta_rule_decode(*args, self.norm_w, self.eps, gate, self.gate, out)
        else:
            mixed = step.ws.buf("delta_mixed", (T, H * V), torch.float32)
            kernels.delta_rule(*args, mixed)
            kernels.head_norm_gate(mixed, self.norm_rows, gate, out, H, self.eps, self.gate)
        self.o(out, residual, accumulate=accumulate)
        return None


register_mixer("gated_delta_rule", GatedDeltaRule)
