"""A plain, slow statement of the Lilulix decoder in PyTorch on the CPU: the oracle of the tests.

One function per mechanism, written from the design's equations and sharing no code with the library's product
path.  ``dtype`` float32 computes everything in float32 (float64 with ``wide=True``); bfloat16 rounds where the
library may: the operands and results of the projections and the activations next to them, while positions,
angles, scores, softmax, norms and the residual stream stay float32.

Notation: d model width, H query heads, G key/value heads, D query/key size, R rotated dimensions, V value size,
C the size of a latent, B the number of buckets of the table of token pairs, T tokens of one sequence.
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Mapping, Optional

import torch


class Plain:
    """How numbers are held: ``act`` is the type of projections' inputs and outputs, ``acc`` the type of
    everything the design computes in 32-bit (float64 stands in for it when a tighter oracle is wanted)."""

    def __init__(self, dtype: torch.dtype = torch.float32, wide: bool = False):
        self.act = dtype
        self.acc = torch.float64 if wide else torch.float32

    def round(self, x: torch.Tensor) -> torch.Tensor:
        return x if self.act == torch.float32 else x.to(self.act).to(self.acc)

    def linear(self, x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
        """y = W x (+ b): operands rounded to ``act``, summed in ``acc``, result rounded to ``act``."""
        y = self.round(x) @ self.round(w).t()
        if b is not None:
            y = y + self.round(b)
        return self.round(y)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.to(x.dtype)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def pair_rows(tokens: List[int], previous: Optional[int], bigram: Mapping[str, int]) -> List[int]:
    """The row of the pair table for every token: (previous * a + token * b) mod B, and row B for a token that has
    no token before it.  ``previous``: the token before the first of these (None: they start the sequence)."""
    B, a, b = int(bigram["buckets"]), int(bigram["mul_prev"]), int(bigram["mul_cur"])
    rows = []
    for t in tokens:
        rows.append(B if previous is None else (previous * a + t * b) % B)
        previous = t
    return rows


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, base: float) -> torch.Tensor:
    """x: [T, heads, R]; dimension i is turned together with i + R/2 by the angle position * base^(-2i/R)."""
    R = x.shape[-1]
    freq = torch.tensor([float(base) ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float64)
    # the angle is formed in 32-bit from a 32-bit frequency, as position * frequency
    ang = (positions.to(torch.float32)[:, None] * freq.to(torch.float32)[None, :]).to(x.dtype)
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :R // 2], x[..., R // 2:]
    return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


def causal(query_pos: torch.Tensor, n_keys: int) -> torch.Tensor:
    return torch.arange(n_keys)[None, :] <= query_pos[:, None]


def softmax_with_sink(s: torch.Tensor, seen: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum over the seen keys of exp(s_j)), row by row; ``sink`` is one number."""
    s = s.masked_fill(~seen, float("-inf"))
    m = torch.maximum(s.max(dim=-1, keepdim=True).values, sink.reshape(1, 1).to(s.dtype))
    e = torch.exp(s - m)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink.to(s.dtype) - m))


def distance_slopes(heads: int) -> List[float]:
    """2^(-8 (h + 1) / H) for every head h."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def _keep(past: Optional[Dict[str, torch.Tensor]], name: str, new: torch.Tensor) -> torch.Tensor:
    """All rows of ``name`` so far: what ``past`` holds, then ``new`` (and ``past`` is brought up to date)."""
    if past is None:
        return new
    if name in past:
        new = torch.cat([past[name], new], dim=0)
    past[name] = new
    return new


def latent_attention(p: Plain, h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping[str, Any], eps: float,
                     past: Optional[Dict[str, torch.Tensor]], first_position: int) -> torch.Tensor:
    """Keys and values made from a normed latent c; one rotated key part shared by all heads; a learned number a head
    in the softmax's denominator; the concatenated heads times sigmoid(W_g h)."""
    T = h.shape[0]
    H, D, R, V, C = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    base = float(m["rot"]["base"])
    pos = torch.arange(first_position, first_position + T)
    q = p.linear(h, w["q"]).view(T, H, D + R)
    q_plain, q_rot = q[..., :D], p.round(rotate_halves(q[..., D:], pos, base))
    down = p.linear(h, w["dkv"])
    c = p.round(rms_norm(down[:, :C], w["dkv.norm"], eps))
    k_rot = p.round(rotate_halves(down[:, None, C:], pos, base)[:, 0, :])
    c, k_rot = _keep(past, "c", c), _keep(past, "k_rot", k_rot)
    n = c.shape[0]
    k_plain = p.linear(c, w["uk"]).view(n, H, D)
    v = p.linear(c, w["uv"]).view(n, H, V)
    seen = causal(pos, n)
    out = torch.zeros(T, H, V, dtype=p.acc)
    for head in range(H):
        s = (q_plain[:, head] @ k_plain[:, head].t() + q_rot[:, head] @ k_rot.t()) * float(m["scale"])
        out[:, head] = softmax_with_sink(s, seen, w["sink"][head]) @ v[:, head]
    return out.reshape(T, H * V) * torch.sigmoid(p.linear(h, w["g"]))


def biased_attention(p: Plain, h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping[str, Any], eps: float,
                     past: Optional[Dict[str, torch.Tensor]], first_position: int) -> torch.Tensor:
    """Grouped-query attention whose values are the projected keys, before their norm; q and k normed a head; no
    rotation, a bias by distance on the scores, one more 1 in the softmax's denominator."""
    T = h.shape[0]
    H, G, D = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = p.linear(h, w["q"], w["q.b"]).view(T, H, D)
    k = p.linear(h, w["k"], w["k.b"]).view(T, G, D)
    v = k
    q = p.round(rms_norm(q, w["q.norm"], eps))
    k = p.round(rms_norm(k, w["k.norm"], eps))
    k, v = _keep(past, "k", k), _keep(past, "v", v)
    pos = torch.arange(first_position, first_position + T)
    n = k.shape[0]
    seen = causal(pos, n)
    distance = (pos[:, None] - torch.arange(n)[None, :]).to(p.acc)
    out = torch.zeros(T, H, D, dtype=p.acc)
    for head, slope in enumerate(distance_slopes(H)):
        g = head // (H // G)
        s = (q[:, head] @ k[:, g].t()) * float(m["scale"]) - slope * distance
        out[:, head] = softmax_with_sink(s, seen, torch.zeros(())) @ v[:, g]
    return out.reshape(T, H * D)


def dense_ff(p: Plain, h: torch.Tensor, w: Mapping[str, torch.Tensor]) -> torch.Tensor:
    return p.linear(p.round(gelu_tanh(p.linear(h, w["gate"])) * p.linear(h, w["up"])), w["down"])


def _sub(tensors: Mapping[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


class PlainLilulix:
    """The whole model over one sequence at a time, with keys, values, latents and the last token kept between calls."""

    def __init__(self, config: Mapping[str, Any], tensors: Mapping[str, torch.Tensor],
                 dtype: torch.dtype = torch.float32, wide: bool = False):
        self.c = config
        self.p = Plain(dtype, wide)
        self.w = {k: v.to(self.p.acc) for k, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])

    def runs(self) -> List[tuple]:
        """(layer, pass number at the first layer of a pass through the repeated run, else None) in running order."""
        n, loop = len(self.c["layers"]), self.c.get("loop")
        if not loop:
            return [(i, None) for i in range(n)]
        a, b = int(loop["start"]), int(loop["stop"])
        order = [(i, None) for i in range(a)]
        for t in range(int(loop["times"])):
            order += [(i, t if i == a else None) for i in range(a, b)]
        return order + [(i, None) for i in range(b, n)]

    def new_state(self) -> Dict[str, Any]:
        return {"last": None, "runs": [{} for _ in self.runs()]}

    def forward(self, tokens: List[int], state: Optional[Dict[str, Any]] = None, first_position: int = 0,
                layers_out: Optional[list] = None) -> torch.Tensor:
        """Logits [T, vocab] of the given tokens, which follow ``first_position`` tokens held in ``state``."""
        c, p, w, eps = self.c, self.p, self.w, self.eps
        rows = pair_rows(tokens, None if state is None else state["last"], c["embedding"]["bigram"])
        if state is not None:
            state["last"] = tokens[-1]
        x = w["embed"][torch.tensor(tokens)] + w["bigram"][torch.tensor(rows)]
        embedded = x
        for place, (i, t) in enumerate(self.runs()):
            if t is not None:
                if t > 0:
                    x = x + embedded
                x = x + w["loop.step"][t]
            layer, lw = c["layers"][i], _sub(w, f"l{i}.")
            h = rms_norm(x, lw["norm1"], eps)
            mixer = {"latent_attention": latent_attention, "attention": biased_attention}[layer["type"]]
            mw = _sub(lw, "mix.")
            y = p.linear(mixer(p, h, mw, layer["mixer"], eps, None if state is None else state["runs"][place],
                               first_position), mw["o"])
            if layer.get("mlp") is not None:
                y = y + dense_ff(p, h, _sub(lw, "mlp."))
            x = x + y
            if layers_out is not None:
                layers_out.append(x.clone())
        h = rms_norm(x, w["final.norm"], eps)
        return (p.round(h) @ p.round(w["embed"]).t()).to(torch.float32)
