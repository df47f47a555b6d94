"""A plain, slow statement of the Mopilorn decoder in PyTorch on the CPU: the oracle of the tests.

One function per mechanism, written from the design's equations and sharing no code with the library's product
path.  ``dtype`` float32 computes everything in float32 (float64 with ``wide=True``); bfloat16 rounds where the
library may: the operands and results of the projections, the short convolutions of the attention and the activations
between the products of a feed-forward, while positions, angles, scores, softmax, norms, decays, write strengths, unit
vectors, recurrent states and the residual streams stay float32.

The design.  A token is carried by s residual streams x_1 .. x_s, all equal to its embedding at first.  A layer has a
mixer and (or not) a feed-forward; around each of them
    u = sum_a in[a] x_a,    y = sublayer(norm(u)),    x_b <- sum_a mix[a, b] x_a + out[b] y
with learned numbers in, out and mix of the sublayer; behind the last layer the streams are summed, normed and
multiplied by the head, and the logits z become c tanh(z / c).  Mixers: ``parallel`` (a windowed grouped-query
attention with a short convolution on q, k and v and rotated adjacent pairs, beside a gated delta rule with one decay
a head; half the sum of the two normed outputs) and ``channel_delta`` (a gated delta rule with one decay a key channel,
made by a product of low rank).  The feed-forward is a dense gated one with silu.

Notation: H heads, G heads of q and k (of k and v in the attention), D query/key size, V value size, R rotated
dimensions, K taps, T tokens of one sequence, S [D, V] a head's state.
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

    def linear(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """y = W x: operands rounded to ``act``, summed in ``acc``, result rounded to ``act``."""
        return self.round(self.round(x) @ self.round(w).t())

    def linear_wide(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        """The same product with the sums left in ``acc``."""
        return self.round(x) @ self.round(w).t()


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_plain(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_unit(x, eps) * w.to(x.dtype)


def unit_vector(x: torch.Tensor) -> torch.Tensor:
    """x / sqrt(sum(x^2) + 1e-6) over the last dimension."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def soft_cap(z: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return z if cap is None else cap * torch.tanh(z / cap)


def frequencies(rot: Mapping[str, Any]) -> List[float]:
    """One angle per position for each pair, stretched by wavelength where the configuration says so: short waves keep
    their frequency, long ones are divided by the factor, those between are blended."""
    R, base = int(rot["dims"]), float(rot["base"])
    out = []
    sc = rot.get("scaling")
    for i in range(R // 2):
        f = base ** (-2.0 * i / R)
        if sc:
            factor, lo, hi, n0 = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > n0 / lo:
                f = f / factor
            elif wave >= n0 / hi:
                share = (n0 / wave - lo) / (hi - lo)
                f = (1.0 - share) * f / factor + share * f
        out.append(f)
    return out


def rotate_adjacent(x: torch.Tensor, positions: torch.Tensor, rot: Mapping[str, Any]) -> torch.Tensor:
    """x: [T, heads, D]; of every head's first R dimensions, 2i turns together with 2i + 1 by position * f_i."""
    R = int(rot["dims"])
    f = torch.tensor(frequencies(rot), dtype=x.dtype)
    a = positions.to(x.dtype)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., 0:R:2], x[..., 1:R:2]
    y = x.clone()
    y[..., 0:R:2] = u * c - v * s
    y[..., 1:R:2] = v * c + u * s
    return y


def in_window(query_pos: torch.Tensor, key_pos: torch.Tensor, size: Optional[int]) -> torch.Tensor:
    """[Tq, Tk] booleans: 0 <= i - j < size (every earlier key without a size)."""
    d = query_pos[:, None] - key_pos[None, :]
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def _keep(past: Optional[Dict[str, torch.Tensor]], name: str, new: torch.Tensor) -> torch.Tensor:
    """Append ``new`` (rows of tokens) to what ``past`` holds under ``name`` and return all rows."""
    if past is None:
        return new
    rows = new if name not in past else torch.cat([past[name], new], dim=0)
    past[name] = rows
    return rows


def short_conv(p: Plain, x: torch.Tensor, w: torch.Tensor, past: Optional[Dict[str, torch.Tensor]],
               name: str) -> torch.Tensor:
    """Per channel: y_t = sum_j w[:, j] x_(t - (K-1) + j), zeros before the start of the sequence."""
    T, C = x.shape
    K = w.shape[1]
    key = "conv." + name
    before = torch.zeros(K - 1, C, dtype=x.dtype) if past is None or key not in past else past[key]
    rows = torch.cat([before, x], dim=0)
    if past is not None:
        past[key] = rows[rows.shape[0] - (K - 1):].clone()
    y = torch.zeros(T, C, dtype=x.dtype)
    for j in range(K):
        y = y + rows[j:j + T] * p.round(w)[:, j][None, :]
    return y


def windowed_attention(p: Plain, h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping[str, Any],
                       past: Optional[Dict[str, torch.Tensor]], first_position: int) -> torch.Tensor:
    """The concatenated heads [T, H V] before W_o."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(first_position, first_position + T)
    made = {n: p.round(short_conv(p, p.linear(h, w[n]), w[n + ".conv"], past, n)) for n in ("q", "k", "v")}
    q = p.round(rotate_adjacent(made["q"].reshape(T, H, D), pos, m["rot"]))
    k = p.round(rotate_adjacent(made["k"].reshape(T, G, D), pos, m["rot"]))
    k_all = _keep(past, "k", k)
    v_all = _keep(past, "v", made["v"].reshape(T, G, V))
    key_pos = torch.arange(k_all.shape[0])
    mask = m.get("mask") or {}
    seen = in_window(pos, key_pos, mask.get("size"))
    out = torch.zeros(T, H, V, dtype=q.dtype)
    for head in range(H):
        g = head // (H // G)
        s = (q[:, head] @ k_all[:, g].t()) * float(m["scale"])
        out[:, head] = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v_all[:, g]
    return p.round(out.reshape(T, H * V))


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, beta: torch.Tensor, g: torch.Tensor,
               S: torch.Tensor):
    """Token by token, per head: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.
    q, k: [T, H, D]; v: [T, H, V]; beta: [T, H]; g: [T, H, D]; S: [H, D, V].  Returns o [T, H, V] and the last S."""
    out = torch.zeros_like(v)
    for t in range(v.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def delta_mixer(p: Plain, h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping[str, Any], eps: float,
                past: Optional[Dict[str, torch.Tensor]]) -> torch.Tensor:
    """The normed and gated heads [T, H V] before W_o; the decay is one a head where the layer has 'a', one a key
    channel where it has 'a1' and 'a2'."""
    T = h.shape[0]
    H, G, D, V = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    made = {n: silu(short_conv(p, p.linear(h, w[n]), w[n + ".conv"], past, n)) for n in ("q", "k", "v")}
    share = torch.arange(H) // (H // G)
    q = (unit_vector(made["q"].reshape(T, G, D)) * D ** -0.5)[:, share]
    k = unit_vector(made["k"].reshape(T, G, D))[:, share]
    v = made["v"].reshape(T, H, V)
    beta = torch.sigmoid(p.linear_wide(h, w["b"]))
    rate = torch.exp(w["A_log"].to(h.dtype))
    if "a" in w:
        step = softplus(p.linear_wide(h, w["a"]) + w["dt_bias"].to(h.dtype))
        g = torch.exp(-rate * step)[:, :, None].expand(T, H, D)
    else:
        step = softplus(p.linear_wide(p.linear(h, w["a1"]), w["a2"]) + w["dt_bias"].to(h.dtype)).reshape(T, H, D)
        rate = rate.reshape(H, -1)                     # a number a head
        g = torch.exp(-rate[None] * step)
    S = torch.zeros(H, D, V, dtype=h.dtype) if past is None or "S" not in past else past["S"]
    o, S = delta_rule(q, k, v, beta, g, S)
    if past is not None:
        past["S"] = S
    o = (rms_unit(o, eps) * w["norm"].to(o.dtype)).reshape(T, H * V)
    gate = silu(p.linear(h, w["g"])) if "g" in w else torch.sigmoid(p.linear(p.linear(h, w["g1"]), w["g2"]))
    return p.round(o * gate)


def gated_mlp(p: Plain, h: torch.Tensor, w: Mapping[str, torch.Tensor]) -> torch.Tensor:
    return p.linear(p.round(silu(p.linear(h, w["gate"])) * p.linear(h, w["up"])), w["down"])


def _sub(tensors: Mapping[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def gather_streams(x: torch.Tensor, hc: Mapping[str, torch.Tensor]) -> torch.Tensor:
    """x: [s, T, d]; the sublayer's input before its norm."""
    return torch.einsum("a,atd->td", hc["in"].to(x.dtype), x)


def spread_streams(x: torch.Tensor, y: torch.Tensor, hc: Mapping[str, torch.Tensor]) -> torch.Tensor:
    """Every new stream is a mixture of the old ones: x_b <- sum_a mix[a, b] x_a + out[b] y."""
    return torch.einsum("ab,atd->btd", hc["mix"].to(x.dtype), x) + hc["out"].to(x.dtype)[:, None, None] * y[None]


class PlainMopilorn:
    """The whole model over one sequence at a time, with keys, values and states kept between calls."""

    def __init__(self, config: Mapping[str, Any], tensors: Mapping[str, torch.Tensor],
                 dtype: torch.dtype = torch.float32, wide: bool = False):
        self.c = config
        self.p = Plain(dtype, wide)
        self.w = {k: (v if v.dtype in (torch.int32, torch.int64) else v.to(self.p.acc)) for k, v in tensors.items()}
        self.eps = float(config["norm"]["eps"])
        self.streams = int(config["streams"])

    def new_state(self) -> List[Dict[str, Any]]:
        return [{"left": {}, "right": {}} for _ in self.c["layers"]]

    def mixer(self, kind: str, h: torch.Tensor, w: Mapping[str, torch.Tensor], m: Mapping[str, Any],
              past: Optional[Dict[str, Any]], first_position: int) -> torch.Tensor:
        p, eps = self.p, self.eps
        sides = {n: None if past is None else past[n] for n in ("left", "right")}
        if kind == "channel_delta":
            return p.linear_wide(delta_mixer(p, h, w, m, eps, sides["right"]), w["o"])
        if kind == "parallel":
            left, right = _sub(w, "left."), _sub(w, "right.")
            a = p.linear_wide(windowed_attention(p, h, left, m["left"], sides["left"], first_position), left["o"])
            b = p.linear_wide(delta_mixer(p, h, right, m["right"], eps, sides["right"]), right["o"])
            return 0.5 * (norm_plain(a, left["out"], eps) + norm_plain(b, right["out"], eps))
        raise ValueError(f"layer type {kind!r} is not part of the design")

    def forward(self, tokens: List[int], state: Optional[List[Dict[str, Any]]] = None,
                first_position: int = 0, layers_out: Optional[list] = None) -> torch.Tensor:
        """Logits [T, vocab] of the given tokens, which follow ``first_position`` tokens held in ``state``."""
        c, w, p = self.c, self.w, self.p
        x = w["embed"][torch.tensor(tokens, dtype=torch.long)][None].repeat(self.streams, 1, 1)
        for i, layer in enumerate(c["layers"]):
            lw = _sub(w, f"l{i}.")
            hc = _sub(lw, "hc1.")
            h = norm_plain(gather_streams(x, hc), lw["norm1"], self.eps)
            y = self.mixer(layer["type"], h, _sub(lw, "mix."), layer["mixer"], None if state is None else state[i],
                           first_position)
            x = spread_streams(x, y, hc)
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp["kind"] != "dense":
                    raise ValueError(f"feed-forward kind {mlp['kind']!r} is not part of the design")
                hc = _sub(lw, "hc2.")
                h = norm_plain(gather_streams(x, hc), lw["norm2"], self.eps)
                x = spread_streams(x, gated_mlp(p, h, _sub(lw, "mlp.")), hc)
            if layers_out is not None:
                layers_out.append(x.sum(dim=0))
        h = norm_plain(x.sum(dim=0), w["final.norm"], self.eps)
        return soft_cap(p.linear_wide(h, w["head"]), c.get("logit_softcap")).to(torch.float32)
