"""Attention through a low-rank latent, with a sigmoid gate on the heads' outputs, a query latent, rotary positions
on a part of the keys that all heads share, and a sliding window, each of which may be left out.

For the normed input h of a layer with H heads of query/key size D (unrotated) and Rr (rotated), value size V and
latent sizes Rq, R:
    c_q = norm(W_dq h)            q  = W_uq c_q            [H, D + Rr]     (``q_rank`` None: q = W_q h)
    [c | r] = W_dkv h             c <- norm(c)             R and Rr elements a position (r is not normed)
    k_j = W_uk c_j,  v_j = W_uv c_j                        [H, D], [H, V]   (j: a position)
    s_ij = (q_i[:D] . k_j + rot(q_i[D:], i) . rot(r_j, j)) * scale,  j <= i and i - j < window
    p = softmax_j(s), with exp(sink_h) also in the denominator  (``sink``: a learned number a head; left out: a plain softmax)
    o_i = sum_j p_ij v_j
    out = W_o (o * sigmoid(W_g h))                                          (``gate`` None: out = W_o o)
Only c and the rotated r are kept per position: one vector of Rr + R elements that is key and value at once
(``KVNeed(values_are_keys=True)``).  The products with W_uk and W_uv are moved to the other side of the
attention, head by head:
    q'_i = [rot(q_i[D:]) | W_uk[h]^T q_i[:D]]  (Rr + R elements per head),   s_ij = (q'_i . [rot(r_j) | c_j]) * scale,
    l_i  = sum_j p_ij [rot(r_j) | c_j],                                      o_i  = W_uv[h] l_i[Rr:],
so the attention itself is the library's attention of H query heads over one key/value head of size Rr + R
whose keys and values are the same pages, and the two per-head products are block-diagonal products (the first also
moves the rotated part of a query to the front of its head; the second skips the first Rr elements).  The projections
of h (W_dq or W_q, W_dkv, W_g) are one matrix product with a float32 result: the norms of the latents, the rotations
and the gate's sigmoid read it in float32.  One kernel (``kernels.latent_prep``) stands between the projections and the
first per-head product: it norms c, turns r and the queries' rotated parts, and writes the token's row of the cache.
The rows of W_q and W_dkv that are rotated are taken in the order that makes the encoding's pairs the halves the kernel
turns.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import kernels
from ..config.spec import MixerSpec, NormSpec
from .base import KVNeed, LayerIO, ParamDecl, Part, StateNeed, norm_class, position_class, register_mixer
from .linear import Linear


class LatentAttention(Part):
    can_overwrite = True

    def __init__(self, spec: MixerSpec, dtype: torch.dtype, device: torch.device):
        super().__init__(spec, dtype, device)
        o = spec.options
        self.n_heads, self.dim = spec.n_heads, spec.head_dim
        self.value_dim, self.kv_rank = int(o["value_dim"]), int(o["kv_rank"])
        self.q_rank = None if o.get("q_rank") is None else int(o["q_rank"])
        self.rot_dim = int(o.get("rot_dim") or 0)
        if spec.scale is None:
            raise ValueError("latent_attention: the spec must give the factor on the scores")
        self.scale = float(spec.scale)
        self.gate = o.get("gate", "sigmoid")
        if self.gate not in (None, "sigmoid"):
            raise ValueError(f"latent_attention: output gate {self.gate!r} is not known (sigmoid)")
        self.window = None if spec.window is None else int(spec.window)
        self.has_sink = bool(o.get("sink"))
        self.kept = self.kept_size(self.rot_dim + self.kv_rank, dtype, float(o.get("pad_to_fast", 1.0)))
        if self.kept > 512:
            raise ValueError(f"latent_attention: a key/value latent of {self.kv_rank} elements beside {self.rot_dim} "
                             "rotated ones is not supported (at most 512 together)")
        self.position = position_class(spec.position.kind)(spec.position, dtype, device)
        table = self.position.rotary_table()
        if self.rot_dim and (table is None or table[1] != self.rot_dim):
            raise ValueError("latent_attention: the position encoding must turn exactly the rotated part of the keys")
        if not self.rot_dim and table is not None:
            raise ValueError("latent_attention: a rotation needs a rotated part of the keys (rot_dim)")
        eps = float(o["norm_eps"])
        self.norm_eps = eps
        self.q_norm = (norm_class("rmsnorm")(NormSpec("rmsnorm", self.q_rank, eps), dtype, device)
                       if self.q_rank is not None else None)
        self.kv_norm_w: Optional[torch.Tensor] = None
        self.sinks: Optional[torch.Tensor] = None
        self.down: Optional[Linear] = None       # [W_dq or W_q; W_dkv; W_g], the last where there is a gate
        self.uq: Optional[Linear] = None         # W_uq where there is a query latent
        self.o: Optional[Linear] = None
        self.uk_t: Optional[torch.Tensor] = None  # [H, kept, D + Rr]: per head, a query into the latent's space
        self.uv: Optional[torch.Tensor] = None    # [H, V, kept]

    @staticmethod
    def kept_size(size: int, dtype: torch.dtype, most: float = 1.0) -> int:
        """The size a position's vector is kept with: a multiple of 8; in bfloat16 the next size the tensor-core attention
        kernels take (64, 128) when that is at most ``most`` times as much (the option ``pad_to_fast``).  What lies behind
        the vector is zero: it adds nothing to a score and its part of the result is not read."""
        kept = -(-size // 8) * 8
        if dtype == torch.bfloat16:
            for fast in (64, 128):
                if kept <= fast <= kept * most:
                    return fast
        return kept

    @classmethod
    def declare(cls, spec: MixerSpec) -> Dict[str, ParamDecl]:
        o = spec.options
        H, D, V, R, d = spec.n_heads, spec.head_dim, int(o["value_dim"]), int(o["kv_rank"]), spec.width
        Rr = int(o.get("rot_dim") or 0)
        p = {"dkv.weight": ParamDecl((R + Rr, d)), "dkv_norm.weight": ParamDecl((R,), init="ones"),
             "uk.weight": ParamDecl((H * D, R)), "uv.weight": ParamDecl((H * V, R)), "o.weight": ParamDecl((d, H * V))}
        if o.get("q_rank") is not None:
            Rq = int(o["q_rank"])
            p.update({"dq.weight": ParamDecl((Rq, d)), "dq_norm.weight": ParamDecl((Rq,), init="ones"),
                      "uq.weight": ParamDecl((H * (D + Rr), Rq))})
        else:
            p["q.weight"] = ParamDecl((H * (D + Rr), d))
        if o.get("gate", "sigmoid") == "sigmoid":
            p["g.weight"] = ParamDecl((H * V, d))
        if o.get("sink"):
            p["sink"] = ParamDecl((H,))
        return p

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        H, D, V, R, Rr, K = self.n_heads, self.dim, self.value_dim, self.kv_rank, self.rot_dim, self.kept
        order = self.position.head_order(Rr) if Rr and hasattr(self.position, "head_order") else None
        order = list(order) if order is not None else list(range(Rr))
        dkv = tensors["dkv.weight"]
        wq = tensors["uq.weight"] if self.q_rank is not None else tensors["q.weight"]
        if order != list(range(Rr)):
            # the rotated rows in the order that makes the encoding's pairs the halves the kernel turns
            dkv = dkv.index_select(0, torch.tensor(list(range(R)) + [R + i for i in order], dtype=torch.long, device=dkv.device))
            head = torch.tensor(list(range(D)) + [D + i for i in order], dtype=torch.long, device=wq.device)
            wq = wq.view(H, D + Rr, -1).index_select(1, head).reshape(H * (D + Rr), -1)
        ws = [tensors["dq.weight"] if self.q_rank is not None else wq, dkv]
        ws += [tensors["g.weight"]] if self.gate else []
        wide = torch.float32 if any(w.dtype == torch.float32 for w in ws) else ws[0].dtype
        self.down = Linear(torch.cat([w.to(wide) for w in ws], dim=0))
        self.uq = Linear(wq) if self.q_rank is not None else None
        self.o = Linear(tensors["o.weight"])
        if self.q_norm is not None:
            self.q_norm.bind({"weight": tensors["dq_norm.weight"]})
        self.kv_norm_w = tensors["dkv_norm.weight"].float().contiguous()
        if self.has_sink:
            self.sinks = tensors["sink"].float().contiguous()
        self.takes_normed_input = self.down.takes_normed()
        uk = tensors["uk.weight"].view(H, D, R)
        into = uk.new_zeros(H, K, D + Rr)                    # row r of a head: what element r of q' is made of
        for r in range(Rr):
            into[:, r, D + r] = 1.0                          # the rotated part moves to the front, exactly
        into[:, Rr:Rr + R, :D] = uk.transpose(1, 2)
        uv = tensors["uv.weight"].view(H, V, R)
        out_of = uv.new_zeros(H, V, K)
        out_of[:, :, Rr:Rr + R] = uv
        self.uk_t = into.contiguous()
        self.uv = out_of.contiguous()

    def kernel_libraries(self) -> Tuple[str, ...]:
        libs = ("elementwise", "block_linear", "attention")
        libs += kernels.fast_attention_libraries(self.dtype, self.kept, min(self.n_heads, self.HEADS_AT_ONCE), 1,
                                                 sinks=self.has_sink)
        for lin in (self.down, self.uq, self.o):
            if lin is not None:
                libs += lin.libraries(self.dtype)
        return libs

    def cache_needs(self) -> Optional[KVNeed]:
        return KVNeed(1, self.kept, self.window, values_are_keys=True)

    def state_needs(self) -> Optional[StateNeed]:
        return None

    fuses_next_norm = True

    def forward(self, step, io: LayerIO, h, residual: torch.Tensor, accumulate: bool = True, next_norm=None):
        """``h``: the normalised rows or a half-done norm (:class:`NormedInput`).  With ``next_norm`` the output projection
        may do the first half of that norm; the result is then its :class:`NormedInput`."""
        T = residual.shape[0]
        H, D, V, Rn, Rr, K = self.n_heads, self.dim, self.value_dim, self.kv_rank, self.rot_dim, self.kept
        first = self.q_rank if self.q_rank is not None else H * (D + Rr)
        proj = step.ws.buf("lat_proj", (T, first + Rn + Rr + (H * V if self.gate else 0)), torch.float32)
        self.down(h, proj)
        if self.q_norm is not None:
            cq = step.ws.buf("lat_cq", (T, first), self.dtype)
            self.q_norm.forward_rows(proj[:, :first], cq)
            q = step.ws.buf("lat_q", (T, H * (D + Rr)), self.dtype)
            self.uq(cq, q)
            turned = q
        else:
            q = proj[:, :first]
            turned = q if self.dtype == torch.float32 else step.ws.buf("lat_q", (T, first), self.dtype)
        table = self.position.rotary_table()
        kernels.latent_prep(proj, first, Rn, first + Rn, Rr, self.kv_norm_w, self.norm_eps, q, turned, H,
                            table[0] if table is not None else None, step.positions, step.seq_of_token, io.block_table,
                            io.k_pages, io.page_size)
        qc = step.ws.buf("lat_qc", (T, H * K), self.dtype)      # the H queries in the latent's space
        kernels.block_linear(turned, self.uk_t, qc)
        heads = step.ws.buf("lat_heads", (T, H * V), self.dtype)
        gate = proj[:, first + Rn + Rr:] if self.gate else None
        # all heads read the one key/value head; the tensor-core kernels take up to 16 query heads a key/value head,
        # so more heads go through them 16 at a time (the queries are a column slice of the rows, the latent pages
        # are the same)
        n = self.HEADS_AT_ONCE if (H > self.HEADS_AT_ONCE and kernels.fast_attention_libraries(
            self.dtype, K, self.HEADS_AT_ONCE, 1)) else H
        for h0 in range(0, H, n):
            h1 = min(H, h0 + n)
            mixed = step.ws.buf("lat_mixed", (T, (h1 - h0) * K), self.dtype)
            kernels.attention(step, qc[:, h0 * K:h1 * K], mixed, h1 - h0, 1, K, self.scale, self.window, io,
                              sinks=self.sinks[h0:h1] if self.has_sink else None)
            if self.gate:
                kernels.block_linear(mixed, self.uv[h0:h1], heads[:, h0 * V:h1 * V], epilogue="sigmoid_gate",
                                     gate=gate[:, h0 * V:h1 * V])
            else:
                kernels.block_linear(mixed, self.uv[h0:h1], heads[:, h0 * V:h1 * V])
        if not accumulate:
            self.o(heads, residual)
            return None
        return self.o.accumulate_with_norm(step, heads, residual, next_norm, "attn_next")

    HEADS_AT_ONCE = 16


register_mixer("latent_attention", LatentAttention)
