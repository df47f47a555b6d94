"""Typed configuration of the Lilulix decoder, read from config.json.

The design: a token's embedding is the sum of its own row and of a row that its pair with the token before chooses by
a hash.  Every layer has ONE norm h = norm(x) that its mixer and its feed-forward both read, ``x += mixer(h) + ff(h)``.
A run of consecutive layers is passed through several times with the same weights, each pass keeping its own cache;
before every pass but the first the embedded tokens are added to the residual once more, and before every pass a
learned vector of that pass.  A layer's mixer is one of two:

``latent_attention``  keys and values are made per head from a normed low-rank latent, beside one rotated key part that
                      all heads share; queries have an unrotated and a rotated part; a learned number per head in the
                      softmax's denominator; one sigmoid gate an element on the concatenated heads.
``attention``         grouped-query attention without rotation: q and k with biases, each head RMS-normed with a weight
                      that all heads of a kind share; the values are the projected keys, before that norm; a bias that
                      grows with the distance, by a fixed slope a head; one more 1 in the softmax's denominator.
The feed-forward is dense and gated with the tanh form of gelu.  The head is the embedding table behind a final norm.

config.json keys
----------------
architecture              "Lilulix"
vocab, width              sizes of the embedding table
embedding.bigram          buckets (rows of the pair table, which has one more for a sequence's first token), mul_prev,
                          mul_cur (the hash's factors)
norm.eps                  epsilon of every norm
layers[i].type            "latent_attention" or "attention"
layers[i].mixer           latent_attention: heads, dim, rot_dim, vdim, kv_rank, scale, rot.base, rot.dims (= rot_dim)
                          attention: heads, kv_heads, dim, vdim (= dim), scale
layers[i].mlp             null, or kind "dense" with ff
loop                      null/absent, or start, stop, times: layers start..stop-1 run ``times`` times in a row

Every size and constant is read from here; nothing is inferred from tensor shapes (the loader checks the shapes
against this configuration).  Tensor names: ``embed``, ``bigram``, ``loop.step``, ``final.norm`` and, under ``l<i>.``,
``norm1``, ``mlp.gate``/``mlp.up``/``mlp.down`` and the mixer's tensors ``mix.*``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .common import ConfigError, architecture_name
from .spec import FeedForwardSpec, HookSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec
from .tumatar import _int, _num, _obj

LAYER_TYPES = ("latent_attention", "attention")

# Constants the design fixes.
BIAS_EXPONENT = 8.0         # attention: head h of H loses 2^(-BIAS_EXPONENT (h + 1) / H) of its score a position

# A choice of this library, not of the design: how much larger than it is a cached latent may be kept in bfloat16 if
# that lets the tensor-core attention kernels take it.
PAD_LATENT = 4.0 / 3.0


@dataclass(frozen=True)
class LilulixConfig:
    ARCHITECTURE = "Lilulix"

    raw: Mapping[str, Any]          # the checked dictionary, as it was read
    vocab: int
    width: int
    eps: float
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: Tuple[Mapping[str, Any], ...]
    loop: Optional[Tuple[int, int, int]]      # start, stop, times

    @property
    def architecture(self) -> str:
        return self.ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def eos_token_ids(self) -> Tuple[int, ...]:
        return ()

    # -------------------------------------------------------------- reading
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "LilulixConfig":
        if architecture_name(d) != cls.ARCHITECTURE:
            raise ConfigError(f"config.json names the architecture {architecture_name(d)!r}, not {cls.ARCHITECTURE!r}")
        vocab = _int(d, "vocab", "")
        width = _int(d, "width", "")
        bigram = _obj(_obj(d, "embedding", ""), "bigram", "embedding.")
        norm = _obj(d, "norm", "")
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]."
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = layer.get("type")
            m = _obj(layer, "mixer", where)
            mw = where + "mixer."
            if kind == "latent_attention":
                for key in ("heads", "dim", "vdim", "kv_rank"):
                    _int(m, key, mw)
                turned = _int(m, "rot_dim", mw)
                rot = _obj(m, "rot", mw)
                if turned % 2 or _int(rot, "dims", mw + "rot.") != turned:
                    raise ConfigError(f"config.json: {mw}rot_dim {turned} must be even and equal to rot.dims {rot['dims']}")
                _num(rot, "base", mw + "rot.")
            elif kind == "attention":
                H, G = _int(m, "heads", mw), _int(m, "kv_heads", mw)
                if H % G:
                    raise ConfigError(f"config.json: {mw}heads {H} is not a multiple of kv_heads {G}")
                D = _int(m, "dim", mw)
                if _int(m, "vdim", mw) != D:
                    raise ConfigError(f"config.json: {mw}vdim {m['vdim']} must equal dim {D}: the values are the keys")
            else:
                raise ConfigError(f"config.json: {where}type {kind!r} is not known ({', '.join(LAYER_TYPES)})")
            _num(m, "scale", mw)
            mlp = _obj(layer, "mlp", where, optional=True)
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind {mlp.get('kind')!r} is not known (dense)")
                _int(mlp, "ff", where + "mlp.")
            checked.append(copy.deepcopy(dict(layer)))
        loop = _obj(d, "loop", "", optional=True)
        loop_t = None
        if loop is not None:
            start, stop = _int(loop, "start", "loop.", 0), _int(loop, "stop", "loop.")
            times = _int(loop, "times", "loop.")
            if not start < stop <= len(checked):
                raise ConfigError(f"config.json: loop {start}..{stop} does not lie within the {len(checked)} layers")
            loop_t = (start, stop, times)
        return cls(raw=copy.deepcopy(dict(d)), vocab=vocab, width=width, eps=_num(norm, "eps", "norm."),
                   buckets=_int(bigram, "buckets", "embedding.bigram."),
                   mul_prev=_int(bigram, "mul_prev", "embedding.bigram.", 0),
                   mul_cur=_int(bigram, "mul_cur", "embedding.bigram.", 0), layers=tuple(checked), loop=loop_t)

    def to_dict(self) -> Dict[str, Any]:
        return copy.deepcopy(dict(self.raw))

    # ------------------------------------------------------------------ layout
    def running_order(self) -> Tuple[Tuple[int, Optional[int]], ...]:
        """(layer, pass number at the first layer of a pass of the repeated run or None) in running order."""
        n = len(self.layers)
        if self.loop is None:
            return tuple((i, None) for i in range(n))
        start, stop, times = self.loop
        order = [(i, None) for i in range(start)]
        for t in range(times):
            order += [(i, t if i == start else None) for i in range(start, stop)]
        return tuple(order + [(i, None) for i in range(stop, n)])

    def _mixer(self, kind: str, m: Mapping[str, Any], names: Dict[str, str]) -> MixerSpec:
        d, eps = self.width, self.eps
        if kind == "latent_attention":
            for p in ("q", "dkv", "uk", "uv", "g", "o"):
                names[f"mixer.{p}.weight"] = f"mix.{p}"
            names["mixer.dkv_norm.weight"] = "mix.dkv.norm"
            names["mixer.sink"] = "mix.sink"
            return MixerSpec(kind="latent_attention", width=d, n_heads=m["heads"], n_kv_heads=1, head_dim=m["dim"],
                             scale=float(m["scale"]),
                             position=PositionSpec(kind="rope", rotary_dim=m["rot_dim"], theta=float(m["rot"]["base"])),
                             options={"value_dim": m["vdim"], "kv_rank": m["kv_rank"], "q_rank": None,
                                      "rot_dim": m["rot_dim"], "gate": "sigmoid", "sink": True, "norm_eps": eps,
                                      "pad_to_fast": PAD_LATENT})
        for p in ("q", "k", "o"):
            names[f"mixer.{p}.weight"] = f"mix.{p}"
        for p in ("q", "k"):
            names[f"mixer.{p}.bias"] = f"mix.{p}.b"
            names[f"mixer.{p}_norm.weight"] = f"mix.{p}.norm"
        return MixerSpec(kind="capped_attention", width=d, n_heads=m["heads"], n_kv_heads=m["kv_heads"], head_dim=m["dim"],
                         bias=True, scale=float(m["scale"]), position=PositionSpec(kind="none"),
                         options={"value_dim": m["vdim"], "values": "keys", "qk_norm": "head_first", "qk_norm_eps": eps,
                                  "distance_bias": BIAS_EXPONENT, "sink": "zero"})

    def model_spec(self) -> ModelSpec:
        d, eps = self.width, self.eps
        norm = NormSpec("rmsnorm", d, eps)
        layers = []
        for i, layer in enumerate(self.layers):
            names: Dict[str, str] = {"mixer_norm.weight": "norm1"}
            mixer = self._mixer(layer["type"], layer["mixer"], names)
            mlp = layer.get("mlp")
            ffn = None
            if mlp is not None:
                ffn = FeedForwardSpec(kind="gated_mlp", width=d, intermediate=mlp["ff"], activation="gelu_tanh")
                for part in ("gate", "up", "down"):
                    names[f"ffn.{part}.weight"] = f"mlp.{part}"
            layers.append(LayerSpec(block="shared_norm", prefix=f"l{i}.", mixer_norm=norm, mixer=mixer, ffn_norm=None,
                                    ffn=ffn, names=names))
        order = self.running_order()
        place_hooks = {place: HookSpec("add_row", {"rows": self.loop[2], "row": t, "width": d, "add_embedding": t > 0},
                                       {"table": "loop.step"})
                       for place, (_, t) in enumerate(order) if t is not None}
        pairs = HookSpec("token_pairs", {"buckets": self.buckets, "width": d, "mul_prev": self.mul_prev,
                                         "mul_cur": self.mul_cur}, {"table": "bigram"})
        return ModelSpec(
            architecture=self.ARCHITECTURE, width=d, vocab_size=self.vocab, layers=tuple(layers),
            schedule=tuple(li for li, _ in order), final_norm=norm, embedding_name="embed",
            final_norm_name="final.norm", head_name=None, embedding_scale=1.0, max_positions=0,
            embed_hook=pairs, place_hooks=place_hooks)
