"""Typed configuration of the Mopilorn decoder, read from config.json.

The design: a token is carried by ``streams`` residual streams (hyper-connections): around a sublayer with learned
numbers in, out and mix, ``u = sum_a in[a] x_a``, ``y = sublayer(norm(u))``, ``x_b <- sum_a mix[a, b] x_a + out[b] y``; behind
the last layer the streams are summed.  Norms are RMS norms of plain weight.  A layer's mixer is one of two:

``parallel``       two mixers on the same rows, half the sum of their outputs, each RMS-normed over the model width with a
                   weight of its own.  Left: grouped-query attention without biases; q, k and v behind a short causal
                   convolution a channel; rotary positions over the first part of every q and k head, dimension 2i paired
                   with 2i + 1, the frequencies optionally stretched by wavelength; a sliding window.  Right: a gated delta
                   rule with one decay a head and a silu gate.
``channel_delta``  a gated delta rule with one decay a key channel, made by a product of low rank, and a sigmoid gate of
                   low rank.
The feed-forward is ``W_down (silu(W_gate h) * (W_up h))``.  The head is a matrix of its own; logits z become
``logit_softcap * tanh(z / logit_softcap)``.

config.json keys
----------------
architecture            "Mopilorn"
vocab, width            sizes of the embedding table and of the head
streams                 residual streams a token
norm.eps                epsilon of every norm
logit_softcap           the cap on the logits (absent or null: none)
layers[i].type          "parallel" or "channel_delta"
layers[i].mixer         parallel: left (heads, kv_heads, dim, vdim, scale, conv, rot.dims, rot.base, rot.scaling with factor,
                        low, high, original or null, mask.size; mask absent or null: causal) and right
                        a delta rule (right, or the mixer of channel_delta): heads, kv_heads, dim, vdim, conv; for
                        channel_delta optionally decay_rank and gate_rank (absent: the ranks the tensors have)
layers[i].mlp           null, or kind "dense" with ff

Every other size and constant is read from here; the loader checks the tensors' shapes against it.  Tensor names:
``embed``, ``final.norm``, ``head`` and, under ``l<i>.``, ``norm1``, ``norm2``, ``hc1|hc2.in|out|mix``, ``mix.*``
(``mix.left.*``, ``mix.right.*``; a convolution under the name of the tensor it follows, ``.conv``) and
``mlp.gate|up|down``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .common import ConfigError, architecture_name
from .spec import FeedForwardSpec, HookSpec, LayerSpec, MixerSpec, ModelSpec, NormSpec, PositionSpec
from .tumatar import _int, _num, _obj

LAYER_TYPES = ("parallel", "channel_delta")
SIDE_FACTOR = 0.5           # of the sum of a parallel layer's two normed outputs


def _heads(m: Mapping[str, Any], where: str) -> None:
    H, G = _int(m, "heads", where), _int(m, "kv_heads", where)
    if H % G:
        raise ConfigError(f"config.json: {where}heads {H} is not a multiple of kv_heads {G}")
    for key in ("dim", "vdim", "conv"):
        _int(m, key, where)


def _check_attention(m: Mapping[str, Any], where: str) -> None:
    _heads(m, where)
    _num(m, "scale", where)
    rot = _obj(m, "rot", where)
    R = _int(rot, "dims", where + "rot.")
    if R % 2 or R > m["dim"]:
        raise ConfigError(f"config.json: {where}rot.dims {R} must be even and at most the head's {m['dim']}")
    _num(rot, "base", where + "rot.")
    scaling = _obj(rot, "scaling", where + "rot.", optional=True)
    if scaling is not None:
        for key in ("factor", "low", "high", "original"):
            _num(scaling, key, where + "rot.scaling.")
    mask = _obj(m, "mask", where, optional=True)
    if mask is not None:
        _int(mask, "size", where + "mask.")


def _check_mixer(kind: Any, m: Mapping[str, Any], where: str) -> None:
    if kind == "parallel":
        _check_attention(_obj(m, "left", where), where + "left.")
        _heads(_obj(m, "right", where), where + "right.")
    elif kind == "channel_delta":
        _heads(m, where)
        for key in ("decay_rank", "gate_rank"):
            if m.get(key) is not None:
                _int(m, key, where)
    else:
        raise ConfigError(f"config.json: {where[:-len('mixer.')]}type {kind!r} is not known ({', '.join(LAYER_TYPES)})")


@dataclass(frozen=True)
class MopilornConfig:
    ARCHITECTURE = "Mopilorn"

    raw: Mapping[str, Any]          # the checked dictionary, as it was read
    vocab: int
    width: int
    streams: int
    eps: float
    softcap: Optional[float]
    layers: Tuple[Mapping[str, Any], ...]

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
    def from_dict(cls, d: Mapping[str, Any]) -> "MopilornConfig":
        if architecture_name(d) != cls.ARCHITECTURE:
            raise ConfigError(f"config.json names the architecture {architecture_name(d)!r}, not {cls.ARCHITECTURE!r}")
        vocab, width, streams = _int(d, "vocab", ""), _int(d, "width", ""), _int(d, "streams", "")
        norm = _obj(d, "norm", "")
        layers = d.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]."
            if not isinstance(layer, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            _check_mixer(layer.get("type"), _obj(layer, "mixer", where), where + "mixer.")
            mlp = _obj(layer, "mlp", where, optional=True)
            if mlp is not None:
                if mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind {mlp.get('kind')!r} is not known (dense)")
                _int(mlp, "ff", where + "mlp.")
            checked.append(copy.deepcopy(dict(layer)))
        softcap = None if d.get("logit_softcap") is None else _num(d, "logit_softcap", "")
        return cls(raw=copy.deepcopy(dict(d)), vocab=vocab, width=width, streams=streams, eps=_num(norm, "eps", "norm."),
                   softcap=softcap, layers=tuple(checked))

    def to_dict(self) -> Dict[str, Any]:
        return copy.deepcopy(dict(self.raw))

    # ------------------------------------------------------------------ layout
    def _attention(self, m: Mapping[str, Any], names: Dict[str, str], local: str, tensors: str) -> MixerSpec:
        for p in ("q", "k", "v"):
            names[f"{local}{p}.weight"] = f"{tensors}{p}"
            names[f"{local}{p}.conv"] = f"{tensors}{p}.conv"
        names[f"{local}o.weight"] = f"{tensors}o"
        scaling = m["rot"].get("scaling")
        if scaling is not None:
            scaling = {"rope_type": "llama3", "factor": float(scaling["factor"]),
                       "low_freq_factor": float(scaling["low"]), "high_freq_factor": float(scaling["high"]),
                       "original_max_position_embeddings": scaling["original"]}
        return MixerSpec(kind="capped_attention", width=self.width, n_heads=m["heads"], n_kv_heads=m["kv_heads"],
                         head_dim=m["dim"], window=(m.get("mask") or {}).get("size"), scale=float(m["scale"]),
                         position=PositionSpec(kind="rope", rotary_dim=m["rot"]["dims"], theta=float(m["rot"]["base"]),
                                               scaling=scaling, options={"pairs": "adjacent"}),
                         options={"value_dim": m["vdim"], "conv": m["conv"]})

    def _delta(self, m: Mapping[str, Any], names: Dict[str, str], local: str, tensors: str, per_channel: bool) -> MixerSpec:
        for p in ("q", "k", "v"):
            names[f"{local}{p}.conv"] = f"{tensors}{p}.conv"
        for p in ("q", "k", "v", "b", "o", "norm") + (("a1", "a2", "g1", "g2") if per_channel else ("a", "g")):
            names[f"{local}{p}.weight"] = f"{tensors}{p}"
        for p in ("A_log", "dt_bias"):
            names[f"{local}{p}"] = f"{tensors}{p}"
        options: Dict[str, Any] = {"value_dim": m["vdim"], "taps": m["conv"], "norm_eps": self.eps}
        if per_channel:
            options.update(decay="channel", gate="sigmoid", gate_low_rank=True, decay_rank=m.get("decay_rank"),
                           gate_rank=m.get("gate_rank"))
        else:
            options.update(decay="head", gate="silu", gate_low_rank=False)
        return MixerSpec(kind="gated_delta_rule", width=self.width, n_heads=m["heads"], n_kv_heads=m["kv_heads"],
                         head_dim=m["dim"], options=options)

    def _layer(self, i: int, layer: Mapping[str, Any]) -> LayerSpec:
        d, s = self.width, self.streams
        norm = NormSpec("stream_norm", d, self.eps, {"streams": s})
        names: Dict[str, str] = {}
        sublayers = [("mixer", 1)] + ([("ffn", 2)] if layer.get("mlp") is not None else [])
        for local, q in sublayers:
            names[f"{local}_norm.weight"] = f"norm{q}"
            names[f"{local}_norm.in"] = f"hc{q}.in"
            names[f"{local}_hc.out"] = f"hc{q}.out"
            names[f"{local}_hc.mix"] = f"hc{q}.mix"
        m = layer["mixer"]
        if layer["type"] == "parallel":
            parts = (("left.", self._attention(m["left"], names, "mixer.left.", "mix.left.")),
                     ("right.", self._delta(m["right"], names, "mixer.right.", "mix.right.", False)))
            for side, _ in parts:
                names[f"mixer.{side}out_norm.weight"] = f"mix.{side}out"
            mixer = MixerSpec(kind="side_by_side", width=d, options={"parts": parts, "norm_eps": self.eps, "factor": SIDE_FACTOR})
        else:
            mixer = self._delta(m, names, "mixer.", "mix.", True)
        ffn = None
        if layer.get("mlp") is not None:
            ffn = FeedForwardSpec(kind="gated_mlp", width=d, intermediate=layer["mlp"]["ff"], activation="silu")
            for part in ("gate", "up", "down"):
                names[f"ffn.{part}.weight"] = f"mlp.{part}"
        return LayerSpec(block="hyper", prefix=f"l{i}.", mixer_norm=norm, mixer=mixer,
                         ffn_norm=norm if ffn is not None else None, ffn=ffn, names=names, options={"streams": s})

    def model_spec(self) -> ModelSpec:
        hook = None if self.softcap is None else HookSpec("soft_cap", {"cap": self.softcap})
        return ModelSpec(
            architecture=self.ARCHITECTURE, width=self.width, vocab_size=self.vocab,
            layers=tuple(self._layer(i, layer) for i, layer in enumerate(self.layers)),
            schedule=tuple(range(len(self.layers))),
            final_norm=NormSpec("stream_norm", self.width, self.eps, {"streams": self.streams, "learned": False}),
            embedding_name="embed", final_norm_name="final.norm", head_name="head", embedding_scale=1.0, max_positions=0,
            logits_hook=hook, streams=self.streams)
