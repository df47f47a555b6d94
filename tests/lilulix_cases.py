"""Small Lilulix configurations for the tests, and how a model with tensors the test controls is built.

The configurations differ from one another in every size and option: heads of 64 and 128 and heads that are no multiple
of 8; groups of 1, 2, 3 and 5 query heads a key/value head; head counts that are no power of two (slopes); latents that
fill a tensor-core head, latents kept with zeros behind them and latents that fit none; rotated parts of two dimensions;
more than sixteen latent heads; runs of layers passed through once, twice, three times and not at all, starting at the
first layer or ending at the last; layers without a feed-forward; one bucket, more buckets than pairs, factors of zero
and factors whose products pass 32 bits.
"""
from __future__ import annotations

import copy
from typing import Callable, Dict, Optional

import torch


def _lat(heads, dim, rot_dim, vdim, rank, scale, base, ff):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _att(heads, kv, dim, scale, ff):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _model(vocab, width, eps, bigram, loop, layers):
    d = {"architecture": "Lilulix", "vocab": vocab, "width": width, "norm": {"eps": eps},
         "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# sizes that are no multiple of 8; the run of layers begins with the first one
CFG_A = _model(157, 72, 1e-5, (211, 7, 3), (0, 2, 3), [
    _att(6, 2, 20, 0.3, 136), _lat(5, 12, 6, 10, 21, 0.3, 50.0, 60), _att(3, 3, 12, 0.5, None), _lat(3, 8, 2, 40, 30, 0.25, 7.0, 50)])
# the head sizes of the tensor-core kernels, eighteen latent heads, the run ends with the last layer
CFG_B = _model(300, 128, 1e-6, (97, 1000003, 998244353), (1, 5, 2), [
    _lat(4, 32, 32, 48, 96, 0.15, 10000.0, 200), _att(4, 1, 64, 0.12, 96), _att(10, 2, 128, 0.08, 64),
    _lat(18, 16, 16, 8, 40, 0.2, 100.0, 72), _att(3, 3, 64, 0.2, None)])
# the values that make mechanisms vanish: one head, one bucket, one pass, one pair of rotated dimensions, no feed-forward
CFG_C = _model(61, 40, 1e-6, (1, 0, 5), (1, 2, 1), [
    _att(1, 1, 8, 0.6, 8), _lat(1, 3, 2, 5, 8, 0.5, 20.0, None), _att(2, 1, 4, 0.7, 24)])
# no run of layers at all; latents kept with zeros behind them in bfloat16
CFG_D = _model(200, 192, 1e-5, (50021, 1, 0), None, [
    _lat(6, 24, 8, 24, 88, 0.2, 1000.0, 160), _att(12, 4, 64, 0.125, 100), _lat(2, 64, 64, 64, 40, 0.1, 500.0, 120)])
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}


def config(name: str) -> dict:
    return copy.deepcopy(CONFIGS[name])


def lively(w: Dict[str, torch.Tensor]) -> None:
    """Biases of the size of the projections' outputs, sinks of the size of the scores, pair rows and pass vectors of the
    size of the embedding: one that is lost, or taken from another row, shows."""
    for name, t in w.items():
        if name.endswith(".b"):
            t.copy_((t.float() * 3.0).to(t.dtype))
        elif name.endswith(".sink"):
            t.copy_((t.float() * 10.0 + 0.5).to(t.dtype))


def build(cfg: dict, seed: int, dn: str, tweak: Optional[Callable] = lively, std: float = 0.12, **options):
    """(engine, config dictionary, tensors on the CPU) of a model with random weights, changed by ``tweak``."""
    from tikalix_cases import build as build_any
    return build_any(cfg, seed, dn, tweak=tweak, std=std, **options)


def plain(cfg: dict, w: Dict[str, torch.Tensor], dn: str, wide: bool = False):
    import plain_lilulix
    return plain_lilulix.PlainLilulix(cfg, w, {"float32": torch.float32, "bfloat16": torch.bfloat16}[dn], wide)


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per row: the difference of the logits (mean taken off, root mean square over the vocabulary) relative to the root
    mean square of the row."""
    got, want = got.detach().float().cpu(), want.detach().float().cpu()
    assert got.shape == want.shape, f"shape {tuple(got.shape)} != {tuple(want.shape)}"
    d = got - want
    d = d - d.mean(dim=1, keepdim=True)
    ref = want - want.mean(dim=1, keepdim=True)
    return d.pow(2).mean(dim=1).sqrt() / ref.pow(2).mean(dim=1).sqrt().clamp_min(1e-6)


def rows_close(got: torch.Tensor, want: torch.Tensor, dn: str, what: str = "") -> None:
    """float32: every row within 3e-5.  bfloat16: all rows but one in fifteen (or two) within 0.05, and those within 0.3."""
    err = row_errors(got, want)
    assert torch.isfinite(err).all(), f"{what}: a row is not finite"
    if dn == "float32":
        assert err.max().item() < 3e-5, f"{what}: row {int(err.argmax())} differs by {err.max().item():.3g}"
    else:
        over = int((err > 0.05).sum())
        assert err.max().item() < 0.3 and over <= max(2, got.shape[0] // 15) and over <= got.shape[0] // 2, \
            f"{what}: {over} of {got.shape[0]} rows differ, the worst (row {int(err.argmax())}) by {err.max().item():.3g}"
