"""Lilulix without a GPU: the configuration reader and its refusals, the layout and the tensor names it produces, the place
the embedding's state has in the cache plan, and the plain implementation's own parts on cases whose answer is known."""
import math

import pytest
import torch

import lilulix_cases as LC
import plain_lilulix as P
from ziglm_b200 import ConfigError, config_from_dict
from ziglm_b200.engine.model import Model, declare_parameters
from ziglm_b200.parts.base import StateNeed


def test_layout_and_names():
    conf = config_from_dict(LC.config("B"))
    spec = conf.model_spec()
    assert spec.architecture == "Lilulix" and spec.head_name is None and spec.embed_hook.kind == "token_pairs"
    assert {l.block for l in spec.layers} == {"shared_norm"} and spec.layers[4].ffn is None
    assert [l.mixer.kind for l in spec.layers] == ["latent_attention", "capped_attention", "capped_attention",
                                                   "latent_attention", "capped_attention"]
    assert spec.layers[0].ffn.kind == "gated_mlp" and spec.layers[0].ffn.activation == "gelu_tanh"
    assert spec.schedule == (0, 1, 2, 3, 4, 1, 2, 3, 4)
    assert sorted(spec.place_hooks) == [1, 5]
    assert [spec.place_hooks[p].options["row"] for p in (1, 5)] == [0, 1]
    assert [spec.place_hooks[p].options["add_embedding"] for p in (1, 5)] == [False, True]
    names = declare_parameters(spec)
    for n, shape in (("embed", (300, 128)), ("bigram", (98, 128)), ("loop.step", (2, 128)), ("final.norm", (128,)),
                     ("l0.norm1", (128,)), ("l0.mix.q", (256, 128)), ("l0.mix.dkv", (128, 128)), ("l0.mix.dkv.norm", (96,)),
                     ("l0.mix.uk", (128, 96)), ("l0.mix.uv", (192, 96)), ("l0.mix.sink", (4,)), ("l0.mix.g", (192, 128)),
                     ("l0.mix.o", (128, 192)), ("l0.mlp.gate", (200, 128)), ("l0.mlp.up", (200, 128)),
                     ("l0.mlp.down", (128, 200)), ("l1.mix.q", (256, 128)), ("l1.mix.q.b", (256,)), ("l1.mix.k", (64, 128)),
                     ("l1.mix.k.b", (64,)), ("l1.mix.q.norm", (64,)), ("l1.mix.k.norm", (64,)), ("l1.mix.o", (128, 256))):
        assert tuple(names[n].shape) == shape, n
    for absent in ("l1.mix.v", "l1.mix.v.b", "l1.mix.sink", "l1.mix.g", "l0.mix.dq", "l4.mlp.gate", "l0.norm2", "head"):
        assert absent not in names, absent
    att, lat = spec.layers[1].mixer, spec.layers[0].mixer
    assert att.options["values"] == "keys" and att.options["sink"] == "zero" and att.bias and att.position.kind == "none"
    assert att.options["distance_bias"] == 8.0 and att.options["qk_norm"] == "head_first" and att.scale == 0.12
    assert lat.options["sink"] is True and lat.options["gate"] == "sigmoid" and lat.position.theta == 10000.0
    assert conf.to_dict() == LC.config("B")


def test_a_model_without_a_run_of_layers():
    for loop in ("absent", None):
        cfg = LC.config("D")
        cfg.pop("loop", None)
        if loop is None:
            cfg["loop"] = None
        spec = config_from_dict(cfg).model_spec()
        assert spec.schedule == (0, 1, 2) and not spec.place_hooks and "loop.step" not in declare_parameters(spec)


def test_a_run_of_layers_at_the_first_layer():
    spec = config_from_dict(LC.config("A")).model_spec()
    assert spec.schedule == (0, 1, 0, 1, 0, 1, 2, 3) and sorted(spec.place_hooks) == [0, 2, 4]
    assert declare_parameters(spec)["loop.step"].shape == (3, 72)


def test_the_embedding_state_is_a_place_behind_the_schedule():
    spec = config_from_dict(LC.config("A")).model_spec()
    model = Model(spec, torch.float32, torch.device("cpu"))
    kv, reads, state = model.cache_plan()
    assert len(kv) == len(reads) == len(state) == len(spec.schedule) + 1
    assert kv[-1] is None and reads[-1] is None and state[-1] == StateNeed((1,), torch.int32)
    assert all(need is not None for need in kv[:-1])
    assert kv[1].values_are_keys and not kv[0].values_are_keys and model.keeps_embedding
    plain = Model(config_from_dict(LC.config("D")).model_spec(), torch.float32, torch.device("cpu"))
    assert not plain.keeps_embedding


@pytest.mark.parametrize("path,value,word", [
    (("vocab",), 0, "vocab"), (("norm",), 3, "norm"), (("embedding",), None, "embedding"),
    (("embedding", "bigram"), None, "bigram"), (("embedding", "bigram", "buckets"), 0, "buckets"),
    (("embedding", "bigram", "mul_prev"), -1, "mul_prev"), (("embedding", "bigram", "mul_cur"), 1.5, "mul_cur"),
    (("layers", 0, "type"), "mamba1", "type"), (("layers", 0, "mixer", "heads"), 5, "kv_heads"),
    (("layers", 0, "mixer", "vdim"), 12, "vdim"), (("layers", 0, "mixer", "scale"), 0.0, "scale"),
    (("layers", 1, "mixer", "rot_dim"), 5, "rot_dim"), (("layers", 1, "mixer", "rot", "dims"), 4, "rot.dims"),
    (("layers", 1, "mixer", "rot", "base"), -2.0, "base"), (("layers", 1, "mixer", "kv_rank"), None, "kv_rank"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"), (("layers", 0, "mlp", "ff"), 0, "ff"),
    (("loop", "stop"), 5, "loop"), (("loop", "start"), 2, "loop"), (("loop", "times"), 0, "times"), (("layers",), [], "layers"),
])
def test_refusals_name_the_key(path, value, word):
    cfg = LC.config("A")
    d = cfg
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert word in str(e.value)


def test_plain_rows_of_pairs():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 2}
    assert P.pair_rows([4, 5, 9], None, b) == [10, (12 + 10) % 10, (15 + 18) % 10]
    assert P.pair_rows([5, 9], 4, b) == P.pair_rows([4, 5, 9], None, b)[1:]


def test_plain_softmax_with_a_sink():
    s = torch.tensor([[1.0, 2.0, 3.0]])
    seen = torch.tensor([[True, True, False]])
    e = [math.exp(1.0), math.exp(2.0)]
    got = P.softmax_with_sink(s, seen, torch.tensor(0.5))[0].tolist()
    den = sum(e) + math.exp(0.5)
    assert got == pytest.approx([e[0] / den, e[1] / den, 0.0], rel=1e-6)


def test_plain_slopes_and_rotation():
    assert P.distance_slopes(8) == [2.0 ** -(h + 1) for h in range(8)]
    assert P.distance_slopes(3)[0] == pytest.approx(2.0 ** (-8.0 / 3.0))
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0]]])
    got = P.rotate_halves(x, torch.tensor([5]), 100.0)[0, 0]
    for i, f in ((0, 1.0), (1, 0.1)):
        u, v, a = x[0, 0, i].item(), x[0, 0, i + 2].item(), 5 * f
        assert got[i].item() == pytest.approx(u * math.cos(a) - v * math.sin(a), abs=1e-5)
        assert got[i + 2].item() == pytest.approx(v * math.cos(a) + u * math.sin(a), abs=1e-5)


def test_plain_attention_sees_the_raw_key_as_its_value():
    """One token: the weight of its own key is e^s / (1 + e^s), and what it weighs is the key before its norm."""
    D, d = 4, 6
    g = torch.Generator().manual_seed(0)
    w = {n: torch.randn(*s, generator=g) for n, s in (("q", (D, d)), ("q.b", (D,)), ("k", (D, d)), ("k.b", (D,)),
                                                      ("q.norm", (D,)), ("k.norm", (D,)))}
    h = torch.randn(1, d, generator=g)
    m = {"heads": 1, "kv_heads": 1, "dim": D, "vdim": D, "scale": 0.5}
    got = P.biased_attention(P.Plain(), h, w, m, 1e-5, None, 0)
    q, k = h @ w["q"].t() + w["q.b"], h @ w["k"].t() + w["k.b"]
    s = (P.rms_norm(q, w["q.norm"], 1e-5) * P.rms_norm(k, w["k.norm"], 1e-5)).sum() * 0.5
    torch.testing.assert_close(got, torch.sigmoid(s) * k)
