"""The Mopilorn configuration reader: its layout, the names and shapes of tensors, dimensions the file gives, refusals that
name the key, and what the plain parts do on known answers (no GPU)."""
import copy
import json
import math
import os

import pytest
import torch

import mopilorn_cases as MC
import plain_mopilorn as pm


def spec_of(cfg):
    from ziglm_b200 import config_from_dict
    return config_from_dict(cfg).model_spec()


def declared(cfg):
    from ziglm_b200.engine.model import declare_parameters
    return {k: tuple(v.shape) for k, v in declare_parameters(spec_of(cfg)).items()}


def test_layout_and_tensor_names():
    cfg = MC.config("A")
    spec = spec_of(cfg)
    assert spec.architecture == "Mopilorn" and spec.schedule == (0, 1, 2, 3) and spec.streams == 3
    assert spec.head_name == "head" and spec.logits_hook.kind == "soft_cap" and spec.logits_hook.options["cap"] == 12.0
    assert [layer.ffn is None for layer in spec.layers] == [False, True, False, True]
    d = declared(cfg)
    assert d["embed"] == d["head"] == (157, 72) and d["final.norm"] == (72,)
    assert d["l0.hc1.in"] == d["l0.hc2.out"] == (3,) and d["l2.hc2.mix"] == (3, 3) and "l1.hc2.in" not in d and "l1.norm2" not in d
    assert d["l0.mix.a1"] == (9, 72) and d["l0.mix.a2"] == (36, 9) and d["l0.mix.g1"] == (5, 72) and d["l0.mix.g2"] == (60, 5)
    assert d["l0.mix.dt_bias"] == (36,) and d["l0.mix.A_log"] == (3,) and d["l0.mix.norm"] == (20,) and d["l0.mix.o"] == (72, 60)
    assert d["l1.mix.left.q"] == (144, 72) and d["l1.mix.left.v.conv"] == (80, 3) and d["l1.mix.left.o"] == (72, 240)
    assert d["l1.mix.right.k"] == (20, 72) and d["l1.mix.right.v.conv"] == (56, 5) and d["l1.mix.right.a"] == (4, 72)
    assert d["l1.mix.right.g"] == (56, 72) and d["l1.mix.left.out"] == d["l1.mix.right.out"] == (72,)
    assert not any(".weight" in name for name in d)


def test_no_cap_no_mask_no_scaling():
    cfg = MC.config("C")
    assert spec_of(cfg).logits_hook is None
    left = spec_of(MC.config("A")).layers[2].mixer.options["parts"][0][1]
    assert left.window is None and left.position.scaling is None
    cfg = MC.config("A")
    cfg["layers"][1]["mixer"]["left"]["mask"] = None
    cfg["layers"][1]["mixer"]["left"]["rot"]["scaling"] = None
    left = spec_of(cfg).layers[1].mixer.options["parts"][0][1]
    assert left.window is None and left.position.scaling is None


def test_ranks_are_the_files_where_the_configuration_does_not_give_them(tmp_path):
    from ziglm_b200 import config_from_dict, write_random_model
    from ziglm_b200.engine.model import declare_parameters
    from ziglm_b200.weights import WeightError, load_tensors
    cfg = MC.config("A")
    folder = str(tmp_path / "m")
    write_random_model(folder, config_from_dict(cfg), 3)
    bare = copy.deepcopy(cfg)
    for layer in bare["layers"]:
        for key in ("decay_rank", "gate_rank"):
            layer["mixer"].pop(key, None)
    shapes = declare_parameters(config_from_dict(bare).model_spec())
    w = load_tensors(folder, shapes, torch.float32, torch.device("cpu"))
    assert tuple(w["l0.mix.a1"].shape) == (9, 72) and tuple(w["l3.mix.g2"].shape) == (54, 12)
    bare["layers"][0]["mixer"]["decay_rank"] = 8                # given, and not what the file has
    with pytest.raises(WeightError) as e:
        load_tensors(folder, declare_parameters(config_from_dict(bare).model_spec()), torch.float32, torch.device("cpu"))
    assert "l0.mix.a1" in str(e.value)
    bare["layers"][0]["mixer"].pop("decay_rank")
    bare["width"] = 80                                          # the other dimension is still checked
    with pytest.raises(WeightError):
        load_tensors(folder, declare_parameters(config_from_dict(bare).model_spec()), torch.float32, torch.device("cpu"))


def _set(cfg, path, value):
    at = cfg
    for p in path[:-1]:
        at = at[p]
    if value is KeyError:
        del at[path[-1]]
    else:
        at[path[-1]] = value


@pytest.mark.parametrize("path,value,says", [
    (("streams",), KeyError, "streams"), (("streams",), 0, "streams"), (("norm", "eps"), 0, "norm.'eps'"),
    (("vocab",), "9", "vocab"), (("logit_softcap",), -1.0, "logit_softcap"), (("layers",), [], "layers"),
    (("layers", 0, "type"), "mamba1", "layers[0].type"), (("layers", 0, "mixer", "vdim"), KeyError, "layers[0].mixer.'vdim'"),
    (("layers", 0, "mixer", "kv_heads"), 2, "layers[0].mixer.heads"), (("layers", 1, "mixer", "left"), None, "'left'"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 15, "left.rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 26, "left.rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "scaling", "low"), KeyError, "rot.scaling.'low'"),
    (("layers", 1, "mixer", "left", "mask", "size"), 0, "mask.'size'"),
    (("layers", 1, "mixer", "right", "conv"), 0, "right.'conv'"), (("layers", 0, "mlp", "kind"), "moe", "mlp.kind"),
    (("layers", 0, "mixer", "gate_rank"), 0, "gate_rank")])
def test_refusals_name_the_key(path, value, says):
    from ziglm_b200 import ConfigError, config_from_dict
    cfg = MC.config("A")
    _set(cfg, path, value)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert says in str(e.value)


def test_config_round_trip(tmp_path):
    from ziglm_b200 import config_from_dict, config_from_folder
    cfg = MC.config("B")
    os.makedirs(tmp_path / "m")
    with open(tmp_path / "m" / "config.json", "w") as f:
        json.dump(cfg, f)
    conf = config_from_folder(str(tmp_path / "m"))
    assert conf.to_dict() == cfg and conf.model_spec() == config_from_dict(cfg).model_spec()


def test_hooks_on_the_residual_do_not_go_with_streams():
    from dataclasses import replace
    from ziglm_b200.config.spec import HookSpec
    spec = spec_of(MC.config("A"))
    with pytest.raises(ValueError):
        replace(spec, embed_hook=HookSpec("scale", {"factor": 2.0}))


# ------------------------------------------------------------- the plain parts on known answers
def test_plain_frequencies_stay_are_blended_and_are_divided():
    from ziglm_b200.parts.rope import inverse_frequencies
    rot = {"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 1024}}
    f, bare = pm.frequencies(rot), pm.frequencies({"dims": 32, "base": 10000.0})
    kinds = set()
    for a, b in zip(f, bare):
        wave = 2 * math.pi / b
        kinds.add("stays" if wave < 256 else "divided" if wave > 1024 else "blended")
        assert a == b if wave < 256 else (a == b / 8 if wave > 1024 else b / 8 < a < b)
    assert kinds == {"stays", "divided", "blended"}
    table = inverse_frequencies(32, 10000.0, {"rope_type": "llama3", "factor": 8.0, "low_freq_factor": 1.0,
                                              "high_freq_factor": 4.0, "original_max_position_embeddings": 1024})
    assert torch.allclose(table, torch.tensor(f), rtol=1e-6)


def test_plain_delta_rule_replaces_what_a_key_holds():
    """With a write strength of one and no decay, writing a value under a unit key makes the state return exactly it."""
    q = torch.eye(3).reshape(3, 1, 3)
    k = torch.stack([torch.eye(3)[0], torch.eye(3)[1], torch.eye(3)[0]]).reshape(3, 1, 3)
    v = torch.tensor([[1.0, 2.0], [3.0, 4.0], [-5.0, 6.0]]).reshape(3, 1, 2)
    o, S = pm.delta_rule(q, k, v, torch.ones(3, 1), torch.ones(3, 1, 3), torch.zeros(1, 3, 2))
    assert torch.equal(o[:, 0], torch.tensor([[1.0, 2.0], [3.0, 4.0], [0.0, 0.0]]))
    assert torch.equal(S[0], torch.tensor([[-5.0, 6.0], [3.0, 4.0], [0.0, 0.0]]))
    _, S = pm.delta_rule(q, k, v, torch.ones(3, 1), torch.tensor([1.0, 0.5, 0.0]).expand(3, 1, 3), torch.zeros(1, 3, 2))
    assert torch.equal(S[0], torch.tensor([[-5.0, 6.0], [1.5, 2.0], [0.0, 0.0]]))


def test_plain_streams_use_the_old_ones_for_all():
    x = torch.tensor([[[1.0]], [[10.0]]])
    hc = {"in": torch.tensor([2.0, 0.5]), "out": torch.tensor([1.0, -1.0]), "mix": torch.tensor([[0.0, 1.0], [3.0, 0.0]])}
    assert pm.gather_streams(x, hc).item() == 7.0
    assert pm.spread_streams(x, torch.tensor([[100.0]]), hc).flatten().tolist() == [130.0, -99.0]


def test_plain_convolution_and_window():
    p = pm.Plain()
    x = torch.tensor([[1.0], [2.0], [3.0], [4.0]])
    w = torch.tensor([[100.0, 10.0, 1.0]])
    past = {}
    whole = pm.short_conv(p, x, w, None, "q")
    assert whole.flatten().tolist() == [1.0, 12.0, 123.0, 234.0]
    parts = torch.cat([pm.short_conv(p, x[:1], w, past, "q"), pm.short_conv(p, x[1:], w, past, "q")])
    assert torch.equal(parts, whole)
    i = torch.arange(5)
    assert pm.in_window(i, i, 2).sum().item() == 9 and pm.in_window(i, i, None).sum().item() == 15
