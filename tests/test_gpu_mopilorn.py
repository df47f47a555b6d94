"""The Mopilorn design through the engine against the plain implementation (tests/plain_mopilorn.py): whole prompts,
prompts then token by token, prompts in portions down to two tokens, unequal batches with slots and pages used again, a
key made to stand out just inside and just outside a window and hundreds of tokens away, a write of the delta rule that is
asked for hundreds of tokens later, states and convolutions that must start at zero, taps that reach over every cut, long
decoding, models of one kind of layer, greedy generation through ``Engine.generate``, and a replay through
``bin/trace_run``; in float32 and in bfloat16, at configurations that differ in every size."""
import json
import os

import pytest
import torch

import mopilorn_cases as MC
from helpers import random_tokens

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


class Zoo:
    """Engines and plain logits, made once per (configuration, type)."""

    def __init__(self):
        self.made = {}

    def get(self, name, dn):
        key = (name, dn)
        if key not in self.made:
            eng, cfg, w = MC.build(MC.config(name), 11, dn)
            reqs = [random_tokens(n, cfg["vocab"], 500 + n) for n in (1, 2, 63, 64, 65, 130, 201)]
            plain = MC.plain(cfg, w, dn)
            want = [plain.forward(r) for r in reqs]
            self.made[key] = (eng, cfg, w, reqs, want)
        return self.made[key]


@pytest.fixture(scope="module")
def zoo():
    return Zoo()


CASES = [(n, d) for n in ("A", "B", "C", "D") for d in DTYPES]


def run(eng, toks, cuts):
    """The tokens as one request in a slot of its own, in steps of the given sizes: the logits of all of them."""
    assert sum(cuts) == len(toks)
    s = eng.alloc_slot()
    rows, at = [], 0
    for n in cuts:
        part = toks[at:at + n]
        rows.append((eng.step([(s, part)]) if n == 1 else eng.step([(s, part)], [list(range(n))])).clone())
        at += n
    eng.free_slot(s)
    return torch.cat(rows)


@pytest.mark.parametrize("name,dn", CASES)
def test_whole_prompts_and_the_first_tokens(zoo, name, dn):
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    for r, wl in zip(reqs, want):          # lengths 1 and 2: the first tokens; 63, 64, 65: around a page border
        MC.rows_close(run(eng, r, [len(r)]), wl, dn, f"{name} whole, {len(r)} tokens")
    eng.cache.slots.check()


@pytest.mark.parametrize("name,dn", CASES)
def test_prompt_then_token_by_token(zoo, name, dn):
    """Decoded tokens cross every window's edge, pages behind a window are let go, states and taps are carried."""
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    for i, first in ((4, 1), (5, 60), (6, 127)):
        n = len(reqs[i])
        MC.rows_close(run(eng, reqs[i], [first] + [1] * (n - first)), want[i], dn, f"{name} {first} tokens then one by one")
    eng.cache.slots.check()


@pytest.mark.parametrize("name,dn", CASES)
def test_prompts_in_portions(zoo, name, dn):
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    for i, cuts in ((6, [2, 2, 3, 57, 2, 64, 1, 33, 37]), (5, [64, 2, 62, 2]), (4, [17, 48]), (2, [2] * 31 + [1])):
        MC.rows_close(run(eng, reqs[i], cuts), want[i], dn, f"{name} in portions {cuts}")


@pytest.mark.parametrize("name,dn", CASES)
def test_unequal_batches_with_slots_and_pages_used_again(zoo, name, dn):
    from test_gpu_model import run_batches
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    # batch after batch in the same few slots: a page's rows and a slot's states are what the last user left
    got = run_batches(eng, reqs, [[6, 0, 3], [5, 1], [2, 4]], [150 if len(r) > 150 else max(1, len(r) - k)
                                                              for r, k in zip(reqs, (0, 1, 3, 0, 32, 30, 0))])
    for i, wl in enumerate(want):
        MC.rows_close(got[i], wl, dn, f"{name} batched, request {i}")
    eng.cache.slots.check()
    assert eng.cache.slots.slots.n_held == 0


@pytest.mark.parametrize("name,dn", [("A", "float32"), ("B", "bfloat16"), ("C", "float32"), ("D", "bfloat16")])
def test_long_decoding(zoo, name, dn):
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    MC.rows_close(run(eng, reqs[6], [3] + [1] * 198), want[6], dn, f"{name} decoded for 198 tokens")


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_float32_logits_do_not_depend_on_the_batch_beyond_rounding(zoo, name):
    eng, cfg, w, reqs, want = zoo.get(name, "float32")
    r = reqs[5]
    whole = run(eng, r, [len(r)])
    s, other = eng.alloc_slot(), eng.alloc_slot()
    a = eng.step([(other, reqs[3]), (s, r[:70])], [[], list(range(70))]).clone()
    b = torch.cat([eng.step([(other, [1]), (s, [t])], [[], [0]]).clone() for t in r[70:]])
    eng.free_slot(s); eng.free_slot(other)
    # a prompt walks the delta rule in chunks, a decoded token alone: they agree to rounding, not to the bit
    assert (torch.cat([a, b]) - whole).abs().max().item() <= 5e-5 * whole.abs().max().item()


@pytest.mark.parametrize("dn", DTYPES)
def test_many_sequences_decode_as_few_do(dn):
    """More sequences in a step than take the small products inside the recurrence's kernel."""
    eng, cfg, w = MC.build(MC.config("B"), 13, dn, max_batch=24, max_tokens=24 * 64)
    plain = MC.plain(cfg, w, dn)
    reqs = [random_tokens(9 + i % 5, cfg["vocab"], 40 + i) for i in range(20)]
    slots = [eng.alloc_slot() for _ in reqs]
    eng.step([(s, r[:5]) for s, r in zip(slots, reqs)], [[] for _ in reqs])
    rows = [[] for _ in reqs]
    for t in range(5, 9):
        got = eng.step([(s, [r[t]]) for s, r in zip(slots, reqs)]).clone()
        for i in range(len(reqs)):
            rows[i].append(got[i])
    for i in (0, 7, 16, 19):
        MC.rows_close(torch.stack(rows[i]), plain.forward(reqs[i])[5:9], dn, f"sequence {i} of 20")


def _one_layer(layer, vocab=90, width=64, streams=2, cap=None):
    return {"architecture": "Mopilorn", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "streams": streams,
            "logit_softcap": cap, "layers": [layer]}


def _bare_streams(w):
    """Every stream the embedding, the sublayer's output added to each."""
    for name, t in w.items():
        if ".hc" in name:
            t.copy_({"in": torch.full_like(t, 1.0 / t.shape[0]), "out": torch.ones_like(t)}.get(
                name.rsplit(".", 1)[1], torch.eye(t.shape[0], device=t.device).to(t.dtype) if t.dim() == 2 else t))
        if name.endswith(("norm1", "left.out", "final.norm")):
            t.fill_(1.0)
        if name.endswith(".conv"):                       # the convolutions pass their input on
            t.zero_()
            t[:, -1] = 1.0


def _standing_out(window, heads=2, kv=1, dim=32, vdim=32):
    """One parallel layer whose attention's query and key are made from different halves of the input through the same
    matrix, and an embedding in which token 5's first half is token 7's second half: where token 5 asks, its score at a
    position that holds token 7 stands out (the rotation is kept to two dimensions that carry nothing; the delta rule beside
    the attention is weighted with zero)."""
    cfg = _one_layer(MC._par(MC._left(heads, kv, dim, vdim, 0.5, 3, 2, 10000.0, window), MC._delta(1, 1, 4, 4, 2), None))
    half = cfg["width"] // 2

    def tweak(w):
        _bare_streams(w)
        p = "l0.mix.left."
        w["l0.mix.right.out"].zero_()
        w[p + "q"][:, half:] = 0
        w[p + "k"][:, :half] = 0
        w[p + "k"][:dim, half:] = w[p + "q"][:dim, :half]
        for h in range(1, heads):
            w[p + "q"][h * dim:(h + 1) * dim, :half] = w[p + "q"][:dim, :half]
        for g in range(1, kv):
            w[p + "k"][g * dim:(g + 1) * dim] = w[p + "k"][:dim]
        for n in ("q", "k"):
            rows = w[p + n].view(-1, dim, w[p + n].shape[1])
            rows[:, :2] = 0
        w["embed"][5, :half] = w["embed"][7, half:]
        w["embed"][5, half:] = 0

    return cfg, tweak


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("window,dim,vdim", [(70, 32, 32), (64, 64, 64), (128, 24, 40), (65, 128, 64)])
def test_a_key_just_inside_and_just_outside_the_window(dn, window, dim, vdim):
    """The key that stands out is the oldest the asking token sees, or the one before it; asked from a prompt's last token,
    from a decoded token, and from a token decoded behind a window of decoded tokens."""
    cfg, tweak = _standing_out(window, dim=dim, vdim=vdim)
    eng, cfg, w = MC.build(cfg, 3, dn, tweak=tweak, max_seq_len=512)
    plain = MC.plain(cfg, w, dn)
    n = 3 * window
    filler = [t if t not in (5, 7) else 6 for t in random_tokens(n, cfg["vocab"], 9)]
    ask = n - 1
    for at, shows in ((ask - window + 1, True), (ask - window, False)):
        toks = list(filler)
        toks[at], toks[ask] = 7, 5
        want = plain.forward(toks)
        quiet = list(toks)
        quiet[at] = 6
        moved = (want[-1] - plain.forward(quiet)[-1]).abs().max() > 0.2 * want[-1].abs().max()
        assert bool(moved) == shows                       # the oracle itself: the key matters exactly inside the window
        for first in (ask, ask + 1, window + 3):
            got = run(eng, toks, [first] + [1] * (n - first))
            MC.rows_close(got[-1:], want[-1:], dn, f"key at {at}, prompt of {first}, last row")
            if dn == "float32":
                MC.rows_close(got, want, dn, f"key at {at}, prompt of {first}")
    eng.cache.slots.check()


@pytest.mark.parametrize("dn", DTYPES)
def test_a_key_hundreds_of_tokens_away_without_a_window(dn):
    cfg, tweak = _standing_out(None, heads=3, kv=3, dim=64, vdim=64)
    eng, cfg, w = MC.build(cfg, 5, dn, tweak=tweak, max_seq_len=1024)
    plain = MC.plain(cfg, w, dn)
    toks = [t if t not in (5, 7) else 6 for t in random_tokens(700, cfg["vocab"], 4)]
    toks[3], toks[-1] = 7, 5
    want = plain.forward(toks)
    quiet = list(toks)
    quiet[3] = 6
    assert (want[-1] - plain.forward(quiet)[-1]).abs().max() > 0.2 * want[-1].abs().max()
    for first in (699, 700, 300):
        MC.rows_close(run(eng, toks, [first] + [1] * (700 - first))[-1:], want[-1:], dn, f"far key, prompt of {first}")


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("kind", ["parallel", "channel_delta"])
def test_a_write_asked_for_hundreds_of_tokens_later(dn, kind):
    """Decays of nearly one and a token whose write is far stronger than every other's: what it wrote shows in the last row
    four hundred tokens later, in prompts, portions and decoding, and only with the state that was carried."""
    if kind == "parallel":
        cfg = _one_layer(MC._par(MC._left(1, 1, 4, 4, 0.5, 1, 2, 100.0, 4), MC._delta(2, 1, 32, 24, 2), None))
        p = "l0.mix.right."
    else:
        cfg = _one_layer(MC._chan(MC._delta(2, 2, 32, 24, 2, (4, 4)), None))
        p = "l0.mix."

    def tweak(w):
        _bare_streams(w)
        if kind == "parallel":
            w["l0.mix.left.out"].zero_()
        w[p + "A_log"].fill_(-9.0)                        # decays of about 1 - 1e-4
        w["embed"][:, 0] = -3.0                           # every token but one hardly writes
        w["embed"][7, 0] = 6.0
        w[p + "b"].zero_()
        w[p + "b"][:, 0] = 2.0

    eng, cfg, w = MC.build(cfg, 6, dn, tweak=tweak, max_seq_len=512)
    plain = MC.plain(cfg, w, dn)
    toks = [t if t != 7 else 6 for t in random_tokens(420, cfg["vocab"], 8)]
    toks[11] = 7
    want = plain.forward(toks)
    quiet = list(toks)
    quiet[11] = 6
    assert (want[-1] - plain.forward(quiet)[-1]).abs().max() > 0.1 * want[-1].abs().max()
    for cuts in ([420], [12, 408], [5, 7, 2, 300] + [1] * 106, [11] + [1] * 20 + [389]):
        got = run(eng, toks, cuts)
        MC.rows_close(got[-1:] if dn == "bfloat16" else got, want[-1:] if dn == "bfloat16" else want, dn, f"steps {cuts[:4]}")


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("kind", ["parallel", "channel_delta"])
def test_taps_reach_over_every_cut(dn, kind):
    """Convolutions that only look at their oldest tap: a kept input that is off by one place changes every row."""
    cfg = _one_layer(MC._par(MC._left(2, 1, 16, 16, 0.3, 5, 8, 100.0, 20), MC._delta(2, 2, 16, 16, 4), None) if kind == "parallel"
                     else MC._chan(MC._delta(3, 3, 16, 16, 5, (4, 4)), None))

    def tweak(w):
        MC.lively(w)
        for name, t in w.items():
            if name.endswith(".conv"):
                t.zero_()
                t[:, 0] = 1.0

    eng, cfg, w = MC.build(cfg, 7, dn, tweak=tweak)
    toks = random_tokens(60, cfg["vocab"], 3)
    want = MC.plain(cfg, w, dn).forward(toks)
    for cuts in ([60], [1] * 60, [2] * 30, [3, 1, 2, 1, 1, 4, 9, 1, 5, 33], [59, 1]):
        MC.rows_close(run(eng, toks, cuts), want, dn, f"steps {cuts[:6]}")


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("kind", ["parallel", "channel_delta"])
def test_states_start_at_zero_in_a_slot_used_before(dn, kind):
    """A second request in the slot of a first one must not see its state or the convolutions' kept inputs."""
    cfg = _one_layer(MC._par(MC._left(2, 2, 24, 40, 0.3, 4, 8, 100.0, 30), MC._delta(3, 3, 20, 12, 4), 40) if kind == "parallel"
                     else MC._chan(MC._delta(3, 1, 24, 40, 4, (6, 6)), 40), width=48)
    eng, cfg, w = MC.build(cfg, 8, dn, max_batch=1)
    plain = MC.plain(cfg, w, dn)
    a, b = random_tokens(150, cfg["vocab"], 1), random_tokens(77, cfg["vocab"], 2)
    s = eng.alloc_slot()
    eng.step([(s, a)])
    eng.free_slot(s)
    MC.rows_close(run(eng, b, [33, 2] + [1] * 42), plain.forward(b), dn, "states in a slot used before")
    s = eng.alloc_slot()
    eng.step([(s, a[:3])])
    eng.free_slot(s)
    MC.rows_close(run(eng, b[:4], [1] * 4), plain.forward(b[:4]), dn, "decoding from the first token")


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("kind", ["parallel", "channel_delta"])
def test_models_of_one_kind_of_layer(dn, kind):
    if kind == "parallel":
        layers = [MC._par(MC._left(4, 4, 8, 16, 0.4, 2, 4, 77.0, 6), MC._delta(2, 2, 64, 64, 4), None),
                  MC._par(MC._left(2, 1, 24, 64, 0.3, 4, 24, 1000.0, 33, (4.0, 1.0, 2.0, 50)), MC._delta(3, 1, 8, 24, 2), 24),
                  MC._par(MC._left(8, 8, 16, 8, 0.3, 3, 16, 1000.0), MC._delta(1, 1, 100, 12, 3), None)]
    else:
        layers = [MC._chan(MC._delta(2, 2, 64, 64, 4, (16, 8)), None), MC._chan(MC._delta(4, 2, 40, 24, 3, (5, 30)), 24),
                  MC._chan(MC._delta(1, 1, 200, 16, 2, (8, 8)), None)]
    cfg = {"architecture": "Mopilorn", "vocab": 120, "width": 56, "norm": {"eps": 1e-5}, "streams": 2, "logit_softcap": 9.0,
           "layers": layers}
    eng, cfg, w = MC.build(cfg, 17, dn)
    r = random_tokens(140, cfg["vocab"], 5)
    MC.rows_close(run(eng, r, [90] + [1] * 50), MC.plain(cfg, w, dn).forward(r), dn, f"{kind} layers only")


@pytest.mark.parametrize("dn", DTYPES)
def test_a_long_prompt_leaves_the_states_that_decoding_it_would(dn):
    layers = [MC._chan(MC._delta(2, 2, 64, 32, 4, (8, 8)), None),
              MC._par(MC._left(2, 1, 32, 32, 0.2, 4, 32, 10000.0, 200), MC._delta(2, 1, 32, 64, 4), None)]
    cfg = {"architecture": "Mopilorn", "vocab": 80, "width": 48, "norm": {"eps": 1e-5}, "streams": 3, "logit_softcap": 20.0,
           "layers": layers}
    eng, cfg, w = MC.build(cfg, 21, dn, max_tokens=2048, max_seq_len=1100)
    r = random_tokens(1010, cfg["vocab"], 6)
    want = MC.plain(cfg, w, dn).forward(r)
    s = eng.alloc_slot()
    rows = [eng.step([(s, r[:1000])], [[0, 500, 999]]).clone()] + [eng.step([(s, [t])]).clone() for t in r[1000:]]
    eng.free_slot(s)
    MC.rows_close(torch.cat(rows), torch.cat([want[[0, 500, 999]], want[1000:]]), dn, "a thousand tokens, then ten")


def test_side_by_side_mixers_norm_and_sum_their_outputs_for_other_blocks():
    """``forward`` of the side-by-side mixer, which a block that knows nothing of streams calls: half the sum of the two
    normed outputs, added to what is there."""
    eng, cfg, w = MC.build(MC.config("B"), 4, "float32")
    mixer = eng.model.blocks[0].mixer
    original, kept = mixer.forward_branches, {}

    def too(step, io, h):
        mixer.forward_branches = original
        kept["h"], kept["rows"] = h.clone(), torch.ones(h.shape[0], cfg["width"], device=h.device)
        mixer.forward(step, io, h, kept["rows"])
        return original(step, io, h)

    mixer.forward_branches = too
    s = eng.alloc_slot()
    eng.step([(s, random_tokens(30, cfg["vocab"], 2))])
    eng.free_slot(s)
    lw = {k[len("l0.mix."):]: v for k, v in w.items() if k.startswith("l0.mix.")}
    want = MC.plain(cfg, w, "float32").mixer("parallel", kept["h"].cpu(), lw, cfg["layers"][0]["mixer"], None, 0)
    assert (kept["rows"].cpu() - 1.0 - want).abs().max().item() < 2e-5 * want.abs().max().item() + 1e-6


@pytest.mark.parametrize("name,dn", [("A", "float32"), ("B", "bfloat16")])
def test_greedy_generation_through_the_entry_point(name, dn):
    from ziglm_b200 import GenerationOptions, SamplerParams
    eng, cfg, w = MC.build(MC.config(name), 5, dn)
    prompts = [random_tokens(n, cfg["vocab"], 70 + n) for n in (3, 40, 9)]
    results, stats = eng.generate(prompts, GenerationOptions(max_tokens=8, ignore_eos=True,
                                                             sampler=SamplerParams(greedy=True)))
    plain = MC.plain(cfg, w, dn)
    for p, r in zip(prompts, results):
        seq = list(p)
        assert len(r.tokens) == 8
        for tok in r.tokens:
            row = plain.forward(seq)[-1]
            slack = 0.0 if dn == "float32" else 0.05 * row.std().item()
            assert row.max().item() - row[tok].item() <= slack, f"token {tok} after {len(seq)} tokens"
            seq.append(tok)
    assert stats.completion_tokens == 24


def test_replay_from_a_folder(tmp_path):
    """A folder written by the library, without the ranks in its config.json, loaded by the name of the architecture and
    replayed by ``bin/trace_run``."""
    from safetensors.torch import load_file
    from test_gpu_replay import Replay
    from ziglm_b200 import config_from_dict, write_random_model
    from ziglm_b200.weights.safetensors_io import write_safetensors
    cfg = MC.config("B")
    folder = str(tmp_path / "model")
    write_random_model(folder, config_from_dict(cfg), 8, dtype=torch.bfloat16, std=0.12, norm_jitter=0.1, device="cuda")
    for layer in cfg["layers"]:
        for key in ("decay_rank", "gate_rank"):
            layer["mixer"].pop(key, None)
    json.dump(cfg, open(os.path.join(folder, "config.json"), "w"))
    w = {k: v.clone() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}
    MC.lively(w)
    write_safetensors(os.path.join(folder, "model.safetensors"), w)
    reqs = [random_tokens(n, cfg["vocab"], 30 + n) for n in (70, 9)]
    for dn in DTYPES:
        plain = MC.plain(cfg, w, dn)
        want = [plain.forward(r) for r in reqs]
        rp = Replay(folder, dn, str(tmp_path / ("logits_" + dn)), max_tokens=256)
        try:
            first = rp.step([{"id": "a", "tokens": reqs[0][:40], "want": list(range(40))},
                             {"id": "b", "tokens": reqs[1][:5], "want": [0, 4]}])
            MC.rows_close(first, torch.cat([want[0][:40], want[1][[0, 4]]]), dn, "replay, first step")
            for i in range(4):
                got = rp.step([{"id": "a", "tokens": [reqs[0][40 + i]], "want": [0]},
                               {"id": "b", "tokens": [reqs[1][5 + i]], "want": [0]}], end=["b"] if i == 3 else [])
                MC.rows_close(got, torch.stack([want[0][40 + i], want[1][5 + i]]), dn, f"replay, step {i + 1}")
            for i in range(44, 70):
                got = rp.step([{"id": "a", "tokens": [reqs[0][i]], "want": [0]}], end=["a"] if i == 69 else [])
                MC.rows_close(got, want[0][i:i + 1], dn, f"replay, token {i}")
        finally:
            rp.close()
