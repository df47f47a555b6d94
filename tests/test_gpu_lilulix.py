"""The Lilulix design through the engine against the plain implementation (tests/plain_lilulix.py): whole prompts, prompts
then token by token, prompts in portions down to two tokens, unequal batches with slots and pages used again, a key made to
stand out hundreds of tokens away in either kind of layer, sinks and biases that show, the token before a cut, the embedding
taken again before a pass, long decoding, models of one kind of layer, greedy generation through ``Engine.generate``, and a
replay through ``bin/trace_run``; in float32 and in bfloat16, at configurations that differ in every size."""
import json
import os

import pytest
import torch

import lilulix_cases as LC
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
            eng, cfg, w = LC.build(LC.config(name), 11, dn)
            reqs = [random_tokens(n, cfg["vocab"], 500 + n) for n in (1, 2, 63, 64, 65, 130, 201)]
            plain = LC.plain(cfg, w, dn)
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
        LC.rows_close(run(eng, r, [len(r)]), wl, dn, f"{name} whole, {len(r)} tokens")
    eng.cache.slots.check()


@pytest.mark.parametrize("name,dn", CASES)
def test_prompt_then_token_by_token(zoo, name, dn):
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    for i, first in ((4, 1), (5, 60), (6, 127)):
        n = len(reqs[i])
        LC.rows_close(run(eng, reqs[i], [first] + [1] * (n - first)), want[i], dn, f"{name} {first} tokens then one by one")
    eng.cache.slots.check()


@pytest.mark.parametrize("name,dn", CASES)
def test_prompts_in_portions(zoo, name, dn):
    """Every cut asks for the token before it, which the step no longer holds."""
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    for i, cuts in ((6, [2, 2, 3, 57, 2, 64, 1, 33, 37]), (5, [64, 2, 62, 2]), (4, [17, 48]), (2, [2] * 31 + [1])):
        LC.rows_close(run(eng, reqs[i], cuts), want[i], dn, f"{name} in portions {cuts}")


@pytest.mark.parametrize("name,dn", CASES)
def test_unequal_batches_with_slots_and_pages_used_again(zoo, name, dn):
    from test_gpu_model import run_batches
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    # batch after batch in the same few slots: a page's rows and a slot's last token are what the last user left
    got = run_batches(eng, reqs, [[6, 0, 3], [5, 1], [2, 4]], [150 if len(r) > 150 else max(1, len(r) - k)
                                                              for r, k in zip(reqs, (0, 1, 3, 0, 32, 30, 0))])
    for i, wl in enumerate(want):
        LC.rows_close(got[i], wl, dn, f"{name} batched, request {i}")
    eng.cache.slots.check()
    assert eng.cache.slots.slots.n_held == 0


@pytest.mark.parametrize("name,dn", [("A", "float32"), ("B", "bfloat16"), ("D", "bfloat16")])
def test_long_decoding(zoo, name, dn):
    eng, cfg, w, reqs, want = zoo.get(name, dn)
    LC.rows_close(run(eng, reqs[6], [3] + [1] * 198), want[6], dn, f"{name} decoded for 198 tokens")


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_float32_logits_do_not_depend_on_the_batch(zoo, name):
    eng, cfg, w, reqs, want = zoo.get(name, "float32")
    r = reqs[5]
    whole = run(eng, r, [len(r)])
    s, other = eng.alloc_slot(), eng.alloc_slot()
    a = eng.step([(other, reqs[3]), (s, r[:70])], [[], list(range(70))]).clone()
    b = torch.cat([eng.step([(other, [1]), (s, [t])], [[], [0]]).clone() for t in r[70:]])
    eng.free_slot(s); eng.free_slot(other)
    assert (torch.cat([a, b]) - whole).abs().max().item() <= 2e-6 * whole.abs().max().item()


@pytest.mark.parametrize("dn", DTYPES)
def test_many_sequences_decode_as_few_do(dn):
    """More rows in a decode step than a norm rides on the products for, beside steps in which it does."""
    eng, cfg, w = LC.build(LC.config("B"), 13, dn, max_batch=72, max_tokens=72 * 64)
    plain = LC.plain(cfg, w, dn)
    reqs = [random_tokens(9 + i % 5, cfg["vocab"], 40 + i) for i in range(70)]
    slots = [eng.alloc_slot() for _ in reqs]
    eng.step([(s, r[:5]) for s, r in zip(slots, reqs)], [[] for _ in reqs])
    rows = [[] for _ in reqs]
    for t in range(5, 9):
        n = 70 if t < 7 else 33
        got = eng.step([(s, [r[t]]) for s, r in zip(slots[:n], reqs[:n])]).clone()
        for i in range(n):
            rows[i].append(got[i])
    for i in (0, 7, 32, 69):
        LC.rows_close(torch.stack(rows[i]), plain.forward(reqs[i])[5:5 + len(rows[i])], dn, f"sequence {i} of 70")


# ------------------------------------------------------------- one mechanism that shows
def _bare(layers, width=64, vocab=90, loop=None):
    return LC._model(vocab, width, 1e-5, (31, 3, 2), loop, layers)


def _asks_across(kind, heads, dim, vdim=None):
    """One layer whose query and key are made from different halves of the input through the same matrix, and an embedding
    in which token 5's first half is token 7's second half: where token 5 asks, its score at a position that holds token 7
    stands out; every rotated part, pair row and bias is zero."""
    layer = _att_layer(heads, dim) if kind == "attention" else LC._lat(heads, dim, 2, vdim or dim, 48, 0.5, 10000.0, None)
    cfg = _bare([layer])
    half = cfg["width"] // 2

    def tweak(w):
        for name, t in w.items():
            if name in ("bigram", "l0.mix.sink") or name.endswith(".b"):
                t.zero_()
            if name.endswith(("norm1", ".norm")):
                t.fill_(1.0)
        w["embed"][5, :half] = w["embed"][7, half:]
        w["embed"][5, half:] = 0
        if kind == "attention":
            for h in range(heads):
                w["l0.mix.q"][h * dim:(h + 1) * dim] = w["l0.mix.q"][:dim]
            w["l0.mix.q"][:, half:] = 0
            w["l0.mix.k"][:, :half] = 0
            w["l0.mix.k"][:dim, half:] = w["l0.mix.q"][:dim, :half]
            return
        q = w["l0.mix.q"].view(heads, dim + 2, -1)
        q[:, dim:] = 0
        q[:, :, half:] = 0
        w["l0.mix.dkv"][48:] = 0
        # the latent is the second half of the input (and 16 elements of nothing), the unrotated key the query's mirror
        w["l0.mix.dkv"][:48] = 0
        for i in range(half):
            w["l0.mix.dkv"][i, half + i] = 1.0
        uk = w["l0.mix.uk"].view(heads, dim, 48)
        uk[:, :, half:] = 0
        uk[:, :, :half] = q[:, :dim, :half]
    return cfg, tweak


def _att_layer(heads, dim):
    return LC._att(heads, 1, dim, 3.0, None)


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("kind,heads,dim,back", [("latent_attention", 2, 24, 690), ("latent_attention", 3, 32, 630),
                                                 ("attention", 8, 32, 690), ("attention", 5, 64, 500), ("attention", 4, 128, 130)])
def test_a_key_far_away(dn, kind, heads, dim, back):
    """Asked for from a prompt's last token, from a decoded token, and from a token behind a run of decoded ones; it stands
    at the far end of a page and at the start of one as well.  In the biased layer the flat heads still see it."""
    cfg, tweak = _asks_across(kind, heads, dim)
    eng, cfg, w = LC.build(cfg, 5, dn, tweak=tweak, max_seq_len=1024)
    plain = LC.plain(cfg, w, dn)
    toks = [t if t not in (5, 7) else 6 for t in random_tokens(700, cfg["vocab"], 4)]
    ask = 699
    for at in (ask - back, (ask - back) // 64 * 64 + 64, (ask - back) // 64 * 64 + 63):
        seq = list(toks)
        seq[at], seq[ask] = 7, 5
        want = plain.forward(seq)
        quiet = list(seq)
        quiet[at] = 6
        moved = (want[-1] - plain.forward(quiet)[-1]).abs().max() / want[-1].abs().max()
        assert moved > 0.05, f"the oracle itself hardly sees the key ({moved:.3g})"
        for first in (699, 700, 680):
            LC.rows_close(run(eng, seq, [first] + [1] * (700 - first))[-1:], want[-1:], dn, f"far key at {at}, prompt of {first}")


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("kind", ["latent_attention", "attention"])
def test_the_denominators_extra_number(dn, kind):
    """Scores near zero, so that the first tokens' outputs are a fraction of what a plain softmax gives: the logits of the
    first tokens tell 1/2 of a value from all of it."""
    layer = LC._lat(3, 16, 4, 16, 24, 0.01, 100.0, None) if kind == "latent_attention" else LC._att(4, 2, 16, 0.01, None)
    cfg = _bare([layer], width=48)

    def tweak(w):
        LC.lively(w)
        if "l0.mix.sink" in w:
            w["l0.mix.sink"].copy_(torch.tensor([-1.0, 0.5, 3.0]))
        w["l0.mix.o"] *= 8.0 if kind == "latent_attention" else 0.15      # of the embedding's size: the final norm hides a common factor
    eng, cfg, w = LC.build(cfg, 9, dn, tweak=tweak)
    plain = LC.plain(cfg, w, dn)
    r = random_tokens(40, cfg["vocab"], 3)
    want = plain.forward(r)
    LC.rows_close(run(eng, r, [40]), want, dn, "prompt")
    LC.rows_close(run(eng, r, [1] * 40), want, dn, "token by token")
    import plain_lilulix
    kept = plain_lilulix.softmax_with_sink
    try:                                              # the oracle without the extra number is far away
        plain_lilulix.softmax_with_sink = lambda s, seen, sink: kept(s, seen, torch.tensor(float("-inf")))
        assert LC.row_errors(plain.forward(r)[:2], want[:2]).min().item() > 0.1
    finally:
        plain_lilulix.softmax_with_sink = kept


@pytest.mark.parametrize("dn", DTYPES)
def test_the_pair_row_of_every_token(dn):
    """An embedding that is all pair rows and layers that add nothing: a token's logits tell which row it took, at every cut
    of the sequence, in a batch, and in a slot used before."""
    cfg = LC._model(50, 64, 1e-5, (1009, 31, 17), (0, 1, 2), [LC._att(2, 1, 16, 0.3, None)])

    def tweak(w):
        w["l0.mix.o"].zero_()
        w["loop.step"].zero_()
        w["bigram"] *= 10.0
    eng, cfg, w = LC.build(cfg, 2, dn, tweak=tweak, max_batch=2)
    plain = LC.plain(cfg, w, dn)
    a, b = random_tokens(90, 50, 1), random_tokens(33, 50, 2)
    wa, wb = plain.forward(a), plain.forward(b)
    for cuts in ([90], [1] * 90, [2] * 45, [1, 64, 1, 1, 23], [3, 1, 86]):
        LC.rows_close(run(eng, a, cuts), wa, dn, f"steps {cuts[:5]}")
        LC.rows_close(run(eng, b, [1] * 33), wb, dn, "in the slot used before")
    s, t = eng.alloc_slot(), eng.alloc_slot()
    got = eng.step([(s, a[:20]), (t, b[:3])], [list(range(20)), [0, 1, 2]]).clone()
    LC.rows_close(got, torch.cat([wa[:20], wb[:3]]), dn, "two sequences")
    got = [eng.step([(t, [b[3 + i]]), (s, [a[20 + i]])]).clone() for i in range(6)]
    LC.rows_close(torch.cat(got), torch.stack([x for i in range(6) for x in (wb[3 + i], wa[20 + i])]), dn, "order turned round")
    eng.free_slot(s); eng.free_slot(t)


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("loop", [(0, 2, 1), (0, 2, 3), (1, 2, 4), (0, 1, 2)])
def test_passes_with_the_embedding_taken_again(dn, loop):
    """Vectors of a pass as large as the embedding, passes from one to four, against the oracle; and the oracle with the
    vectors of two passes exchanged is far away."""
    cfg = _bare([LC._lat(2, 16, 8, 16, 24, 0.25, 100.0, 40), LC._att(4, 2, 16, 0.3, 24)], width=48, loop=loop)

    def tweak(w):
        LC.lively(w)
        w["loop.step"].mul_(1.5)
    eng, cfg, w = LC.build(cfg, 21, dn, tweak=tweak)
    plain = LC.plain(cfg, w, dn)
    r = random_tokens(77, cfg["vocab"], 8)
    want = plain.forward(r)
    for cuts in ([77], [40, 2] + [1] * 35):
        LC.rows_close(run(eng, r, cuts), want, dn, f"loop {loop}, steps {cuts[:3]}")
    if loop[2] > 1:
        other = LC.plain(cfg, {**w, "loop.step": w["loop.step"].flip(0)}, dn).forward(r)
        assert LC.row_errors(other, want).median().item() > 0.1


@pytest.mark.parametrize("dn", DTYPES)
@pytest.mark.parametrize("kind", ["latent_attention", "attention"])
def test_models_of_one_kind_of_layer(dn, kind):
    if kind == "latent_attention":
        layers = [LC._lat(4, 16, 16, 8, 48, 0.2, 10000.0, None), LC._lat(1, 64, 2, 64, 126, 0.1, 5.0, 40),
                  LC._lat(17, 4, 4, 4, 12, 0.3, 77.0, 24)]
    else:
        layers = [LC._att(4, 4, 64, 0.1, None), LC._att(7, 1, 40, 0.2, 40), LC._att(16, 2, 128, 0.05, 24)]
    cfg = LC._model(120, 56, 1e-5, (77, 5, 9), (1, 3, 2), layers)
    eng, cfg, w = LC.build(cfg, 17, dn)
    r = random_tokens(140, cfg["vocab"], 5)
    LC.rows_close(run(eng, r, [90] + [1] * 50), LC.plain(cfg, w, dn).forward(r), dn, f"{kind} layers only")


@pytest.mark.parametrize("dn", DTYPES)
def test_a_long_prompt_leaves_the_cache_that_decoding_it_would(dn):
    cfg = LC._model(80, 64, 1e-5, (400, 3, 5), (0, 2, 2), [LC._lat(4, 32, 32, 32, 96, 0.15, 10000.0, 48), LC._att(6, 2, 64, 0.1, 48)])
    eng, cfg, w = LC.build(cfg, 21, dn, max_tokens=2048, max_seq_len=1100)
    r = random_tokens(1010, cfg["vocab"], 6)
    want = LC.plain(cfg, w, dn).forward(r)
    s = eng.alloc_slot()
    rows = [eng.step([(s, r[:1000])], [[0, 500, 999]]).clone()] + [eng.step([(s, [t])]).clone() for t in r[1000:]]
    eng.free_slot(s)
    LC.rows_close(torch.cat(rows), torch.cat([want[[0, 500, 999]], want[1000:]]), dn, "a thousand tokens, then ten")


# ------------------------------------------------------------------ entry points
@pytest.mark.parametrize("name,dn", [("A", "float32"), ("B", "bfloat16"), ("D", "bfloat16")])
def test_greedy_generation_through_the_entry_point(name, dn):
    from ziglm_b200 import GenerationOptions, SamplerParams
    eng, cfg, w = LC.build(LC.config(name), 5, dn)
    prompts = [random_tokens(n, cfg["vocab"], 70 + n) for n in (3, 40, 9)]
    results, stats = eng.generate(prompts, GenerationOptions(max_tokens=8, ignore_eos=True,
                                                             sampler=SamplerParams(greedy=True)))
    plain = LC.plain(cfg, w, dn)
    for p, r in zip(prompts, results):
        seq = list(p)
        assert len(r.tokens) == 8
        for tok in r.tokens:
            row = plain.forward(seq)[-1]
            slack = 1e-4 if dn == "float32" else 0.05 * row.std().item()
            assert row.max().item() - row[tok].item() <= slack, f"token {tok} after {len(seq)} tokens"
            seq.append(tok)
    assert stats.completion_tokens == 24


def test_replay_from_a_folder(tmp_path):
    """A folder written by the library, loaded by the name of the architecture and replayed by ``bin/trace_run``."""
    from safetensors.torch import load_file
    from test_gpu_replay import Replay
    from ziglm_b200 import config_from_dict, write_random_model
    from ziglm_b200.weights.safetensors_io import write_safetensors
    cfg = LC.config("B")
    folder = str(tmp_path / "model")
    write_random_model(folder, config_from_dict(cfg), 8, dtype=torch.bfloat16, std=0.12, norm_jitter=0.1, device="cuda")
    assert json.load(open(os.path.join(folder, "config.json")))["architecture"] == "Lilulix"
    w = {k: v.clone() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}
    LC.lively(w)
    write_safetensors(os.path.join(folder, "model.safetensors"), w)
    reqs = [random_tokens(n, cfg["vocab"], 30 + n) for n in (70, 9)]
    for dn in DTYPES:
        plain = LC.plain(cfg, w, dn)
        want = [plain.forward(r) for r in reqs]
        rp = Replay(folder, dn, str(tmp_path / ("logits_" + dn)), max_tokens=256)
        try:
            first = rp.step([{"id": "a", "tokens": reqs[0][:40], "want": list(range(40))},
                             {"id": "b", "tokens": reqs[1][:5], "want": [0, 4]}])
            LC.rows_close(first, torch.cat([want[0][:40], want[1][[0, 4]]]), dn, "replay, first step")
            for i in range(4):
                got = rp.step([{"id": "a", "tokens": [reqs[0][40 + i]], "want": [0]},
                               {"id": "b", "tokens": [reqs[1][5 + i]], "want": [0]}], end=["b"] if i == 3 else [])
                LC.rows_close(got, torch.stack([want[0][40 + i], want[1][5 + i]]), dn, f"replay, step {i + 1}")
            for i in range(44, 70):
                got = rp.step([{"id": "a", "tokens": [reqs[0][i]], "want": [0]}], end=["a"] if i == 69 else [])
                LC.rows_close(got, want[0][i:i + 1], dn, f"replay, token {i}")
        finally:
            rp.close()
