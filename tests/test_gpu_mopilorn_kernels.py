"""The kernels of the Mopilorn design against plain statements of the same operation: the gated delta rule (prompts,
portions, single tokens, batches of unequal sequences, decays of zero, one and in between, a decay a head and one a key
channel), the convolution that keeps its own inputs, residual streams, and the cap on the logits."""
from types import SimpleNamespace

import pytest
import torch

import plain_mopilorn as pm

pytestmark = pytest.mark.gpu
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def step_of(past, new, slots):
    """The parts of a step the kernels read: ``past`` and ``new`` tokens of every sequence, and its slot."""
    from ziglm_b200.engine.workspace import Workspace
    dev = torch.device("cuda:0")
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    cu = [0]
    for n in new:
        cu.append(cu[-1] + n)
    return SimpleNamespace(
        n_tokens=cu[-1], n_seqs=len(new), single_token=all(n == 1 for n in new), max_new=max(new), cu_seqlens=i32(cu),
        past_lens=i32(past), slots=i32(slots), seq_of_token=i32([b for b, n in enumerate(new) for _ in range(n)]),
        positions=i32([p + i for p, n in zip(past, new) for i in range(n)]), ws=Workspace(dev), cu=cu)


class Rule:
    """A delta rule with random operands for whole sequences, its plain result, and a way to run tokens of them."""

    def __init__(self, H, G, D, V, K, per_channel, dn, lens, seed=0, rate=1.0, n_slots=None):
        gen = torch.Generator().manual_seed(seed)
        r = lambda *s: torch.randn(*s, generator=gen)
        self.H, self.G, self.D, self.V, self.K, self.dn, self.dt = H, G, D, V, K, dn, DTYPES[dn]
        self.C = 2 * G * D + H * V
        per = H * D if per_channel else H
        self.x = [r(n, self.C).to(self.dt) for n in lens]
        self.a, self.b = [r(n, per) for n in lens], [r(n, H) for n in lens]
        self.taps, self.rate, self.bias = r(K, self.C) * 0.5, torch.rand(H, generator=gen) * rate, r(per)
        self.norm, self.gate = torch.rand(V, generator=gen) + 0.5, [r(n, H * V).to(self.dt) for n in lens]
        dev = "cuda:0"
        from ziglm_b200 import kernels
        self.n_slots = n_slots or len(lens)
        self.ring = torch.zeros(self.n_slots, K, self.C, device=dev)
        self.state = torch.zeros(self.n_slots, H, V, kernels.delta_state_size(D), device=dev)
        self.dev = {k: v.to(dev).contiguous() for k, v in (("taps", self.taps), ("rate", self.rate), ("bias", self.bias),
                                                           ("norm", self.norm))}
        self.want, self.end = zip(*[self.plain(i) for i in range(len(lens))])

    def plain(self, i):
        """o [n, H V] and the state [H, D, V] behind the sequence, in float64."""
        H, G, D, V = self.H, self.G, self.D, self.V
        p = pm.Plain(torch.float32, wide=True)
        x = self.x[i].double()
        y = pm.silu(pm.short_conv(p, x, self.taps.t().double(), None, ""))
        n = x.shape[0]
        share = torch.arange(H) // (H // G)
        q = (pm.unit_vector(y[:, :G * D].reshape(n, G, D)) * D ** -0.5)[:, share]
        k = pm.unit_vector(y[:, G * D:2 * G * D].reshape(n, G, D))[:, share]
        v = y[:, 2 * G * D:].reshape(n, H, V)
        stepsize = pm.softplus(self.a[i].double() + self.bias.double()).reshape(n, H, -1)
        g = torch.exp(-self.rate.double()[None, :, None] * stepsize).expand(n, H, D)
        o, S = pm.delta_rule(q, k, v, torch.sigmoid(self.b[i].double()), g, torch.zeros(H, D, V, dtype=torch.float64))
        return o.reshape(n, H * V), S

    def run(self, parts, decode=False):
        """parts: (sequence, slot, first, count).  The rows of the step, per sequence; decode: through the single-token kernel,
        normed and gated."""
        from ziglm_b200 import kernels
        step = step_of([f for _, _, f, _ in parts], [n for _, _, _, n in parts], [s for _, s, _, _ in parts])
        cat = lambda rows: torch.cat([rows[i][f:f + n] for i, _, f, n in parts]).to("cuda:0").contiguous()
        d = self.dev
        args = (cat(self.x), d["taps"], self.ring, self.H, self.G, self.D, self.V, cat(self.a), cat(self.b), d["rate"],
                d["bias"], self.state, step)
        if decode:
            out = torch.empty(step.n_tokens, self.H * self.V, dtype=self.dt, device="cuda:0")
            kernels.delta_rule_decode(*args, d["norm"], 1e-5, cat(self.gate), "silu", out)
        else:
            out = torch.empty(step.n_tokens, self.H * self.V, device="cuda:0")
            kernels.delta_rule(*args, out)
        torch.cuda.synchronize()
        return [out[step.cu[j]:step.cu[j + 1]].float().cpu() for j in range(len(parts))]

    def gated(self, i, rows):
        """The plain normed and gated rows of sequence i."""
        o = self.want[i][rows].reshape(-1, self.H, self.V)
        o = (pm.rms_unit(o, 1e-5) * self.norm.double()).reshape(-1, self.H * self.V)
        return o * pm.silu(self.gate[i][rows].double())


def close(got, want, tol, what=""):
    got, want = got.double(), want.double()
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-6)
    assert err == err and err < tol, f"{what}: {err:.3g}"


SHAPES = [(6, 2, 24, 40, 4, False), (6, 2, 24, 40, 4, True), (3, 3, 10, 7, 3, True), (2, 1, 130, 36, 2, False),
          (2, 2, 130, 36, 5, True), (4, 4, 128, 128, 4, True), (4, 2, 128, 64, 4, False), (1, 1, 1, 1, 1, True),
          (2, 2, 300, 20, 11, True), (2, 1, 64, 96, 4, False)]


@pytest.mark.parametrize("dn", list(DTYPES))
@pytest.mark.parametrize("shape", SHAPES, ids=[f"H{s[0]}G{s[1]}D{s[2]}V{s[3]}K{s[4]}{'c' if s[5] else 'h'}" for s in SHAPES])
def test_delta_rule_whole_sequences_portions_and_single_tokens(shape, dn):
    H, G, D, V, K, ch = shape
    lens = [45, 1, 8, 17, 2]
    rule = Rule(H, G, D, V, K, ch, dn, lens, seed=D)
    for i, got in enumerate(rule.run([(i, i, 0, n) for i, n in enumerate(lens)])):
        close(got, rule.want[i], 2e-5, f"sequence {i} of the batch")
    for i in range(len(lens)):
        close(rule.state[i].transpose(1, 2)[:, :D].cpu(), rule.end[i], 2e-5, f"state {i}")
    # the same tokens in other slots, in portions, with another sequence going on in the same steps
    rule.ring.zero_(); rule.state.zero_()
    at, rows = 0, []
    for n, m in ((2, 3), (9, 2), (1, 1), (8, 4), (16, 5)):
        a, b = rule.run([(0, 3, at, n), (3, 1, sum(c for c in (3, 2, 1, 4, 5)[:len(rows)]), m)])
        close(b, rule.want[3][sum((3, 2, 1, 4, 5)[:len(rows)]):][:m], 2e-5, "the other sequence")
        rows.append(a)
        at += n
    close(torch.cat(rows), rule.want[0][:at], 2e-5, "portions")
    # and on with single tokens, normed and gated
    tol = 2e-5 if dn == "float32" else 1e-2
    for t in range(at, lens[0]):
        a, = rule.run([(0, 3, t, 1)], decode=True)
        close(a, rule.gated(0, slice(t, t + 1)), tol, f"token {t}")
    close(rule.state[3].transpose(1, 2)[:, :D].cpu(), rule.end[0], 2e-5, "state behind portions and single tokens")


@pytest.mark.parametrize("ch", [False, True])
def test_delta_rule_decays_that_vanish_and_decays_of_one(ch):
    """Rates so large that decays underflow to zero inside a chunk, and of zero: no quotient of decays may turn up."""
    for rate in (2000.0, 30.0, 0.0):
        rule = Rule(4, 2, 32, 24, 4, ch, "float32", [61], rate=rate, seed=3)
        got, = rule.run([(0, 0, 0, 61)])
        close(got, rule.want[0], 3e-5, f"rate {rate}")
        assert torch.isfinite(rule.state).all()


def test_a_long_sequence_agrees_with_the_rule_stepped_token_by_token():
    rule = Rule(2, 1, 64, 32, 4, True, "float32", [1200], rate=0.02, seed=5)
    got, = rule.run([(0, 0, 0, 1200)])
    close(got, rule.want[0], 5e-5, "1200 tokens")
    close(rule.state[0].transpose(1, 2).cpu(), rule.end[0], 5e-5, "its state")


def test_single_tokens_of_a_batch_share_the_channels_of_q_and_k():
    """Eight heads over one head of q and k, many steps: the convolution's inputs are read and written by all of them."""
    rule = Rule(8, 1, 48, 16, 4, False, "float32", [30, 30, 30], seed=9)
    for t in range(30):
        for i, got in enumerate(rule.run([(i, 2 - i, t, 1) for i in range(3)], decode=True)):
            close(got, rule.gated(i, slice(t, t + 1)), 2e-5, f"sequence {i}, token {t}")


@pytest.mark.parametrize("dn", list(DTYPES))
@pytest.mark.parametrize("H,G,D,V,d,r,ch", [(3, 3, 20, 28, 96, 8, True), (4, 2, 128, 128, 256, 128, True),
                                            (4, 1, 40, 24, 520, 0, False), (2, 2, 64, 64, 64, 40, True)])
def test_single_tokens_with_the_products_before_decays_and_gate_in_the_kernel(H, G, D, V, d, r, ch, dn):
    """The same step with a, b and the gate made before and with their products left to the kernel."""
    from ziglm_b200 import kernels
    dt, dev = DTYPES[dn], "cuda:0"
    gen = torch.Generator().manual_seed(D)
    n = lambda *s: (torch.randn(*s, generator=gen) * 0.3).to(dt).to(dev)
    B, K, C = 3, 4, 2 * G * D + H * V
    per = H * D if ch else H
    at = -(-C // 8) * 8
    proj, h = n(B, at + 2 * r), n(B, d)
    w_b, w_a, w_a2, w_g2 = n(H, d), n(H, d), n(H * D, r), n(H * V, r)
    taps, rate, bias = n(K, C).float(), torch.rand(H, generator=gen).to(dev), n(per).float()
    norm = torch.ones(V, device=dev)
    outs = []
    for inside in (False, True):
        ring = torch.zeros(B, K, C, device=dev)
        state = torch.linspace(-1, 1, B * H * V * kernels.delta_state_size(D), device=dev).view(B, H, V, -1).contiguous()
        if D % 4:
            state[..., D:] = 0
        out = torch.empty(B, H * V, dtype=dt, device=dev)
        step = step_of([5] * B, [1] * B, [2, 0, 1])
        f = lambda w, x: (x.float() @ w.float().t()).contiguous()
        a1, g1 = proj[:, at:at + r], proj[:, at + r:at + 2 * r]
        if ch:
            kw = dict(h=h, w_b=w_b, a2=(w_a2, at), g2=(w_g2, at + r)) if inside else {}
            rows = (None, None) if inside else (f(w_a2, a1), f(w_b, h))
            gate, kind = (None if inside else f(w_g2, g1).to(dt)), "sigmoid"
        else:
            kw = dict(h=h, w_b=w_b, w_a=w_a) if inside else {}
            rows = (None, None) if inside else (f(w_a, h), f(w_b, h))
            gate, kind = n(B, H * V) * 0 + 0.5, "silu"
        kernels.delta_rule_decode(proj, taps, ring, H, G, D, V, *rows, rate, bias, state, step, norm, 1e-5, gate, kind, out, **kw)
        outs.append((out.float().cpu(), state.cpu()))
    close(outs[1][0], outs[0][0], 2e-5 if dn == "float32" else 2e-2, "rows")
    close(outs[1][1], outs[0][1], 1e-5, "state")


@pytest.mark.parametrize("dn", list(DTYPES))
@pytest.mark.parametrize("C,K,act", [(40, 4, None), (13, 3, "silu"), (128, 1, None), (24, 12, None), (20, 2, "silu")])
def test_causal_conv_that_keeps_its_inputs(C, K, act, dn):
    from ziglm_b200 import kernels
    dt = DTYPES[dn]
    gen = torch.Generator().manual_seed(C)
    lens = [50, 3, 1, 20]
    wide = [torch.randn(n, C + 8, generator=gen).to(dt) for n in lens]
    taps = torch.randn(K, C, generator=gen)
    p = pm.Plain(torch.float32, wide=True)
    want = [pm.short_conv(p, x[:, :C].double(), taps.t().double(), None, "") for x in wide]
    if act:
        want = [pm.silu(w) for w in want]
    ring = torch.zeros(4, K, C, device="cuda:0")
    at = [0] * 4
    for news in ([30, 3, 0, 2], [2, 0, 1, 1], [1, 0, 0, 16], [1, 0, 0, 1], [16, 0, 0, 0]):
        live = [i for i in range(4) if news[i]]
        step = step_of([at[i] for i in live], [news[i] for i in live], [3 - i for i in live])
        x = torch.cat([wide[i][at[i]:at[i] + news[i]] for i in live]).to("cuda:0")
        y = torch.empty(x.shape[0], C, dtype=dt, device="cuda:0")
        kernels.causal_conv_ring(x[:, :C], taps.to("cuda:0"), ring, step, y, activation=act)
        ref = torch.cat([want[i][at[i]:at[i] + news[i]] for i in live])
        close(y.float().cpu(), ref, 1e-6 if dn == "float32" else 1e-2, f"{news}")
        for i in live:
            at[i] += news[i]
    assert at == lens


@pytest.mark.parametrize("s,d", [(1, 64), (2, 96), (3, 50), (4, 256), (5, 33), (7, 128)])
@pytest.mark.parametrize("dn", list(DTYPES))
def test_residual_streams(s, d, dn):
    from ziglm_b200 import kernels
    dt = DTYPES[dn]
    gen = torch.Generator().manual_seed(s * d)
    T = 9
    r = lambda *sh: torch.randn(*sh, generator=gen)
    x, y, y2 = r(T, s, d), r(T, d), r(T, d)
    hc = {"in": r(s), "out": r(s), "mix": r(s, s)}
    nin, w, w1, w2 = r(s), r(d), r(d), r(d)
    dev = lambda t: t.to("cuda:0").contiguous()
    tol = 3e-6 if dn == "float32" else 8e-3
    h = torch.empty(T, d, dtype=dt, device="cuda:0")
    kernels.stream_norm(dev(x.reshape(T, s * d)), s, dev(hc["in"]), dev(w), 1e-5, h)
    streams = x.double().permute(1, 0, 2)
    close(h.float().cpu(), pm.norm_plain(pm.gather_streams(streams, hc), w.double(), 1e-5), tol, "stream_norm")
    rows = torch.tensor([7, 0, 7], dtype=torch.int32, device="cuda:0")
    h3 = torch.empty(3, d, dtype=dt, device="cuda:0")
    kernels.stream_norm(dev(x.reshape(T, s * d)), s, None, dev(w), 1e-5, h3, rows=rows)
    close(h3.float().cpu(), pm.norm_plain(streams.sum(0), w.double(), 1e-5)[[7, 0, 7]], tol, "the sum's norm, chosen rows")
    coef = dev(torch.cat([hc["mix"].reshape(-1), hc["out"]]))
    for branches, out in (([y], y.double()),
                          ([y, y2], 0.5 * (pm.norm_plain(y.double(), w1.double(), 1e-5)
                                           + pm.norm_plain(y2.double(), w2.double(), 1e-5)))):
        for follow in (False, True):
            xs = dev(x.reshape(T, s * d))
            kernels.stream_mix(xs, s, coef, [dev(b) for b in branches], None if len(branches) == 1 else [dev(w1), dev(w2)],
                               1e-5, 0.5, nxt=(dev(nin), dev(w), 1e-5, h) if follow else None)
            new = pm.spread_streams(streams, out, hc)
            close(xs.reshape(T, s, d).cpu(), new.permute(1, 0, 2), 3e-6, f"stream_mix, {len(branches)} branches")
            if follow:
                close(h.float().cpu(), pm.norm_plain(pm.gather_streams(new, {"in": nin}), w.double(), 1e-5), tol, "next rows")
    table = r(11, d).to(dt)
    toks = torch.tensor([3, 10, 0, 3, 5, 5, 1, 2, 9], dtype=torch.int32, device="cuda:0")
    e = torch.empty(T, s * d, device="cuda:0")
    kernels.embed_streams(dev(table), toks, e, s, 1.5)
    assert torch.equal(e.cpu(), (table.float()[toks.long().cpu()] * 1.5).repeat(1, s))


def test_the_cap_on_the_logits():
    from ziglm_b200 import kernels
    z = torch.randn(5, 333) * 60
    for cap in (30.0, 1.5, 200.0):
        zd = z.to("cuda:0")
        kernels.soft_cap_(zd, cap)
        close(zd.cpu(), pm.soft_cap(z.double(), cap), 1e-6, f"cap {cap}")
