"""Each mechanism of the Lilulix design alone: the kernel against the plain function that states its formula
(tests/plain_lilulix.py), at sizes that are no multiple of a tile, with strided rows, several sequences in a step,
shuffled pages, prompts and decoded tokens, slots used again, and inputs made so that a fault shows."""
from types import SimpleNamespace

import pytest
import torch

import plain_lilulix as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
TYPES = [torch.float32, torch.bfloat16]


def _r(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(dtype).to(DEV)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _tol(dtype, f32=(1e-5, 1e-5), bf16=(2e-2, 2e-2)):
    a, r = f32 if dtype == torch.float32 else bf16
    return dict(atol=a, rtol=r)


def _step(pasts, news, slots, tokens=None):
    from ziglm_b200.engine.workspace import Workspace
    cu = [0]
    for n in news:
        cu.append(cu[-1] + n)
    pos = [p + i for p, n in zip(pasts, news) for i in range(n)]
    seq = [b for b, n in enumerate(news) for _ in range(n)]
    return SimpleNamespace(tokens=None if tokens is None else _i32(tokens), positions=_i32(pos), seq_of_token=_i32(seq),
                           cu_seqlens=_i32(cu), past_lens=_i32(pasts), slots=_i32(slots), n_seqs=len(news), n_tokens=cu[-1],
                           single_token=all(n == 1 for n in news), max_new=max(news),
                           max_total=max(p + n for p, n in zip(pasts, news)), ws=Workspace(torch.device(DEV)))


# ------------------------------------------------------------------ token pairs
@pytest.mark.parametrize("types", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16),
                                   (torch.float32, torch.bfloat16), (torch.bfloat16, torch.float32)])
@pytest.mark.parametrize("d", [40, 33, 1024])
@pytest.mark.parametrize("bigram", [(97, 31, 7), (1, 5, 5), (5003, 1000003, 998244353), (64, 0, 1), (64, 1, 0)])
def test_embedding_with_token_pairs(types, d, bigram):
    """Three sequences in the slots 4, 0, 2: a prompt of 300 tokens and one of 1, then one that goes on, then a step of
    one token each, then slot 0 used again by a sequence that starts: its first token must not see the old state."""
    from ziglm_b200 import kernels
    kernels.require(("elementwise",))
    buckets, a, b = bigram
    vocab = 77
    table, pairs = _r(vocab, d, seed=1, dtype=types[0]), _r(buckets + 1, d, seed=2, dtype=types[1])
    last = torch.full((6, 1), 70, dtype=torch.int32, device=DEV)
    g = torch.Generator().manual_seed(d)
    draw = lambda n: torch.randint(0, vocab, (n,), generator=g).tolist()
    history = {4: [], 0: [], 2: []}

    def run(slots, parts):
        pasts = [len(history[s]) for s in slots]
        toks = [t for p in parts for t in p]
        step = _step(pasts, [len(p) for p in parts], slots, toks)
        out, kept = torch.empty(len(toks), d, device=DEV), torch.empty(len(toks), d, device=DEV)
        kernels.embed_pairs(table, pairs, last, a, b, step, out, kept, scale=1.5)
        rows = []
        for s, p in zip(slots, parts):
            rows += P.pair_rows(p, history[s][-1] if history[s] else None, {"buckets": buckets, "mul_prev": a, "mul_cur": b})
            history[s] += p
        want = table.float()[torch.tensor(toks)] * 1.5 + pairs.float()[torch.tensor(rows)]
        torch.testing.assert_close(out, want, atol=1e-6, rtol=1e-6)
        assert torch.equal(out, kept)
        assert [last[s].item() for s in slots] == [history[s][-1] for s in slots]

    run([4, 0], [draw(300), draw(1)])
    run([0, 4, 2], [draw(5), draw(2), draw(9)])
    run([2, 4, 0], [draw(1), draw(1), draw(1)])
    run([0, 2], [draw(1), draw(1)])
    history[0] = []
    run([0, 4], [draw(1), draw(1)])                      # one starts, one goes on, in the kernel of one token each
    history[2] = []
    run([2, 0], [draw(40), draw(3)])
    assert last[1].item() == last[3].item() == last[5].item() == 70


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("T,d", [(1, 33), (5, 64), (300, 72)])
def test_a_row_and_kept_rows_are_added(dtype, T, d):
    from ziglm_b200 import kernels
    kernels.require(("elementwise",))
    x, kept, row = _r(T, d, seed=1), _r(T, d, seed=2), _r(d, seed=3, dtype=dtype)
    for rows in (kept, None):
        got = x.clone()
        kernels.add_row(got, row, rows=rows)
        want = (x + rows if rows is not None else x) + row.float()
        assert torch.equal(got, want)


# ------------------------------------------------- norm of heads, values that are the keys
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,G,D,hd,rot", [(6, 2, 20, 24, 0), (4, 1, 64, 64, 0), (3, 3, 128, 128, 0), (1, 1, 5, 8, 0),
                                          (8, 4, 72, 72, 16), (4, 2, 40, 40, 6)])
def test_norm_of_heads_with_values_that_are_the_keys_before_it(dtype, H, G, D, hd, rot):
    """The value pages hold the key heads exactly as the rows did; the key pages the normed (and turned) ones."""
    from ziglm_b200 import kernels
    kernels.require(("attention",))
    eps, page = 1e-5, 64
    positions, seq = list(range(60, 80)) + [3], [0] * 20 + [1]
    T = len(positions)
    rows = _r(T, (H + G) * hd + 16, seed=1, dtype=dtype)
    rows.view(T, -1)[:, :(H + G) * hd].view(T, H + G, hd)[:, :, D:] = 0
    before = rows.clone()
    wq, wk = torch.zeros(hd, device=DEV), torch.zeros(hd, device=DEV)
    wq[:D], wk[:D] = _r(D, seed=4).abs() + 0.5, _r(D, seed=5) * 2.0
    inv = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(rot // 2)], device=DEV) if rot else None
    k_pages = torch.full((4, G, page, hd), 999.0, dtype=dtype, device=DEV)
    v_pages = torch.full((4, G, page, hd), 999.0, dtype=dtype, device=DEV)
    table = _i32([[3, 0], [2, -1]])
    kernels.rope_norm_store(rows, H, G, hd, rot, inv, 1.0, D, eps, _i32(positions), _i32(seq), table, k_pages, v_pages,
                            page, norm_first=True, q_weight=wq, k_weight=wk, values_from_keys=True)
    heads = before[:, :(H + G) * hd].view(T, H + G, hd)
    plain = heads.float().cpu()[:, :, :D]
    q = P.rms_norm(plain[:, :H], wq.cpu()[:D], eps)
    k = P.rms_norm(plain[:, H:], wk.cpu()[:D], eps)
    if rot:
        turn = lambda x: torch.cat([P.rotate_halves(x[..., :rot], torch.tensor(positions), 50.0), x[..., rot:]], dim=-1)
        q, k = turn(q), turn(k)
    got = rows[:, :(H + G) * hd].view(T, H + G, hd)
    torch.testing.assert_close(got[:, :H, :D].float().cpu(), q, **_tol(dtype))
    torch.testing.assert_close(got[:, H:, :D].float().cpu(), k, **_tol(dtype))
    assert (got[:, :, D:] == 0).all() and torch.equal(rows[:, (H + G) * hd:], before[:, (H + G) * hd:])
    tb = table.cpu()
    for t, (pos, b) in enumerate(zip(positions, seq)):
        pg = tb[b, pos // page].item()
        assert torch.equal(k_pages[pg, :, pos % page], got[t, H:])
        assert torch.equal(v_pages[pg, :, pos % page], heads[t, H:])
    assert (k_pages == 999.0).sum().item() == (4 * page - T) * G * hd


# ------------------------------------------------------------ distance bias and sinks
def _plain_attention(q, k, v, scale, slopes, sinks, window=None):
    n, H = q.shape[0], q.shape[1]
    G = k.shape[1]
    q, k, v = q.float().cpu(), k.float().cpu(), v.float().cpu()
    i = torch.arange(n)
    seen = P.causal(i, n)
    if window is not None:
        seen = seen & (i[:, None] - i[None, :] < window)
    out = torch.zeros(n, H, v.shape[2])
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t()) * scale
        if slopes is not None:
            s = s - slopes[h].item() * (i[:, None] - i[None, :]).float()
        none = torch.tensor(float("-inf"))
        out[:, h] = P.softmax_with_sink(s, seen, none if sinks is None else sinks[h].cpu()) @ v[:, g]
    return out.reshape(n, -1)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,G,hd,sink,window", [(6, 2, 40, True, None), (4, 1, 64, True, None), (3, 3, 128, True, None),
                                                (5, 1, 64, False, None), (12, 4, 128, True, 70), (16, 1, 64, True, None),
                                                (2, 2, 24, False, 9), (20, 1, 64, True, None)])
def test_attention_with_a_distance_bias(dtype, H, G, hd, sink, window):
    """Prompts of two sequences, portions of one and of twenty tokens behind them, and decoded tokens, against the
    formula.  Slopes from steep to nearly flat; in every head one key far back is made to outweigh its bias, so that a
    bias that is too large, missing or of the wrong head shows."""
    from ziglm_b200 import kernels
    from ziglm_b200.parts.base import LayerIO
    kernels.require(("attention",) + kernels.fast_attention_libraries(dtype, hd, H, G, sinks=True))
    lens, page, scale = [330, 70], 64, 0.3
    slopes = torch.tensor(P.distance_slopes(H), device=DEV)
    sinks = (_r(H, seed=5) * 2.0 + 1.0) if sink else None
    ks = [_r(L, G, hd, seed=i, dtype=dtype) for i, L in enumerate(lens)]
    vs = [_r(L, G, hd, seed=3 + i, dtype=dtype) for i, L in enumerate(lens)]
    qs = [_r(L, H, hd, seed=7 + i, scale=0.6, dtype=dtype) for i, L in enumerate(lens)]
    for k, q in zip(ks, qs):
        for h in range(H):
            g = h // (H // G)
            far = 3 + h % 5
            k[far, g] = q[-1, h].sign() * 1.5            # the last token asks for a key at the very front
            k[far, g] *= (slopes[h].item() * (q.shape[0] - far) + 4.0) / max(
                1e-3, (q[-1, h].float() @ k[far, g].float()).item() * scale)
    want = [_plain_attention(q, k, v, scale, slopes, sinks, window) for q, k, v in zip(qs, ks, vs)]
    k_pages = torch.zeros(9, G, page, hd, dtype=dtype, device=DEV)
    v_pages = torch.zeros(9, G, page, hd, dtype=dtype, device=DEV)
    table = _i32([[5, 2, 7, 0, 8, 3], [1, 6, -1, -1, -1, -1]])
    tb = table.cpu()
    for b, L in enumerate(lens):
        for p in range(L):
            k_pages[tb[b, p // page], :, p % page] = ks[b][p]
            v_pages[tb[b, p // page], :, p % page] = vs[b][p]
    tol = _tol(dtype, (2e-5, 2e-5), (3e-2, 3e-2))

    def attend(pasts, news):
        step = _step(pasts, news, [0, 1])
        io = LayerIO(k_pages=k_pages, v_pages=v_pages, block_table=table, page_size=page)
        rows = torch.cat([q[p:p + n] for q, p, n in zip(qs, pasts, news)]).reshape(sum(news), H * hd).contiguous()
        out = torch.empty(sum(news), H * hd, dtype=dtype, device=DEV)
        kernels.attention(step, rows, out, H, G, hd, scale, window, io, sinks=sinks, slopes=slopes)
        ref = torch.cat([w[p:p + n] for w, p, n in zip(want, pasts, news)])
        torch.testing.assert_close(out.float().cpu(), ref, **tol, msg=lambda m: f"pasts {pasts}, news {news}: {m}")

    attend([0, 0], lens)
    attend([300, 67], [30, 3])
    attend([310, 40], [20, 30])
    attend([326, 64], [2, 5])
    for back in (1, 2, 66):
        attend([lens[0] - back, max(0, lens[1] - back)], [1, 1])
    for lib in (kernels.attention_tc_status, kernels.attention_fmha_status):
        if dtype == torch.bfloat16 and hd in (64, 128) and H // G <= 16:
            assert lib() == 0


def test_a_bias_goes_with_no_kept_first_tokens():
    from ziglm_b200 import kernels
    from ziglm_b200.config.spec import MixerSpec, PositionSpec
    from ziglm_b200.parts import mixer_class
    o = {"value_dim": 16, "distance_bias": 8.0}
    spec = lambda **kw: MixerSpec(kind="capped_attention", width=32, n_heads=2, n_kv_heads=1, head_dim=16, scale=0.25,
                                  position=PositionSpec(kind="none"), **kw)
    make = lambda s: mixer_class("capped_attention")(s, torch.float32, torch.device("cpu"))
    make(spec(options=o))
    with pytest.raises(ValueError, match="distance bias"):
        make(spec(window=8, options={**o, "keep_first": 2}))
    with pytest.raises(ValueError, match="values that are the keys"):
        make(spec(options={"value_dim": 8, "values": "keys"}))
    with pytest.raises(ValueError, match="values 'queries'"):
        make(spec(options={"value_dim": 16, "values": "queries"}))
    with pytest.raises(kernels.KernelError, match="per query head"):
        kernels._head_numbers(torch.ones(3, device=DEV), 2, "slopes")


# ------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,D,rot,rank,kept,wide_q", [(5, 12, 6, 21, 32, True), (4, 32, 32, 96, 128, True), (2, 8, 16, 40, 64, True),
                                                      (3, 16, 0, 64, 64, True), (6, 24, 8, 88, 128, True), (4, 64, 16, 48, 64, False),
                                                      (3, 10, 4, 12, 16, False), (2, 8, 0, 24, 24, False), (40, 64, 32, 96, 128, True)])
def test_latent_norm_rotations_and_cache_row(dtype, H, D, rot, rank, kept, wide_q):
    """One token a sequence and prompts, shuffled pages; queries from float32 columns beside the latent's or in the rows'
    type in place; the row [rotated | normed | zeros]."""
    from ziglm_b200 import kernels
    kernels.require(("attention",))
    eps, page = 1e-5, 64
    for positions, seq in ((list(range(60, 90)) + [3], [0] * 30 + [1]), ([127, 5], [0, 1])):
        T = len(positions)
        q_cols = H * (D + rot)
        first = q_cols if wide_q else 8
        proj = _r(T, first + rank + rot + 24, seed=1)
        q_in = proj[:, :q_cols].clone() if wide_q else _r(T, q_cols, seed=2, dtype=dtype)
        q = proj[:, :q_cols] if wide_q else q_in.clone()
        out = q if q.dtype == dtype else torch.empty(T, q_cols, dtype=dtype, device=DEV)
        w = _r(rank, seed=3).abs() + 0.5
        inv = torch.tensor([50.0 ** (-2.0 * i / rot) for i in range(rot // 2)], device=DEV) if rot else None
        down = proj.clone()
        pages = torch.full((4, 1, page, kept), 999.0, dtype=dtype, device=DEV)
        table = _i32([[3, 0], [2, -1]])
        kernels.latent_prep(proj, first, rank, first + rank, rot, w, eps, q, out, H, inv, _i32(positions), _i32(seq), table,
                            pages, page)
        pos = torch.tensor(positions)
        c = P.rms_norm(down[:, first:first + rank].cpu(), w.cpu(), eps)
        r = down[:, first + rank:first + rank + rot].cpu()
        heads = q_in.float().cpu().view(T, H, D + rot)
        if rot:
            r = P.rotate_halves(r[:, None], pos, 50.0)[:, 0]
            heads = torch.cat([heads[..., :D], P.rotate_halves(heads[..., D:], pos, 50.0)], dim=-1)
        tol = _tol(dtype, (1e-5, 1e-5), (1e-2, 1e-2))
        torch.testing.assert_close(out.float().cpu().view(T, H, D + rot), heads, **tol)
        tb = table.cpu()
        for t, (p, b) in enumerate(zip(positions, seq)):
            row = pages[tb[b, p // page], 0, p % page].float().cpu()
            torch.testing.assert_close(row[:rot], r[t], **tol)
            torch.testing.assert_close(row[rot:rot + rank], c[t], **tol)
            assert (row[rot + rank:] == 0).all()
        assert (pages == 999.0).sum().item() == (4 * page - T) * kept
        assert torch.equal(proj[:, first + rank + rot:], down[:, first + rank + rot:])


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,hd", [(4, 128), (5, 40), (16, 64), (3, 136)])
def test_attention_over_one_shared_head_with_learned_sinks(dtype, H, hd):
    """Keys that are their own values, one key/value head for all query heads, sinks that outweigh most keys: prompts,
    portions and decoded tokens."""
    from ziglm_b200 import kernels
    from ziglm_b200.parts.base import LayerIO
    kernels.require(("attention",) + kernels.fast_attention_libraries(dtype, hd, H, 1, sinks=True))
    L, page, scale = 150, 64, 0.2
    k, q = _r(L, 1, hd, seed=1, dtype=dtype), _r(L, H, hd, seed=2, dtype=dtype)
    sinks = torch.linspace(-3.0, 9.0, H, device=DEV)
    want = _plain_attention(q, k, k, scale, None, sinks)
    pages = torch.zeros(3, 1, page, hd, dtype=dtype, device=DEV)
    table = _i32([[2, 0, 1]])
    for p in range(L):
        pages[table[0, p // page], 0, p % page] = k[p, 0]
    io = LayerIO(k_pages=pages, v_pages=pages, block_table=table, page_size=page)
    for past, n in ((0, L), (100, 50), (140, 3), (L - 1, 1), (63, 1), (64, 1), (0, 1)):
        step = _step([past], [n], [0])
        out = torch.empty(n, H * hd, dtype=dtype, device=DEV)
        kernels.attention(step, q[past:past + n].reshape(n, H * hd).contiguous(), out, H, 1, hd, scale, None, io, sinks=sinks)
        torch.testing.assert_close(out.float().cpu(), want[past:past + n], **_tol(dtype, (2e-5, 2e-5), (2e-2, 2e-2)))


@pytest.mark.parametrize("H,G,D,hd,n_blocks", [(4, 1, 64, 64, 0), (12, 4, 128, 128, 0), (3, 3, 56, 64, 7), (16, 1, 100, 128, 3),
                                               (8, 2, 64, 64, 1), (32, 8, 64, 64, 0)])
def test_decode_kernel_that_norms_heads_and_writes_the_cache(H, G, D, hd, n_blocks):
    """One token of several sequences, lengths around page borders: the kernel that norms the query heads as it loads them
    and puts the new key (normed) and value (as it was) into the cache, with sinks and the bias, against the formula; pages
    and rows it does not own are left alone."""
    from ziglm_b200 import kernels
    kernels.require(("attention_tc",))
    dtype, page, scale, eps = torch.bfloat16, 64, 0.2, 1e-5
    lens = [1, 64, 65, 300, 63, 128, 777]                 # with the new token
    B = len(lens)
    slopes, sinks = torch.tensor(P.distance_slopes(H), device=DEV), _r(H, seed=5) * 2.0
    per = -(-max(lens) // page)
    order = torch.randperm(B * per, generator=torch.Generator().manual_seed(1)).view(B, per)
    table = order.to(torch.int32).to(DEV)
    raw = [_r(L, G, hd, seed=i, dtype=dtype) for i, L in enumerate(lens)]
    rows = _r(B, (H + G) * hd + 16, seed=9, dtype=dtype)
    heads = rows[:, :(H + G) * hd].view(B, H + G, hd)
    heads[:, :, D:] = 0
    wq, wk = torch.zeros(hd, device=DEV), torch.zeros(hd, device=DEV)
    wq[:D], wk[:D] = _r(D, seed=4).abs() + 0.5, _r(D, seed=5).abs() + 0.5
    k_pages = torch.zeros(B * per, G, page, hd, dtype=dtype, device=DEV)
    v_pages = torch.zeros(B * per, G, page, hd, dtype=dtype, device=DEV)
    for b, L in enumerate(lens):
        raw[b][:, :, D:] = 0
        raw[b][-1] = heads[b, H:]
        keys = (P.rms_norm(raw[b].float().cpu()[:, :, :D], wk.cpu()[:D], eps)).to(dtype)
        for p in range(L - 1):
            k_pages[order[b, p // page], :, p % page, :D] = keys[p].to(DEV)
            v_pages[order[b, p // page], :, p % page] = raw[b][p]
    before = k_pages.clone()
    positions, seq = _i32([L - 1 for L in lens]), _i32(list(range(B)))
    out = torch.empty(B, H * hd, dtype=dtype, device=DEV)
    blocks = n_blocks or kernels.attention_decode_flat_blocks(B, H, G, hd)
    scratch = torch.empty(kernels.attention_decode_flat_scratch(B, H, G, hd, blocks), device=DEV)
    counters = torch.zeros(B * G, dtype=torch.int32, device=DEV)
    for _ in range(2):                                    # the counters are back at zero: a second call is the same
        assert kernels.attention_decode_flat(rows, out, H, G, hd, scale, None, positions, seq, table, k_pages, v_pages, page,
                                             blocks, counters, scratch, rope=(None, 0, True), norm=(D, eps, wq, wk),
                                             values_from_keys=True, sinks=sinks, slopes=slopes)
    q = P.rms_norm(heads[:, :H].float().cpu()[:, :, :D], wq.cpu()[:D], eps).to(dtype)
    for b, L in enumerate(lens):
        k = P.rms_norm(raw[b].float().cpu()[:, :, :D], wk.cpu()[:D], eps).to(dtype)
        qs = torch.zeros(L, H, D, dtype=dtype)
        qs[-1] = q[b]
        want = _plain_attention(qs, k, raw[b], scale, slopes, sinks)[-1]
        torch.testing.assert_close(out[b].float().cpu(), want, atol=2e-2, rtol=2e-2, msg=lambda m: f"length {L}: {m}")
        pg, r = order[b, (L - 1) // page], (L - 1) % page
        torch.testing.assert_close(k_pages[pg, :, r, :D].float().cpu(), k[-1].float(), atol=2e-2, rtol=1e-2)
        assert (k_pages[pg, :, r, D:] == 0).all() and torch.equal(v_pages[pg, :, r], heads[b, H:])
        k_pages[pg, :, r] = before[pg, :, r]
    assert torch.equal(k_pages, before) and kernels.attention_tc_status() == 0
