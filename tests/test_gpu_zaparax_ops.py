"""Each Zaparax mechanism alone on the GPU against its float64 statement in oracle/zaparax_oracle.py: RMS sublayer closes with a second
weighted result, the hashed-pair embedding and its carried token, unit-RMS heads with the query temperature into pages, capped and
distance-biased attention with a sink (window edges, far keys that stand out, every kernel form), the router with a choice correction and
identity experts, the gated experts in both forms, the state-space recurrence as an op (chunks, portions, single tokens, extreme steps) and
both mixers. Packed batches mix sequences that start, continue and advance by one token, over shuffled pages and slots."""
import math

import pytest
import torch

from oracle import zaparax_oracle as O
from tests import hybrid_util as HU
from tests import zaparax_util as U

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ---- closes and norms ----
@pytest.mark.parametrize("width,wdt", [(7, torch.float32), (40, torch.bfloat16), (250, torch.bfloat16), (1000, torch.bfloat16), (2048, torch.float32), (3001, torch.bfloat16),
                                       (9000, torch.bfloat16)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["rms_centred", "rms"])
def test_rms_sandwich_close(width, wdt, dtype, kind):
    """x + N1(y + coef u) into the residual in place, N2 of the sum; a row whose second result has weight 0, rows that are all zero; then
    without the second result, without y, with gathered rows."""
    from vyomai_b200 import ops
    g = _gen(0)
    rows, eps = 9, 1e-3
    x, y, u = (torch.randn(rows, width, generator=g) * s for s in (1.0, 3.0, 2.0))
    u = u.to(dtype)
    y[2] += 50.0      # an RMS norm keeps the mean
    y[3] = 0.0
    coef = torch.rand(rows, generator=g)
    coef[3] = coef[5] = 0.0
    w1, w2 = ((0.3 * torch.randn(width, generator=g)).to(wdt) for _ in range(2))
    d = lambda t: t.to(DEV)  # noqa: E731
    norm = lambda t, w: O.centred_norm(t, w.double(), eps) if kind == "rms_centred" else O.rms(t, eps) * w.double()  # noqa: E731
    s = x.double() + norm(y.double() + coef.double()[:, None] * u.double(), w1)
    tol = 3e-5 if dtype == torch.float32 else 1e-2
    xd = d(x)
    got = ops.sandwich_norm(xd, d(y), d(w1), d(w2), eps=eps, x_out=xd, out_dtype=dtype, kind=kind, second=(d(u), d(coef)))
    assert HU.rel_err(xd.cpu(), s) < 3e-5 and HU.rel_err(got.cpu(), norm(s, w2)) < tol
    xd = d(x)
    assert ops.sandwich_norm(xd, d(y), d(w1), eps=eps, x_out=xd, kind=kind) is None and HU.rel_err(xd.cpu(), x.double() + norm(y.double(), w1)) < 3e-5
    idx = _i32([4, 0, 8, 4])
    got = ops.sandwich_norm(d(x), norm2=d(w2), eps=eps, row_index=idx, out_dtype=dtype, kind=kind)
    assert HU.rel_err(got.cpu(), norm(x.double(), w2)[[4, 0, 8, 4]]) < tol


@pytest.mark.parametrize("groups,width", [(1, 3000), (2, 4096), (3, 2051), (1, 8192), (1, 8200)])
def test_grouped_norm_of_wide_rows(groups, width):
    from vyomai_b200 import ops
    g = _gen(1)
    x, w = torch.randn(5, groups * width, generator=g), torch.randn(groups * width, generator=g)
    got = ops.rms_norm(x.to(DEV), w.to(DEV), eps=1e-5, groups=groups, w_full=True).cpu()
    assert HU.rel_err(got, O.rms(x.double().view(5, groups, width), 1e-5).reshape(5, -1) * w.double()) < 1e-5


# ---- embedding ----
@pytest.mark.parametrize("buckets,mp,mc", [(53, 7, 3), (1, 5, 9), (211, 10 ** 12 + 39, 2 ** 40 + 1), (509, 0, 1)])
def test_hashed_pair_embedding_and_the_carried_token(buckets, mp, mc):
    """Three sequences over three steps: one starts while another continues and one advances by single tokens; slots that held another
    sequence's token; position 0 reads the extra row whatever the slot holds."""
    from vyomai_b200 import ops
    g = _gen(2)
    vocab, width = 61, 21
    table, pairs = torch.randn(vocab, width, generator=g).to(torch.bfloat16), torch.randn(buckets + 1, width, generator=g).to(torch.bfloat16)
    prev = torch.full((5, 1), 60, dtype=torch.int32, device=DEV)
    toks = [HU.tokens(n, vocab, 3 + n) for n in (13, 6, 4)]
    want = [O.embedding(t, table.double(), 1.7, pairs.double(), {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}) for t in toks]
    at, slots = [0, 0, 0], [4, 1, 2]
    for step in ([(0, 7), (1, 1)], [(1, 1), (0, 5), (2, 2)], [(0, 1), (2, 1), (1, 1)], [(1, 3), (2, 1)]):
        cu = [0]
        for _, n in step:
            cu.append(cu[-1] + n)
        batch = ops.PackedBatch(_i32(cu), _i32([at[s] for s, _ in step]), _i32([slots[s] for s, _ in step]), max(n for _, n in step))
        ids = _i32([t for s, n in step for t in toks[s][at[s]:at[s] + n]])
        got = ops.pair_embed(batch, ids, table.to(DEV), 1.7, pairs.to(DEV), prev, mul_prev=mp, mul_cur=mc).cpu()
        for i, (s, n) in enumerate(step):
            assert HU.rel_err(got[cu[i]:cu[i + 1]], want[s][at[s]:at[s] + n]) < 1e-6
            at[s] += n
            assert int(prev[slots[s], 0]) == toks[s][at[s] - 1]
    assert int(prev[0, 0]) == int(prev[3, 0]) == 60


# ---- attention ----
@pytest.mark.parametrize("dim,vdim,every", [(12, 10, 5), (10, 33, 1), (200, 8, 4096)])
def test_unit_heads_query_temperature_and_page_write(dim, vdim, every):
    from vyomai_b200 import ops
    H, G, bs, eps, coef = 4, 2, 4, 1e-4, 0.7
    lengths, pos0 = [9, 1, 5], [0, 4095, 3]
    batch, table, _, n_blocks, _ = HU.shuffled_batch(lengths, pos0, bs, DEV)
    g = _gen(3)
    n = sum(lengths)
    P = torch.randn(n, H * dim + G * dim + G * vdim, generator=g)
    kp, vp = torch.full((n_blocks, bs, G, dim), 7.0, device=DEV), torch.full((n_blocks, bs, G, vdim), 7.0, device=DEV)
    Pd = P.to(DEV)
    q, k, v = Pd[:, :H * dim], Pd[:, H * dim:(H + G) * dim], Pd[:, (H + G) * dim:]
    ops.rope_kv_write(batch, q, k, v, torch.zeros(1, device=DEV), kp, vp, heads=H, kv_heads=G, dim=dim, vdim=vdim, rot_dims=0, layout="half", unit_rms=True,
                      eps=eps, q_temp=(coef, every))
    at = 0
    for s, (ln, p) in enumerate(zip(lengths, pos0)):
        x = P[at:at + ln].double()
        temp = O.query_temperature(p + ln, coef, every)[p:]
        qs = O.rms(x[:, :H * dim].view(ln, H, dim), eps) * temp[:, None, None]
        assert HU.rel_err(Pd[at:at + ln, :H * dim].cpu().view(ln, H, dim), qs) < 1e-5
        for i in range(ln):
            blk, off = table[s][(p + i) // bs], (p + i) % bs
            assert HU.rel_err(kp[blk, off].cpu(), O.rms(x[i, H * dim:(H + G) * dim].view(G, dim), eps)) < 1e-5
            assert torch.equal(vp[blk, off].cpu(), P[at + i, (H + G) * dim:].view(G, vdim))
        at += ln
    assert int((kp == 7.0).all(-1).all(-1).sum()) == n_blocks * bs - n    # nothing else was written


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 8, 12), (8, 1, 8, 8), (16, 2, 12, 20), (3, 3, 10, 5), (4, 1, 130, 70), (8, 2, 16, 16)])
@pytest.mark.parametrize("window,bs,cap,sinks", [(1, 4, 2.0, True), (7, 4, 0.0, True), (16, 16, 1.2, True), (64, 16, 3.0, False), (100, 8, 2.5, True), (0, 8, 2.0, True)])
def test_biased_attention_over_pages(H, G, d, dv, window, bs, cap, sinks):
    """Four sequences in one step and each alone: a whole prompt, a long portion that starts inside a window, a portion of a few tokens,
    a single token (alone it takes the single-token forms). Keys just inside and just outside the last query's window are made to stand
    out, each with a value of its own: a window one token off in either direction is far outside the tolerance."""
    from vyomai_b200 import ops
    scale, far = 0.8, (window or 60)
    T = [2 * far + 35, far + 24, far + 9, far + 5]
    new = [T[0], 20, 5, 1]
    g = _gen(5)
    # the design's slopes, but flat enough on the last head that a key at the window's far end still counts
    slopes = [min(s, 0.5 / far) if h == H - 1 else s for h, s in enumerate(O.head_slopes(H))]
    sink = torch.randn(H, generator=g) if sinks else None
    qs = [torch.randn(t, H, d, generator=g).double() / d ** 0.25 for t in T]
    ks = [torch.randn(t, G, d, generator=g).double() / d ** 0.25 for t in T]
    vs = [torch.randn(t, G, dv, generator=g).double() for t in T]
    for s, t in enumerate(T):
        for back, val in ((far - 1, 4.0), (far, -6.0)):   # the window's last key and the first one out of it
            j = t - 1 - back
            if j >= 0:
                ks[s][j, -1] = 4.0 * qs[s][t - 1, -1]
                vs[s][j] += val
    pos0 = [t - n for t, n in zip(T, new)]
    kw = dict(scale=scale, softcap=cap, slopes=slopes, sink=None if sink is None else sink.double())
    want = [O.biased_attention(qs[s], ks[s], vs[s], window=window, **kw)[pos0[s]:].reshape(new[s], -1) for s in range(4)]
    if window > 1:
        for off in (window - 1, window + 1):
            assert HU.rel_err(O.biased_attention(qs[3], ks[3], vs[3], window=off, **kw)[-1], want[3].view(H, dv)) > 1e-2
    sd = torch.tensor(slopes, dtype=torch.float32, device=DEV)
    for group in ([0, 1, 2, 3], [0], [1], [2], [3]):
        batch, table, _, n_blocks, _ = HU.shuffled_batch([new[s] for s in group], [pos0[s] for s in group], bs, DEV, seed=window)
        kp = torch.full((n_blocks, bs, G, d), 1e3, device=DEV)      # rows no query may read
        vp = torch.full((n_blocks, bs, G, dv), 1e3, device=DEV)
        for n, s in enumerate(group):
            for p in range(T[s]):
                blk, off = table[n][p // bs], p % bs
                kp[blk, off], vp[blk, off] = ks[s][p].float().to(DEV), vs[s][p].float().to(DEV)
        q = torch.cat([qs[s][pos0[s]:].reshape(new[s], H * d) for s in group]).float().to(DEV)
        got = ops.window_attn(batch, q, kp, vp, heads=H, kv_heads=G, dim=d, vdim=dv, scale=scale, window=window, keep_first=0, softcap=cap, head_slope=sd,
                              sink=None if sink is None else sink.to(DEV)).cpu()
        assert HU.rel_err(got, torch.cat([want[s] for s in group])) < 3e-5, group


@pytest.mark.parametrize("H,G", [(4, 2), (8, 1)])
def test_a_far_key_among_hundreds_is_found(H, G):
    """No window: one key 700 positions back carries the only large score of a head with a small slope; decoded and as a prompt's end."""
    from vyomai_b200 import ops
    T, d, bs, back = 800, 16, 16, 700
    g = _gen(6)
    slopes = [1e-3] * H
    q, k, v = torch.randn(T, H, d, generator=g) * 0.1, torch.randn(T, G, d, generator=g) * 0.1, torch.randn(T, G, d, generator=g)
    k[T - 1 - back] = 40.0 * q[T - 1].view(G, H // G, d).mean(1) / q[T - 1].view(G, H // G, d).mean(1).norm(dim=-1, keepdim=True)
    v[T - 1 - back] = 5.0
    want = O.biased_attention(q.double(), k.double(), v.double(), scale=4.0, softcap=30.0, window=0, slopes=slopes, sink=torch.zeros(H).double())
    missing = v.clone()
    missing[T - 1 - back] = 0.0
    assert HU.rel_err(O.biased_attention(q.double(), k.double(), missing.double(), scale=4.0, softcap=30.0, window=0, slopes=slopes, sink=torch.zeros(H).double())[-1], want[-1]) > 0.3
    for n in (1, 3, 50, T):
        batch, table, _, n_blocks, _ = HU.shuffled_batch([n], [T - n], bs, DEV)
        kp, vp = (torch.zeros((n_blocks, bs, G, d), device=DEV) for _ in range(2))
        order = torch.tensor(table[0], device=DEV)
        pos = torch.arange(T, device=DEV)
        kp[order[pos // bs].long(), pos % bs], vp[order[pos // bs].long(), pos % bs] = k.to(DEV), v.to(DEV)
        got = ops.window_attn(batch, q[T - n:].reshape(n, -1).to(DEV), kp, vp, heads=H, kv_heads=G, dim=d, vdim=d, scale=4.0, window=0, keep_first=0, softcap=30.0,
                              head_slope=torch.tensor(slopes, device=DEV), sink=torch.zeros(H, device=DEV)).cpu()
        assert HU.rel_err(got, want[T - n:].reshape(n, -1)) < 3e-5


# ---- router and experts ----
@pytest.mark.parametrize("rows,experts,identity,top", [(1, 5, 2, 3), (33, 12, 0, 4), (70, 1, 3, 4), (9, 40, 24, 33), (5, 3, 1, 1)])
def test_router_with_correction_and_identity_experts(rows, experts, identity, top):
    from vyomai_b200 import ops
    g = _gen(7)
    n = experts + identity
    z, corr = torch.randn(rows, n, generator=g) * 2.0, torch.randn(n, generator=g) * 0.3
    idx, wt, dense, *rest = ops.moe_route(z.to(DEV), n, top, 1.0, kind="softmax", normalize=False, correction=corr.to(DEV), identity=identity)
    oi, ow = O.route(z.double(), corr.double(), top)
    assert torch.equal(idx.cpu().long(), oi) and HU.rel_err(wt.cpu(), ow) < 1e-5
    full = torch.zeros(rows, n, dtype=torch.float64).scatter_(1, oi, ow)
    assert dense.shape == (rows, experts) and float((dense.cpu().double() - full[:, :experts]).abs().max()) < 1e-6
    if identity:
        assert float((rest[0].cpu().double() - full[:, experts:].sum(1)).abs().max()) < 1e-6
    else:
        assert not rest
    if top < n:   # the correction did change choices, and only choices
        assert not torch.equal(torch.sort(oi, 1).values, torch.sort(torch.softmax(z.double(), 1).topk(top, 1).indices, 1).values) or rows < 8


def test_router_normalises_plain_scores_when_asked():
    from vyomai_b200 import ops
    z, corr = torch.randn(6, 8, generator=_gen(8)), torch.linspace(-1, 1, 8)
    idx, wt, _ = ops.moe_route(z.to(DEV), 8, 3, 2.5, kind="sigmoid", correction=corr.to(DEV))
    s = torch.sigmoid(z.double())
    oi = (s + corr.double()).topk(3, 1).indices
    w = s.gather(1, oi)
    assert torch.equal(idx.cpu().long(), oi) and HU.rel_err(wt.cpu(), 2.5 * w / w.sum(1, keepdim=True)) < 1e-5


@pytest.mark.parametrize("experts,ff,shared_ff", [(3, 5, 7), (4, 16, 8), (2, 8, 0), (0, 1, 24)])
@pytest.mark.parametrize("interleaved", [True, False])
def test_gated_experts_activation_options(experts, ff, shared_ff, interleaved):
    from vyomai_b200 import ops
    g = _gen(9)
    rows = 6
    gate, up = (torch.randn(rows, experts * ff + shared_ff, generator=g) for _ in range(2))
    dense = torch.rand(rows, experts, generator=g) if experts else None
    if experts:
        dense[:, 0] = 0.0
    sg = torch.randn(rows, 1, generator=g) if shared_ff else None
    blocks = []
    for a, n in [(e * ff, ff) for e in range(experts)] + ([(experts * ff, shared_ff)] if shared_ff else []):
        p = (gate[:, a:a + n], up[:, a:a + n])
        blocks.append(torch.stack(p, 2).reshape(rows, 2 * n) if interleaved else torch.cat(p, 1))
    h = torch.cat(blocks, 1)
    got = ops.moe_glu(h.to(DEV), None if dense is None else dense.to(DEV), experts=experts, ff=ff, shared_ff=shared_ff, limit=0.0, alpha=1.0, out_dtype=torch.float32,
                      interleaved=interleaved, shift=False, shared_gate=None if sg is None else sg.to(DEV)).cpu()
    w = torch.cat(([dense.double().repeat_interleave(ff, 1)] if experts else []) + ([torch.sigmoid(sg.double()).expand(rows, shared_ff)] if shared_ff else []), 1)
    assert HU.rel_err(got, O.silu(gate.double()) * up.double() * w) < 1e-5


def _experts(f, width, dtype, seed=11, **kw):
    from vyomai_b200 import ZaparaxConfig, ZaparaxForCausalLM
    from vyomai_b200.layers.mixers import MoEFeedForward
    cfg = ZaparaxConfig(U.config([U.layer("mamba2", U.mamba(), f)], width=width))
    w = {k[len("l0.mlp."):]: v for k, v in ZaparaxForCausalLM.random_weights(cfg, seed=seed).items() if k.startswith("l0.mlp.")}
    r = f["router"]
    m = MoEFeedForward({k: v.to(DEV, dtype) for k, v in w.items()}, r["experts"], r["top"], 1.0, dtype, True, shared=bool(f.get("shared")), router="softmax",
                       normalize=False, form="swiglu", identity=int(r.get("identity") or 0), **kw)
    return m, {k: v.double() for k, v in w.items()}


@pytest.mark.parametrize("rows", [1, 5, 40, 150])
@pytest.mark.parametrize("f,width,dtype", [(U.moe(), 40, torch.float32), (U.moe(identity=None, shared=None), 40, torch.float32), (U.moe(experts=1, top=2, identity=1), 24, torch.float32),
                                           (U.moe(ff=64, experts=6, top=3, identity=2, shared=96), 128, torch.bfloat16), (U.moe(ff=20, experts=3, top=2, shared=12), 64, torch.bfloat16)])
@pytest.mark.parametrize("sort", [False, True])
def test_mixture_in_both_forms(rows, f, width, dtype, sort):
    """All experts over all rows, and each expert over the rows routed to it; identity experts as a weight per row."""
    m, W = _experts(f, width, dtype, sorted_min_rows=2 if sort else 10 ** 9, force_sorted=sort)
    h = torch.randn(rows, width, generator=_gen(12)).to(torch.bfloat16)
    batch = type("B", (), {"max_new": rows})()
    y, ident = m.forward_parts(h.to(DEV, dtype), batch)
    got = y.cpu().double()
    if ident is not None:
        got = got + ident.cpu().double()[:, None] * h.double()
        from vyomai_b200 import _lib
        with pytest.raises(_lib.VyomError):
            m.forward(h.to(DEV, dtype), batch)
    assert HU.rel_err(got, O.mixture(h.double(), W, f)) < (3e-5 if dtype == torch.float32 else 1.5e-2)


@pytest.mark.parametrize("sort", [False, True])
def test_every_choice_is_an_identity_expert(sort):
    f = U.moe(experts=3, top=2, identity=2, shared=None)
    m, W = _experts(f, 40, torch.float32, sorted_min_rows=2 if sort else 10 ** 9, force_sorted=sort)
    m.correction = torch.tensor([-9.0, -9.0, -9.0, 9.0, 9.0], device=DEV)
    W["correction"] = m.correction.cpu().double()
    h = torch.randn(50, 40, generator=_gen(13))
    y, ident = m.forward_parts(h.to(DEV), type("B", (), {"max_new": 50})())
    assert float(y.abs().max()) == 0.0
    assert HU.rel_err(ident.cpu().double()[:, None] * h.double(), O.mixture(h.double(), W, f)) < 1e-5


# ---- state space ----
def _ssd_op(cuts, *, H=4, G=2, N=9, dv=10, taps=3, ng=2, seed=20, dt_shift=0.0, a_shift=0.0, gate=True, bias=True, wdt=torch.float32):
    """Runs vy_ssd over several sequences, each cut into portions that run side by side in packed steps; returns per sequence
    (got, want, final state, oracle state)."""
    from vyomai_b200 import ops
    g = _gen(seed)
    eps, inner, gn = 1e-5, H * dv, G * N
    ch = inner + 2 * gn
    cw, cb = (torch.randn(ch, taps, generator=g) * 0.5).to(wdt), (torch.randn(ch, generator=g) * 0.3).to(wdt) if bias else None
    a_log, dt_b, D = (torch.rand(H, generator=g) - 1.0 + a_shift).to(wdt), torch.randn(H, generator=g).to(wdt), torch.randn(H, generator=g).to(wdt)
    norm = (1.0 + 0.2 * torch.randn(inner, generator=g)).to(wdt)
    lens = [sum(c) for c in cuts]
    n_slots = len(lens) + 2
    state = torch.full((n_slots, H, N, dv), 5.0, device=DEV)
    conv = torch.full((n_slots, taps, ch), 5.0, device=DEV)
    done = torch.zeros((n_slots, 1), dtype=torch.int32, device=DEV)
    seqs = [{k: torch.randn(n, c, generator=g) for k, c in (("x", inner), ("b", gn), ("c", gn), ("dt", H), ("z", inner))} for n in lens]
    for t in seqs:
        t["dt"] += dt_shift
    dev = lambda t: None if t is None else t.to(DEV)  # noqa: E731
    got, at = [[] for _ in lens], [0] * len(lens)
    slots = list(range(n_slots))[::-1][:len(lens)]
    for step in range(max(len(c) for c in cuts)):
        work = [(s, cuts[s][step]) for s in range(len(lens)) if step < len(cuts[s])]
        cu = [0]
        for _, n in work:
            cu.append(cu[-1] + n)
        batch = ops.PackedBatch(_i32(cu), _i32([at[s] for s, _ in work]), _i32([slots[s] for s, _ in work]), max(n for _, n in work))
        x = {k: dev(torch.cat([seqs[s][k][at[s]:at[s] + n] for s, n in work])) for k in seqs[0]}
        out = ops.ssd(batch, x["x"], x["b"], x["c"], x["dt"], x["z"] if gate else None, dev(cw), dev(cb), conv, dev(dt_b), dev(a_log), dev(D), dev(norm), state, done,
                      heads=H, groups=G, dim=N, vdim=dv, taps=taps, norm_groups=ng, norm_eps=eps).cpu()
        for i, (s, n) in enumerate(work):
            got[s].append(out[cu[i]:cu[i + 1]])
            at[s] += n
    assert int(done.abs().max()) == 0
    for s in set(range(n_slots)) - set(slots):
        assert float((state[s] - 5.0).abs().max()) == 0.0 and float((conv[s] - 5.0).abs().max()) == 0.0     # other sequences' slots untouched
    res = []
    for s, t in enumerate(seqs):
        T = lens[s]
        d = {k: v.double() for k, v in t.items()}
        xbc = O.causal_conv(torch.cat([d["x"], d["b"], d["c"]], 1), cw.double(), cb.double() if bias else torch.zeros(ch, dtype=torch.float64))
        fin = []
        y = O.state_space(xbc[:, :inner].reshape(T, H, dv), xbc[:, inner:inner + gn].reshape(T, G, N), xbc[:, inner + gn:].reshape(T, G, N),
                          O.softplus(d["dt"] + dt_b.double()), a_log.double(), D.double(), state=fin).reshape(T, inner)
        o = O.gate_then_group_norm(y, d["z"], norm.double(), ng, eps) if gate else O.rms(y.view(T, ng, inner // ng), eps).reshape(T, inner) * norm.double()
        res.append((torch.cat(got[s]), o, state[slots[s]].cpu(), torch.stack(fin)))
    return res


@pytest.mark.parametrize("kw", [dict(), dict(H=3, G=1, N=40, dv=33, taps=4, ng=3), dict(H=2, G=2, N=130, dv=8, taps=7, ng=1), dict(H=6, G=2, N=16, dv=140, taps=2, ng=4),
                                dict(H=1, G=1, N=1, dv=2, taps=1, ng=1), dict(H=20, G=4, N=64, dv=12, taps=16, ng=20), dict(H=4, G=1, N=128, dv=64, taps=4, ng=1, wdt=torch.bfloat16),
                                dict(H=8, G=2, N=128, dv=64, taps=4, ng=2), dict(H=4, G=2, N=64, dv=128, taps=3, ng=2), dict(H=2, G=2, N=256, dv=16, taps=4, ng=1), dict(H=2, G=1, N=8, dv=600, taps=3, ng=5), dict(H=1, G=1, N=3, dv=301, taps=2, ng=7), dict(bias=False, gate=False)])
def test_state_space_over_a_packed_batch(kw):
    """Unequal sequences side by side: prompts over several chunks, portions that end off the chunks, a sequence of one token, single tokens
    beside portions, then single tokens only (their own kernel); states, groups, norm groups and taps of unrelated sizes."""
    cuts = [[141, 1, 1], [6, 64, 1, 1], [1, 1, 1], [3, 2, 70, 1, 1, 1]]
    for got, want, st, ost in _ssd_op(cuts, **kw):
        assert HU.rel_err(got, want) < 1e-4 and HU.rel_err(st, ost) < 2e-5


@pytest.mark.parametrize("H,G,N,dv", [(4, 2, 9, 10), (8, 1, 16, 8), (8, 1, 5, 3), (12, 3, 20, 32), (8, 2, 64, 64), (4, 1, 32, 128), (6, 3, 256, 32)])
def test_state_space_single_tokens_of_many_sequences(H, G, N, dv):
    """Batches large enough that a CTA takes two or four heads of a group."""
    cuts = [[1 + s % 3, 1, 1] for s in range(230)]
    got, want, st, ost = (torch.cat(x) if x[0].dim() == 2 else torch.stack(x) for x in zip(*_ssd_op(cuts, H=H, G=G, N=N, dv=dv)))
    assert HU.rel_err(got, want) < 1e-4 and HU.rel_err(st, ost) < 2e-5


@pytest.mark.parametrize("cuts", [[100], [37, 63], [1] * 40])
@pytest.mark.parametrize("dt_shift,a_shift", [(60.0, 1.0), (-60.0, 0.0), (400.0, 3.0), (-8.0, 6.0), (3.0, -12.0)])
def test_state_space_at_extreme_steps(dt_shift, a_shift, cuts):
    """Decays that underflow to 0 in a step, steps so small that nothing is written, long sums of log decays (differences of large sums
    inside a chunk), decays near 1 with large writes."""
    for got, want, st, ost in _ssd_op([cuts], dt_shift=dt_shift, a_shift=a_shift):
        assert bool(torch.isfinite(got).all())
        assert HU.rel_err(got, want) < 2e-4 and HU.rel_err(st, ost) < 1e-4


def test_state_space_remembers_across_chunks():
    """One large write at the first token under a slow decay still stands out 300 tokens later, in chunks and token by token."""
    for cuts in ([320], [300] + [1] * 20, [65] * 4 + [60]):
        (got, want, st, ost), = _ssd_op([cuts], dt_shift=-3.0, a_shift=-7.0)
        assert HU.rel_err(got, want) < 1e-4 and HU.rel_err(st, ost) < 2e-5


# ---- mixers ----
def _run_mixer(mix, h, steps, bs=4):
    """Feeds h [T, width] (one sequence) to the mixer in portions through real pages and a state slot; returns [T, width]."""
    from vyomai_b200 import ops
    from vyomai_b200.paged import LayerCacheView
    T = h.shape[0]
    n_blocks = (T + bs - 1) // bs + 2
    order = torch.randperm(n_blocks, generator=_gen(5)).tolist()
    spec, view = mix.cache_spec(), LayerCacheView()
    if spec["pages"]:
        G, dk, dv = spec["pages"]
        view.k_pool, view.v_pool = torch.zeros((n_blocks, bs, G, dk), device=DEV), torch.zeros((n_blocks, bs, G, dv), device=DEV)
    for name, shape in spec["states"].items():
        dt = spec.get("state_dtypes", {}).get(name, torch.float32)
        view.states[name] = torch.full((3,) + tuple(shape), 0 if dt == torch.int32 else 3.0, device=DEV, dtype=dt)   # what an earlier owner of the slot left
    outs, at = [], 0
    for n in steps:
        batch = ops.PackedBatch(_i32([0, n]), _i32([at]), _i32([2]), n, _i32(order).view(1, -1), bs, all_start=at == 0)
        x = h[at:at + n].to(DEV)
        parts = [ops.linear_plain(x, wt.float(), bias=None if b is None else b.float()) for wt, b in zip(mix.input_weights(), mix.input_biases())]
        outs.append(mix.forward(parts, batch, view).float().cpu())
        at += n
    return torch.cat(outs)


def _weights(kind, m, width, seed):
    from vyomai_b200 import ZaparaxConfig, ZaparaxForCausalLM
    cfg = ZaparaxConfig(U.config([U.layer(kind, m, None)], width=width))
    w = {k[len("l0.mix."):]: v for k, v in ZaparaxForCausalLM.random_weights(cfg, seed=seed).items() if k.startswith("l0.mix.")}
    return {k: v.to(DEV, torch.float32) for k, v in w.items()}, {k: v.double() for k, v in w.items()}


STEPS = [[37], [20, 1, 1, 1, 14], [2] * 18 + [1], [16, 21], [5, 3, 7, 22], [1] * 37]


@pytest.mark.parametrize("steps", STEPS)
@pytest.mark.parametrize("m", [U.attention(window=9), U.attention(heads=8, kv_heads=1, dim=6, vdim=18, window=None, softcap=None), U.attention(heads=1, kv_heads=1, dim=2, vdim=2, window=1, q_temp=None)])
def test_attention_mixer(steps, m):
    from vyomai_b200.layers.mixers import BiasedAttention
    w, W = _weights("attention", m, 40, 6)
    h = torch.randn(37, 40, generator=_gen(7))
    assert HU.rel_err(_run_mixer(BiasedAttention(m, w, 1e-5, torch.float32, True), h, steps), O.attention_mixer(h.double(), W, m, 1e-5)) < 3e-5


@pytest.mark.parametrize("steps", STEPS)
@pytest.mark.parametrize("m", [U.mamba(), U.mamba(heads=3, vdim=33, state=40, groups=1, conv=4, norm_groups=9), U.mamba(heads=2, vdim=8, state=5, groups=2, conv=1, norm_groups=1)])
def test_state_space_mixer(steps, m):
    from vyomai_b200.layers.mixers import StateSpaceMixer
    w, W = _weights("mamba2", m, 40, 8)
    h = torch.randn(37, 40, generator=_gen(9))
    assert HU.rel_err(_run_mixer(StateSpaceMixer(m, w, 1e-5, torch.float32, True), h, steps), O.mamba_mixer(h.double(), W, m, 1e-5)) < 1e-4


def test_ops_refuse_what_they_do_not_take():
    from vyomai_b200 import _lib, ops
    batch, *_ = HU.shuffled_batch([4], [0], 4, DEV)
    z = lambda *s: torch.zeros(*s, device=DEV)  # noqa: E731
    i = lambda *s: torch.zeros(*s, device=DEV, dtype=torch.int32)  # noqa: E731
    with pytest.raises(_lib.VyomError):   # an RMS norm has no bias, whatever the kind is called
        ops.sandwich_norm(z(4, 8), norm2=z(8), eps=1e-5, kind="rms_shifted")
    with pytest.raises(_lib.VyomError):   # a second result goes beside a first one
        ops.sandwich_norm(z(4, 8), norm2=z(8), eps=1e-5, kind="rms", second=(z(4, 8), z(4)))
    with pytest.raises(_lib.VyomError):   # a negative cap
        ops.window_attn(batch, z(4, 8), z(4, 4, 1, 8), z(4, 4, 1, 8), heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0, window=0, keep_first=0, softcap=-1.0)
    with pytest.raises(_lib.VyomError):   # no expert with weights
        ops.moe_route(z(4, 3), 3, 1, 1.0, identity=3)
    with pytest.raises(_lib.VyomError):   # the carried token is an integer
        ops.pair_embed(batch, i(4), z(5, 8), 1.0, z(3, 8), z(5, 1), mul_prev=1, mul_cur=1)
    kw = dict(heads=2, groups=1, dim=8, vdim=4, taps=3, norm_groups=1, norm_eps=1e-5)
    args = lambda **o: {**dict(x=z(4, 8), b=z(4, 8), c=z(4, 8), dt=z(4, 2), gate=None, conv_w=z(24, 3), conv_b=None, conv_state=z(5, 3, 24), dt_bias=z(2), a_log=z(2),  # noqa: E731
                               skip=z(2), norm=z(8), state=z(5, 2, 8, 4), tickets=i(5, 1), **kw), **o}
    ops.ssd(batch, **args())
    for bad in (dict(norm_groups=3), dict(groups=3), dict(conv_state=z(5, 2, 24)), dict(tickets=z(5, 1)), dict(taps=17, conv_w=z(24, 17), conv_state=z(5, 17, 24)), dict(dt=z(4, 1))):
        with pytest.raises(_lib.VyomError):
            ops.ssd(batch, **args(**bad))
