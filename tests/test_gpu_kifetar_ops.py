"""Each Kifetar mechanism alone on the GPU against its float64 statement in oracle/kifetar_oracle.py: the sublayer close (norm, add,
norm), the gated activation, head norm + half-split rotation + page write with the raw keys as values, sigmoid-weighted attention as an
op (window edges, far keys that stand out, many heads per key head) and as a mixer, the gated delta rule with one decay per head as an
op (blocks, portions, single tokens, extreme decays and strengths) and as a mixer. Packed batches mix sequences that start, continue
and advance by one token, over shuffled pages and slots."""
import math

import pytest
import torch

from oracle import kifetar_oracle as O
from tests import hybrid_util as HU
from tests import kifetar_util as U

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _gen(seed):
    return torch.Generator().manual_seed(seed)


@pytest.mark.parametrize("width,wdt", [(7, torch.float32), (40, torch.bfloat16), (250, torch.bfloat16), (1000, torch.bfloat16), (1024, torch.bfloat16), (2048, torch.float32),
                                       (3001, torch.bfloat16), (6000, torch.bfloat16), (9000, torch.bfloat16)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sandwich_norm(width, wdt, dtype):
    """x + norm1(y) into the residual in place, a copy in another dtype, norm2 of the sum; rows with a large mean; then the forms without
    y, without norm2 and with gathered rows."""
    from vyomai_b200 import ops
    g = _gen(0)
    rows, eps = 9, 1e-3
    x, y = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g) * 3.0
    y[2] += 50.0      # the variance is that of the deviations, not of the values
    y[3] = 0.25       # a constant row: only eps and the bias are left
    w1, b1, w2, b2 = ((1.0 + 0.3 * torch.randn(width, generator=g)).to(wdt), torch.randn(width, generator=g).to(wdt),
                      (1.0 + 0.3 * torch.randn(width, generator=g)).to(wdt), torch.randn(width, generator=g).to(wdt))
    d = lambda t: t.to(DEV)  # noqa: E731
    s = x.double() + O.layer_norm(y.double(), w1.double(), b1.double(), eps)
    n = O.layer_norm(s, w2.double(), b2.double(), eps)
    tol = 3e-5 if dtype == torch.float32 else 1e-2
    xd = d(x)
    both = torch.full((rows, 2 * ((width + 7) // 8 * 8)), 9.0, device=DEV, dtype=dtype)
    got = ops.sandwich_norm(xd, d(y), (d(w1), d(b1)), (d(w2), d(b2)), eps=eps, x_out=xd, copy_out=both[:, :width], out_dtype=dtype)
    assert HU.rel_err(xd.cpu(), s) < 3e-5 and HU.rel_err(got.cpu(), n) < tol and HU.rel_err(both[:, :width].cpu(), s) < tol
    assert bool((both[:, width:] == 9.0).all())
    idx = torch.tensor([4, 0, 8, 4], dtype=torch.int32, device=DEV)
    got = ops.sandwich_norm(d(x), norm2=(d(w2), d(b2)), eps=eps, row_index=idx, out_dtype=dtype)
    assert HU.rel_err(got.cpu(), O.layer_norm(x.double(), w2.double(), b2.double(), eps)[[4, 0, 8, 4]]) < tol
    xd = d(x)
    assert ops.sandwich_norm(xd, d(y), (d(w1), d(b1)), eps=eps, x_out=xd) is None and HU.rel_err(xd.cpu(), s) < 3e-5


@pytest.mark.parametrize("ff,dtype", [(5, torch.float32), (44, torch.float32), (1000, torch.bfloat16), (3000, torch.float32)])
def test_gated_activation_over_interleaved_columns(ff, dtype):
    from vyomai_b200 import ops
    z = torch.randn(6, 2 * ff, generator=_gen(1)) * 3.0
    got = ops.glu(z.to(DEV), "silu", dtype).cpu()
    assert HU.rel_err(got, O.silu(z.double()[:, 0::2]) * z.double()[:, 1::2]) < (1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("rows", [3, 32, 33, 100])
@pytest.mark.parametrize("width,ff,dtype", [(40, 44, torch.float32), (128, 192, torch.bfloat16), (256, 40, torch.bfloat16), (64, 36, torch.bfloat16)])
def test_gated_feed_forward(rows, width, ff, dtype):
    """Every form: activation in a tensor-core epilogue, in the small-batch product's epilogue, as its own launch; fp32."""
    from vyomai_b200.layers.mixers import GatedMLP
    g = _gen(2)
    w = {n: (torch.randn(s, generator=g) / math.sqrt(s[1])).to(torch.bfloat16) for n, s in (("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff)))}
    h = torch.randn(rows, width, generator=g).to(torch.bfloat16)
    mlp = GatedMLP({k: v.to(DEV, dtype) for k, v in w.items()}, dtype, True)
    want = O.gated_mlp(h.double(), *(w[n].double() for n in ("gate", "up", "down")))
    assert HU.rel_err(mlp.forward(h.to(DEV, dtype)).cpu(), want) < (2e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("rot_dims,dim", [(8, 12), (12, 12), (0, 10), (64, 200)])
def test_head_norm_rotation_and_raw_keys_into_pages(rot_dims, dim):
    from vyomai_b200 import ops
    H, G, bs, eps = 4, 2, 4, 1e-4
    lengths, pos0 = [9, 1, 5], [0, 3000, 3]
    batch, table, _, n_blocks, _ = HU.shuffled_batch(lengths, pos0, bs, DEV)
    g = _gen(3)
    n = sum(lengths)
    P = torch.randn(n, H * dim + G * dim + 3, generator=g)
    qw, kw = (1.0 + 0.3 * torch.randn(dim, generator=g)).to(torch.bfloat16), (1.0 + 0.3 * torch.randn(dim, generator=g)).to(torch.bfloat16)
    rot = {"base": 40.0, "dims": rot_dims, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40}}
    f = torch.tensor(O.frequencies(rot) or [0.0]).float().to(DEV)
    kp, vp = (torch.full((n_blocks, bs, G, dim), 7.0, device=DEV) for _ in range(2))
    Pd = P.to(DEV)
    q, k = Pd[:, :H * dim], Pd[:, H * dim:H * dim + G * dim]
    ops.rope_kv_write(batch, q, k, k, f, kp, vp, heads=H, kv_heads=G, dim=dim, vdim=dim, rot_dims=rot_dims, layout="half", eps=eps,
                      q_norm=qw.to(DEV), k_norm=kw.to(DEV))
    at = 0
    for s, (ln, p) in enumerate(zip(lengths, pos0)):
        qs, kraw = P[at:at + ln, :H * dim].double().view(ln, H, dim), P[at:at + ln, H * dim:H * dim + G * dim].double().view(ln, G, dim)
        pad = lambda t: torch.cat([torch.zeros(p, *t.shape[1:], dtype=torch.float64), t])  # noqa: E731
        qs, ks = (O.rotate_half(pad(O.rms(t, eps) * w.double()), rot)[p:] for t, w in ((qs, qw), (kraw, kw)))
        tol = 4e-3 if p > 1000 else 1e-5     # fp32 angles: 3000 * 2^-24 rad
        assert float((Pd[at:at + ln, :H * dim].cpu().double().view(ln, H, dim) - qs).abs().max()) < tol
        for i in range(ln):
            blk, off = table[s][(p + i) // bs], (p + i) % bs
            assert float((kp[blk, off].cpu().double() - ks[i]).abs().max()) < tol
            assert torch.equal(vp[blk, off].cpu().double(), kraw[i])
        at += ln
    assert torch.equal(Pd[:, H * dim:].cpu(), P[:, H * dim:])              # the projected keys stay as they are
    assert int((kp == 7.0).all(-1).all(-1).sum()) == n_blocks * bs - n    # nothing else was written


@pytest.mark.parametrize("H,G,d", [(4, 2, 8), (8, 1, 8), (16, 2, 12), (3, 3, 10), (4, 1, 130)])
@pytest.mark.parametrize("window,bs", [(1, 4), (7, 4), (16, 16), (64, 16), (100, 8), (0, 8)])
def test_sigmoid_attention_over_pages(H, G, d, window, bs):
    """Four sequences in one step and each alone: a whole prompt, a long portion that starts inside a window, a portion of a few tokens,
    a single token (alone it takes the single-token forms). Keys just inside and just outside the last query's window are made to stand
    out, each with a value of its own."""
    from vyomai_b200 import ops
    scale, far = 0.5, (window or 60)
    T = [2 * far + 35, far + 24, far + 9, far + 5]
    new = [T[0], 20, 5, 1]
    g = _gen(5)
    temp, bias = 1.0 + torch.rand(H, generator=g), torch.randn(H, generator=g) - 1.0
    qs = [torch.randn(t, H, d, generator=g).double() / d ** 0.25 for t in T]
    ks = [torch.randn(t, G, d, generator=g).double() / d ** 0.25 for t in T]
    vs = [torch.randn(t, G, d, generator=g).double() for t in T]
    gate = [torch.randn(t, H, generator=g).double() for t in T]
    for s, t in enumerate(T):
        for back, val in ((far - 1, 4.0), (far, -6.0)):   # the window's last key and the first one out of it
            j = t - 1 - back
            if j >= 0:
                ks[s][j] = 3.0 * qs[s][t - 1].view(G, H // G, d).mean(1)
                vs[s][j] += val
    pos0 = [t - n for t, n in zip(T, new)]
    want = [O.sigmoid_attention(qs[s], ks[s], vs[s], scale=scale, window=window, temp=temp.double(), bias=bias.double(), gate_logits=gate[s])[pos0[s]:].reshape(new[s], -1)
            for s in range(4)]
    for group in ([0, 1, 2, 3], [0], [1], [2], [3]):
        batch, table, _, n_blocks, _ = HU.shuffled_batch([new[s] for s in group], [pos0[s] for s in group], bs, DEV, seed=window)
        kp = torch.full((n_blocks, bs, G, d), 1e3, device=DEV)      # rows no query may read
        vp = torch.full((n_blocks, bs, G, d), 1e3, device=DEV)
        for n, s in enumerate(group):
            for p in range(T[s]):
                blk, off = table[n][p // bs], p % bs
                kp[blk, off], vp[blk, off] = ks[s][p].float().to(DEV), vs[s][p].float().to(DEV)
        q = torch.cat([qs[s][pos0[s]:].reshape(new[s], H * d) for s in group]).float().to(DEV)
        gt = torch.cat([gate[s][pos0[s]:] for s in group]).float().to(DEV)
        got = ops.window_attn(batch, q, kp, vp, heads=H, kv_heads=G, dim=d, vdim=d, scale=scale, window=window, keep_first=0, gate=gt,
                              weights="sigmoid", head_scale=temp.to(DEV), head_bias=bias.to(DEV)).cpu()
        assert HU.rel_err(got, torch.cat([want[s] for s in group])) < 3e-5, group


def test_softmax_attention_takes_the_per_head_scale_and_bias_too():
    """Softmax weights with a sink: the bias is not the same as no bias (the sink does not get it)."""
    from vyomai_b200 import ops
    H, d, T = 2, 6, 20
    g = _gen(6)
    q, k, v = (torch.randn(T, H * d, generator=g) for _ in range(3))
    hs, hb, sink = torch.tensor([0.5, 2.0]), torch.tensor([1.0, -1.5]), torch.tensor([0.3, -0.2])
    for n in (T, 5, 1):
        p0 = T - n
        batch, table, *_ = HU.shuffled_batch([n], [p0], 4, DEV)
        kp, vp = torch.zeros((9, 4, H, d), device=DEV), torch.zeros((9, 4, H, d), device=DEV)
        for p in range(T):
            kp[table[0][p // 4], p % 4], vp[table[0][p // 4], p % 4] = k[p].view(H, d).to(DEV), v[p].view(H, d).to(DEV)
        got = ops.window_attn(batch, q[p0:].to(DEV), kp, vp, heads=H, kv_heads=H, dim=d, vdim=d, scale=0.4, window=0, keep_first=0, sink=sink.to(DEV),
                              head_scale=hs.to(DEV), head_bias=hb.to(DEV)).cpu()
        for h in range(H):
            s = (q.view(T, H, d)[:, h].double() @ k.view(T, H, d)[:, h].double().T) * 0.4 * float(hs[h]) + float(hb[h])
            e = torch.exp(s) * torch.tril(torch.ones(T, T, dtype=torch.float64))
            want = (e / (e.sum(1, keepdim=True) + math.exp(float(sink[h])))) @ v.view(T, H, d)[:, h].double()
            assert HU.rel_err(got.view(n, H, d)[:, h], want[p0:]) < 2e-5


def _views(spec, n_blocks, bs, n_slots):
    from vyomai_b200.paged import LayerCacheView
    view = LayerCacheView()
    if spec["pages"]:
        G, dk, dv = spec["pages"]
        view.k_pool, view.v_pool = torch.zeros((n_blocks, bs, G, dk), device=DEV), torch.zeros((n_blocks, bs, G, dv), device=DEV)
    for name, shape in spec["states"].items():
        view.states[name] = torch.full((n_slots,) + tuple(shape), 3.0, device=DEV)   # what an earlier owner of the slot left
    return view


def _run_mixer(mix, h, steps, bs=4):
    """Feeds h [T, width] (one sequence) to the mixer in portions through real pages and a state slot; returns [T, width]."""
    from vyomai_b200 import ops
    T = h.shape[0]
    n_blocks = (T + bs - 1) // bs + 2
    order = torch.randperm(n_blocks, generator=_gen(5)).tolist()
    view = _views(mix.cache_spec(), n_blocks, bs, 3)
    t = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)  # noqa: E731
    outs, at = [], 0
    for n in steps:
        batch = ops.PackedBatch(t([0, n]), t([at]), t([2]), n, t(order).view(1, -1), bs, all_start=at == 0)
        x = h[at:at + n].to(DEV)
        parts = [ops.linear_plain(x, wt.float(), bias=None if b is None else b.float()) for wt, b in zip(mix.input_weights(), mix.input_biases())]
        outs.append(mix.forward(parts, batch, view).float().cpu())
        at += n
    return torch.cat(outs), view


def _weights(kind, m, width, seed):
    from vyomai_b200 import KifetarConfig, KifetarForCausalLM
    cfg = KifetarConfig(U.config([U.layer(kind, m, None)], width=width))
    w = {k[len("l0.mix."):]: v for k, v in KifetarForCausalLM.random_weights(cfg, seed=seed).items() if k.startswith("l0.mix.")}
    return {k: v.to(DEV, torch.float32) for k, v in w.items()}, {k: v.double() for k, v in w.items()}


STEPS = [[37], [20, 1, 1, 1, 14], [2] * 18 + [1], [16, 21], [5, 3, 7, 22], [1] * 37]


@pytest.mark.parametrize("steps", STEPS)
@pytest.mark.parametrize("m", [U.attention(window=9, scaling=U.LENGTHEN), U.attention(heads=8, kv_heads=1, dim=6, window=None, rot_dims=None), U.attention(heads=1, kv_heads=1, dim=2, window=1, rot_dims=2)])
def test_attention_mixer(steps, m):
    from vyomai_b200.layers.mixers import SigmoidAttention
    w, W = _weights("attention", m, 40, 6)
    h = torch.randn(37, 40, generator=_gen(7))
    got, _ = _run_mixer(SigmoidAttention(m, w, 1e-5, torch.float32, True), h, steps)
    assert HU.rel_err(got, O.attention_mixer(h.double(), W, m, 1e-5)) < 3e-5


@pytest.mark.parametrize("steps", STEPS)
@pytest.mark.parametrize("m", [U.delta(), U.delta(heads=3, kv_heads=1, dim=40, vdim=33, conv=4), U.delta(heads=2, kv_heads=2, dim=5, vdim=70, conv=1),
                               U.delta(heads=2, kv_heads=1, dim=130, vdim=8, conv=7), U.delta(heads=1, kv_heads=1, dim=96, vdim=140, conv=2)])
def test_delta_mixer(steps, m):
    from vyomai_b200.layers.mixers import HeadDecayDeltaMixer
    w, W = _weights("delta", m, 40, 8)
    h = torch.randn(37, 40, generator=_gen(9))
    got, view = _run_mixer(HeadDecayDeltaMixer(m, w, 1e-5, torch.float32, True), h, steps)
    assert HU.rel_err(got, O.delta_mixer(h.double(), W, m, 1e-5)) < 1e-4
    for st in view.states.values():
        assert float((st[:2] - 3.0).abs().max()) == 0.0    # other sequences' slots untouched


def _delta_op(lens, pos_cuts, *, H=4, G=2, dk=8, dv=12, taps=3, seed=20, a_shift=0.0, b_shift=0.0, gate=True, same_key=False):
    """Runs vy_gated_delta over several sequences, each cut into portions that run side by side in packed steps; returns per sequence
    (got, want, final state, oracle state)."""
    from vyomai_b200 import ops
    g = _gen(seed)
    eps = 1e-5
    cw = [torch.randn(c, taps, generator=g) * 0.5 for c in (G * dk, G * dk, H * dv)]
    a_log, norm = torch.rand(H, generator=g) - 1.0, 1.0 + 0.2 * torch.randn(dv, generator=g)
    n_slots = len(lens) + 2
    state = torch.full((n_slots, H, dk, dv), 5.0, device=DEV)
    conv = torch.full((n_slots, taps, 2 * G * dk + H * dv), 5.0, device=DEV)
    seqs = []
    for n in lens:
        t = {k: torch.randn(n, c, generator=g) for k, c in (("q", G * dk), ("k", G * dk), ("v", H * dv), ("a", H), ("b", H), ("g", H * dv))}
        t["a"] += a_shift
        t["b"] += b_shift
        if same_key:
            t["k"][:] = t["k"][0]
        seqs.append(t)
    dev = lambda t: t.to(DEV)  # noqa: E731
    got, at = [[] for _ in lens], [0] * len(lens)
    slots = list(range(n_slots))[::-1][:len(lens)]
    for step in range(max(len(c) for c in pos_cuts)):
        work = [(s, pos_cuts[s][step]) for s in range(len(lens)) if step < len(pos_cuts[s])]
        ti = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)  # noqa: E731
        cu = [0]
        for _, n in work:
            cu.append(cu[-1] + n)
        batch = ops.PackedBatch(ti(cu), ti([at[s] for s, _ in work]), ti([slots[s] for s, _ in work]), max(n for _, n in work))
        x = {k: dev(torch.cat([seqs[s][k][at[s]:at[s] + n] for s, n in work])) for k in "qkvabg"}
        out = ops.gated_delta(batch, x["q"], x["k"], x["v"], x["a"], x["b"], x["g"] if gate else None, [dev(w) for w in cw], conv, dev(a_log), dev(norm), state,
                              heads=H, kv_heads=G, dim=dk, vdim=dv, taps=taps, norm_eps=eps).cpu()
        for i, (s, n) in enumerate(work):
            got[s].append(out[cu[i]:cu[i + 1]])
            at[s] += n
    res = []
    for s, t in enumerate(seqs):
        T = lens[s]
        d = {k: v.double() for k, v in t.items()}
        q = O.unit(O.causal_conv(d["q"], cw[0].double()).view(T, G, dk)) * dk ** -0.5
        k = O.unit(O.causal_conv(d["k"], cw[1].double()).view(T, G, dk))
        v = O.causal_conv(d["v"], cw[2].double()).view(T, H, dv)
        decay = torch.exp(-torch.exp(a_log.double()) * torch.nn.functional.softplus(d["a"], threshold=1e9))
        fin = []
        o = O.rms(O.gated_delta_rule(q, k, v, decay, torch.sigmoid(d["b"]), state=fin), eps) * norm.double()
        if gate:
            o = o * O.silu(d["g"]).view(T, H, dv)
        res.append((torch.cat(got[s]), o.reshape(T, H * dv), state[slots[s]].cpu(), torch.stack(fin)))
    return res


@pytest.mark.parametrize("dk,dv,taps", [(8, 12, 3), (128, 128, 4), (64, 36, 16), (200, 40, 2), (3, 2, 1)])
def test_delta_rule_over_a_packed_batch(dk, dv, taps):
    """Unequal sequences side by side: a long prompt, portions that end off the blocks of four, a sequence of one token, single tokens
    beside portions, then single tokens only (their own kernel)."""
    cuts = [[41, 1, 1], [6, 17, 1, 1], [1, 1, 1], [3, 2, 9, 1, 1, 1]]
    for got, want, st, ost in _delta_op([sum(c) for c in cuts], cuts, dk=dk, dv=dv, taps=taps):
        assert HU.rel_err(got, want) < 1e-4 and HU.rel_err(st, ost) < 2e-5


@pytest.mark.parametrize("cuts", [[40], [13, 27], [1] * 40])
@pytest.mark.parametrize("a_shift,b_shift,same_key", [(60.0, 0.0, False), (-60.0, 30.0, True), (-60.0, -30.0, False), (400.0, 30.0, False)])
def test_delta_rule_at_extreme_decays_and_strengths(a_shift, b_shift, same_key, cuts):
    """Decays that underflow to 0 (every block starts from nothing), decays of 1 with full overwrites under ONE key, strength 0 (the state
    stays empty: the read-out is 0 and only eps holds the norm up)."""
    for got, want, st, ost in _delta_op([40], [cuts], a_shift=a_shift, b_shift=b_shift, same_key=same_key):
        assert bool(torch.isfinite(got).all())
        if b_shift < 0:
            assert float((got.double() - want).abs().max()) < 1e-6
        else:
            assert HU.rel_err(got, want) < 2e-4 and HU.rel_err(st, ost) < 1e-4


def test_delta_rule_without_a_gate():
    for got, want, _, _ in _delta_op([9], [[7, 1, 1]], gate=False):
        assert HU.rel_err(got, want) < 1e-4


def test_ops_refuse_what_they_do_not_take():
    from vyomai_b200 import _lib, ops
    batch, *_ = HU.shuffled_batch([4], [0], 4, DEV)
    q = torch.zeros(4, 8, device=DEV)
    pool = torch.zeros(4, 4, 1, 8, device=DEV)
    with pytest.raises(_lib.VyomError):   # a sink belongs to a softmax
        ops.window_attn(batch, q, pool, pool, heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0, window=0, keep_first=0, weights="sigmoid", sink=torch.zeros(1, device=DEV))
    with pytest.raises(_lib.VyomError):   # a norm before the rotation and one after it
        ops.rope_kv_write(batch, q, q, q, torch.zeros(1, device=DEV), pool, pool.clone(), heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=2, unit_rms=True,
                          q_norm=torch.ones(8, device=DEV))
    z = lambda *s: torch.zeros(*s, device=DEV)  # noqa: E731
    with pytest.raises(_lib.VyomError):   # 17 taps
        ops.gated_delta(batch, z(4, 8), z(4, 8), z(4, 8), z(4, 1), z(4, 1), None, [z(8, 17)] * 3, z(5, 17, 24), z(1), z(8), z(5, 1, 8, 8), heads=1, kv_heads=1,
                        dim=8, vdim=8, taps=17, norm_eps=1e-5)
