"""Host-side pieces of the Kifetar family that need no GPU: the configuration's checks, run order and tensor list, the registry, the
cache specs (one per layer run: a looped layer owns pages and states per pass), the frequency table, and the oracle's own mechanisms
against brute-force loops and closed forms."""
import math

import pytest
import torch

from oracle import kifetar_oracle as O
from tests import kifetar_util as U


def test_config_lists_the_tensors_of_every_layer_kind():
    from vyomai_b200 import KifetarConfig
    s = KifetarConfig(U.small_config()).tensor_shapes()
    assert s["embed"] == (97, 40) and "head" not in s and s["loop.in"] == (40, 80) and s["final.norm.b"] == (40,)
    assert s["l0.mix.q"] == (48, 40) and s["l0.mix.q.b"] == (48,) and s["l0.mix.k"] == (24, 40) and s["l0.mix.q.norm"] == (12,) and "l0.mix.v" not in s
    assert s["l0.mix.temp"] == (4,) and s["l0.mix.pb"] == (4,) and s["l0.mix.g"] == (4, 40) and s["l0.mix.o"] == (40, 48)
    assert s["l1.mix.q"] == (20, 40) and s["l1.mix.v"] == (56, 40) and s["l1.mix.v.conv"] == (56, 3) and s["l1.mix.g"] == (56, 40)
    assert s["l1.mix.a"] == (4, 40) and s["l1.mix.dt_bias"] == (4,) and s["l1.mix.norm"] == (14,) and s["l1.mix.o"] == (40, 56)
    assert s["l2.norm1b.b"] == (40,) and "l2.norm2" not in s and "l2.mlp.up" not in s and s["l3.mlp.gate"] == (20, 40) and s["l3.norm2b"] == (40,)
    assert "loop.in" not in KifetarConfig(U.many_heads_config()).tensor_shapes()


@pytest.mark.parametrize("bad", ["heads", "vdim", "rot", "type", "kind", "loop_empty", "loop_past", "loop_times", "arch", "taps"])
def test_config_rejects_what_the_design_does_not_have(bad):
    from vyomai_b200 import KifetarConfig
    d = U.small_config()
    if bad == "heads":
        d["layers"][1]["mixer"]["kv_heads"] = 3
    elif bad == "vdim":
        d["layers"][0]["mixer"]["vdim"] = 8
    elif bad == "rot":
        d["layers"][0]["mixer"]["rot"]["dims"] = 14
    elif bad == "type":
        d["layers"][0]["type"] = "retention"
    elif bad == "kind":
        d["layers"][0]["mlp"]["kind"] = "moe"
    elif bad == "loop_empty":
        d["loop"]["stop"] = d["loop"]["start"]
    elif bad == "loop_past":
        d["loop"]["stop"] = 6
    elif bad == "loop_times":
        d["loop"]["times"] = 0
    elif bad == "arch":
        d["architecture"] = "Gelutar"
    else:
        d["layers"][1]["mixer"]["conv"] = 0
    with pytest.raises(ValueError):
        KifetarConfig(d)


def test_registry_knows_the_architecture():
    from vyomai_b200.registry import architectures
    assert "Kifetar" in architectures()


def test_loop_runs_and_a_cache_per_pass():
    from vyomai_b200 import KifetarConfig, KifetarForCausalLM
    from vyomai_b200.paged import HybridCacheManager
    cfg = KifetarConfig(U.small_config())
    assert [i for i, _ in cfg.runs()] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] and [n for n, (_, o) in enumerate(cfg.runs()) if o] == [1, 4, 7]
    assert cfg.runs() == O.layer_runs(cfg.raw)
    assert KifetarConfig(U.aligned_config()).runs() == [(0, True), (1, False), (0, True), (1, False), (2, False)]
    assert KifetarConfig(U.many_heads_config()).runs() == [(0, False), (1, False), (2, False)]
    model = KifetarForCausalLM(cfg, KifetarForCausalLM.random_weights(cfg), dtype=torch.float32, device="cpu")
    specs = model.cache_specs()
    assert len(specs) == 11 and specs[0][0]["pages"] == (2, 12, 12) and specs[1] == [{"pages": None, "states": {"S": (4, 10, 14), "conv": (3, 96)}}]
    assert specs[1] == specs[4] == specs[7] and specs[2][0]["pages"] == (3, 6, 6)
    mgr = HybridCacheManager(model, max_tokens=16, block_size=4, max_seqs=2, device="cpu")
    assert mgr.views[1][0].states["S"].data_ptr() != mgr.views[4][0].states["S"].data_ptr() and mgr.views[2][0].k_pool.data_ptr() != mgr.views[5][0].k_pool.data_ptr()
    assert mgr.views[1][0].states["S"].shape == (2, 4, 10, 14) and mgr.views[0][0].v_pool.shape[1:] == (4, 2, 12)


def test_checkpoint_shapes_are_checked():
    from vyomai_b200 import KifetarConfig, KifetarForCausalLM
    cfg = KifetarConfig(U.small_config())
    w = KifetarForCausalLM.random_weights(cfg)
    bad = dict(w)
    bad["l0.mix.temp"] = bad["l0.mix.temp"][:3]
    with pytest.raises(ValueError):
        KifetarForCausalLM(cfg, bad, dtype=torch.float32, device="cpu")
    del bad["l0.mix.temp"]
    with pytest.raises(KeyError):
        KifetarForCausalLM(cfg, bad, dtype=torch.float32, device="cpu")


def test_frequency_table_follows_the_wavelength_rule():
    """The table the mixer hands to the kernels against the definition where every branch comes up, and the branches' limits."""
    from vyomai_b200.layers.mixers import rotary_frequencies
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 256}}
    f, m = rotary_frequencies(rot, 32, "cpu")
    want = torch.tensor(O.frequencies(rot), dtype=torch.float64)
    assert m == 1.0 and float(((f.double() - want) / want).abs().max()) < 1e-7
    plain = torch.tensor([10000.0 ** (-2.0 * i / 32) for i in range(16)], dtype=torch.float64)
    ratio, wave = want / plain, 2 * math.pi / plain
    assert bool((ratio[wave < 64] == 1.0).all()) and bool(((ratio[wave > 256] - 0.125).abs() < 1e-12).all())
    mid = (wave >= 64) & (wave <= 256)
    assert int(mid.sum()) >= 2 and bool(((ratio[mid] > 0.125) & (ratio[mid] < 1.0)).all())
    s = (256 / wave[mid] - 1.0) / 3.0
    assert float((ratio[mid] - ((1 - s) / 8 + s)).abs().max()) < 1e-12
    # the other scaling rule keeps its own keys
    g, gm = rotary_frequencies({"base": 100.0, "dims": 8, "scaling": {"factor": 2.0, "original": 32, "fast": 16.0, "slow": 2.0}}, 8, "cpu")
    assert gm > 1.0 and g.numel() == 4


def test_oracle_attention_by_hand():
    """One head: the output is the plain sum of sigmoid-weighted values inside the window; doubling every key's weight doubles it (no
    normalisation over keys)."""
    g = torch.Generator().manual_seed(0)
    T, d, n = 6, 3, 2
    q, k = torch.randn(T, 1, d, generator=g, dtype=torch.float64), torch.randn(T, 1, d, generator=g, dtype=torch.float64)
    v = torch.randn(T, 1, 2, generator=g, dtype=torch.float64)
    one, half = torch.tensor([1.5], dtype=torch.float64), torch.tensor([-0.5], dtype=torch.float64)
    got = O.sigmoid_attention(q, k, v, scale=0.7, window=n, temp=one, bias=half, gate_logits=torch.full((T, 1), 40.0, dtype=torch.float64))
    for i in range(T):
        want = sum(v[j, 0] / (1.0 + math.exp(-(float(q[i, 0] @ k[j, 0]) * 0.7 * 1.5 - 0.5))) for j in range(max(0, i - n + 1), i + 1))
        assert float((got[i, 0] - want).abs().max()) < 1e-12


def test_oracle_delta_rule_stores_and_overwrites():
    """Strength 1, decay 1, orthonormal keys: reading a key returns the last value written under it."""
    e = torch.eye(3, dtype=torch.float64)
    k = torch.stack([e[0], e[1], e[0]])[:, None]
    q = torch.stack([e[0], e[0], e[0]])[:, None]
    v = torch.tensor([[[1.0, 2.0]], [[5.0, 6.0]], [[7.0, 8.0]]], dtype=torch.float64)
    ones = torch.ones(3, 1, dtype=torch.float64)
    o = O.gated_delta_rule(q, k, v, ones, ones)
    assert torch.equal(o[:, 0], torch.tensor([[1.0, 2.0], [1.0, 2.0], [7.0, 8.0]], dtype=torch.float64))
    o = O.gated_delta_rule(q, k, v, 0.5 * ones, ones)     # the state halves before every write
    assert torch.equal(o[:, 0], torch.tensor([[1.0, 2.0], [0.5, 1.0], [7.0, 8.0]], dtype=torch.float64))


def test_oracle_convolution_and_norms():
    x = torch.arange(1.0, 5.0, dtype=torch.float64)[:, None]
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64)     # the last column is the current token's
    assert float((O.causal_conv(x, w) - O.silu(torch.tensor([[1.0], [12.0], [123.0], [234.0]], dtype=torch.float64))).abs().max()) < 1e-12
    y = O.layer_norm(torch.tensor([[1.0, 3.0]], dtype=torch.float64), torch.tensor([2.0, 2.0]), torch.tensor([0.5, 0.5]), 0.0)
    assert torch.equal(y, torch.tensor([[-1.5, 2.5]], dtype=torch.float64))


def test_oracle_rotation_is_relative_and_partial():
    rot = {"base": 20.0, "dims": 4}
    g = torch.Generator().manual_seed(1)
    a, b = torch.randn(6, generator=g, dtype=torch.float64), torch.randn(6, generator=g, dtype=torch.float64)
    ra, rb = O.rotate_half(a.repeat(50, 1)[:, None], rot)[:, 0], O.rotate_half(b.repeat(50, 1)[:, None], rot)[:, 0]
    s = [float(ra[p + 3] @ rb[p]) for p in (0, 5, 40)]
    assert abs(s[0] - s[1]) < 1e-12 and abs(s[0] - s[2]) < 1e-12 and torch.equal(ra[7, 4:], a[4:])
    assert abs(float(ra[7, 0]) - (float(a[0]) * math.cos(7.0) - float(a[2]) * math.sin(7.0))) < 1e-12
    assert abs(float(ra[7, 2]) - (float(a[2]) * math.cos(7.0) + float(a[0]) * math.sin(7.0))) < 1e-12
