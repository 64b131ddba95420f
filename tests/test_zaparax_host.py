"""Host-side pieces of the Zaparax family that need no GPU: the configuration's checks, run order and tensor list, the registry, the
cache specs (one entry for the embedding and one per layer RUN), and the oracle's own mechanisms against brute-force loops and closed
forms."""
import math

import pytest
import torch

from oracle import zaparax_oracle as O
from tests import zaparax_util as U


def test_config_lists_the_tensors_of_every_layer_kind():
    from vyomai_b200 import ZaparaxConfig
    s = ZaparaxConfig(U.small_config()).tensor_shapes()
    assert s["embed"] == (97, 40) and s["head"] == (97, 40) and s["bigram"] == (54, 40) and s["final.norm"] == (40,)
    assert s["l0.mix.q"] == (48, 40) and s["l0.mix.q.b"] == (48,) and s["l0.mix.k"] == (24, 40) and s["l0.mix.v"] == (20, 40) and s["l0.mix.v.b"] == (20,)
    assert s["l0.mix.sink"] == (4,) and s["l0.mix.o"] == (40, 40) and s["l0.norm2b"] == (40,)
    assert s["l0.mlp.e4.gate"] == (20, 40) and "l0.mlp.e5.gate" not in s and s["l0.mlp.router"] == (7, 40) and s["l0.mlp.correction"] == (7,)
    assert s["l0.mlp.shared.down"] == (40, 28) and s["l0.mlp.shared.sg"] == (1, 40)
    assert s["l1.mix.in"] == (2 * 40 + 2 * 18 + 4, 40) and s["l1.mix.conv"] == (76, 3) and s["l1.mix.conv.b"] == (76,) and s["l1.mix.norm"] == (40,)
    assert s["l1.mix.D"] == (4,) and s["l1.mix.o"] == (40, 40)
    assert "l2.norm2" not in s and "l2.mlp.router" not in s and s["l3.mlp.router"] == (4, 40) and "l3.mlp.shared.sg" not in s
    assert "bigram" not in ZaparaxConfig(U.config([], bigram=None)).tensor_shapes()


@pytest.mark.parametrize("bad", ["heads", "groups", "norm_groups", "type", "kind", "top", "every", "buckets", "loop_empty", "loop_past", "loop_times", "arch", "taps"])
def test_config_rejects_what_the_design_does_not_have(bad):
    from vyomai_b200 import ZaparaxConfig
    d = U.small_config()
    if bad == "heads":
        d["layers"][0]["mixer"]["kv_heads"] = 3
    elif bad == "groups":
        d["layers"][1]["mixer"]["groups"] = 3
    elif bad == "norm_groups":
        d["layers"][1]["mixer"]["norm_groups"] = 7
    elif bad == "type":
        d["layers"][0]["type"] = "delta"
    elif bad == "kind":
        d["layers"][0]["mlp"]["kind"] = "dense"
    elif bad == "top":
        d["layers"][0]["mlp"]["router"]["top"] = 8
    elif bad == "every":
        d["layers"][0]["mixer"]["q_temp"]["every"] = 0
    elif bad == "buckets":
        d["embedding"]["bigram"]["buckets"] = 0
    elif bad == "loop_empty":
        d["loop"]["stop"] = d["loop"]["start"]
    elif bad == "loop_past":
        d["loop"]["stop"] = 6
    elif bad == "loop_times":
        d["loop"]["times"] = 0
    elif bad == "arch":
        d["architecture"] = "Kifetar"
    else:
        d["layers"][1]["mixer"]["conv"] = 0
    with pytest.raises(ValueError):
        ZaparaxConfig(d)


def test_registry_knows_the_architecture():
    from vyomai_b200.registry import architectures
    assert "Zaparax" in architectures()


def test_loop_runs_and_a_cache_per_pass():
    from vyomai_b200 import ZaparaxConfig, ZaparaxForCausalLM
    from vyomai_b200.paged import HybridCacheManager
    cfg = ZaparaxConfig(U.small_config())
    assert cfg.runs() == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4] == O.layer_runs(cfg.raw)
    assert ZaparaxConfig(U.many_heads_config()).runs() == [0, 1, 2, 3]
    model = ZaparaxForCausalLM(cfg, ZaparaxForCausalLM.random_weights(cfg), dtype=torch.float32, device="cpu")
    specs = model.cache_specs()
    assert len(specs) == 12 and specs[0][0]["states"] == {"prev": (1,)} and specs[1][0]["pages"] == (2, 12, 10)
    assert specs[2][0]["states"] == {"S": (4, 9, 10), "conv": (3, 76), "done": (1,)} and specs[2] == specs[5] == specs[8]
    mgr = HybridCacheManager(model, max_tokens=16, block_size=4, max_seqs=2, device="cpu")
    assert mgr.views[2][0].states["S"].data_ptr() != mgr.views[5][0].states["S"].data_ptr() and mgr.views[3][0].k_pool.data_ptr() != mgr.views[6][0].k_pool.data_ptr()
    assert mgr.views[0][0].states["prev"].dtype == torch.int32 and mgr.views[2][0].states["done"].dtype == torch.int32
    assert mgr.views[2][0].states["S"].dtype == torch.float32 and mgr.views[1][0].v_pool.shape[1:] == (4, 2, 10)
    mgr.views[0][0].states["prev"][1, 0] = 7
    mgr._grow_slots(3)     # growing keeps what the slots hold, in its own type
    assert mgr.views[0][0].states["prev"].shape == (5, 1) and int(mgr.views[0][0].states["prev"][1, 0]) == 7


def test_checkpoint_shapes_are_checked():
    from vyomai_b200 import ZaparaxConfig, ZaparaxForCausalLM
    cfg = ZaparaxConfig(U.small_config())
    bad = dict(ZaparaxForCausalLM.random_weights(cfg))
    bad["l0.mlp.correction"] = bad["l0.mlp.correction"][:5]
    with pytest.raises(ValueError):
        ZaparaxForCausalLM(cfg, bad, dtype=torch.float32, device="cpu")
    del bad["l0.mlp.correction"]
    with pytest.raises(KeyError):
        ZaparaxForCausalLM(cfg, bad, dtype=torch.float32, device="cpu")


def test_oracle_bigram_rows():
    assert O.bigram_rows([4, 9, 4], 3, 10, 7) == [7, (12 + 90) % 7, (27 + 40) % 7]
    table, pairs = torch.eye(10, dtype=torch.float64), 100.0 * torch.arange(8, dtype=torch.float64)[:, None].repeat(1, 10)
    x = O.embedding([4, 9], table, 0.5, pairs, {"buckets": 7, "mul_prev": 3, "mul_cur": 10})
    assert float(x[0, 4]) == 700.5 and float(x[0, 0]) == 700.0 and float(x[1, 9]) == 100.0 * (102 % 7) + 0.5


def test_oracle_query_temperature():
    t = O.query_temperature(9, 0.5, 4)
    assert [float(v) for v in t[:3]] == [1.0, 1.0, 1.0] and float(t[3]) == 1.0 + 0.5 * math.log(2.0) == float(t[6]) and float(t[7]) == 1.0 + 0.5 * math.log(3.0)


def test_oracle_attention_by_hand():
    """Two heads over one key head: capped scores, the bias per distance, the window, the sink in the denominator only."""
    g = torch.Generator().manual_seed(0)
    T, d, n, cap = 6, 3, 3, 0.8
    q, k = torch.randn(T, 2, d, generator=g, dtype=torch.float64), torch.randn(T, 1, d, generator=g, dtype=torch.float64)
    v = torch.randn(T, 1, 2, generator=g, dtype=torch.float64)
    sink = torch.tensor([0.4, -2.0], dtype=torch.float64)
    assert O.head_slopes(2) == [2.0 ** -4, 2.0 ** -8] and O.head_slopes(1) == [2.0 ** -8]
    got = O.biased_attention(q, k, v, scale=0.7, softcap=cap, window=n, slopes=O.head_slopes(2), sink=sink)
    for h in range(2):
        for i in range(T):
            w = {j: math.exp(cap * math.tanh(float(q[i, h] @ k[j, 0]) * 0.7 / cap) - 2.0 ** (-4 * (h + 1)) * (i - j)) for j in range(max(0, i - n + 1), i + 1)}
            want = sum(a * v[j, 0] for j, a in w.items()) / (sum(w.values()) + math.exp(float(sink[h])))
            assert float((got[i, h] - want).abs().max()) < 1e-12
    # a constant shift of all scores (slope * j in place of slope * (i - j)) is not the same beside a sink
    rows = O.biased_attention(q, k, v, scale=0.7, softcap=0.0, window=0, slopes=[0.0, 0.0], sink=None)
    assert float((rows[0, 0] - v[0, 0]).abs().max()) < 1e-12


def test_oracle_state_space_by_hand():
    """One head, N = 1: a leaky sum; D passes x through."""
    x = torch.tensor([[[2.0]], [[3.0]], [[5.0]]], dtype=torch.float64)
    one = torch.ones(3, 1, 1, dtype=torch.float64)
    dt = torch.tensor([[1.0], [0.5], [2.0]], dtype=torch.float64)
    a, D = torch.tensor([math.log(0.3)], dtype=torch.float64), torch.tensor([10.0], dtype=torch.float64)
    fin = []
    y = O.state_space(x, one, 2.0 * one, dt, a, D, state=fin)
    s0 = 2.0
    s1 = math.exp(-0.15) * s0 + 0.5 * 3.0
    s2 = math.exp(-0.6) * s1 + 2.0 * 5.0
    assert [round(float(v), 12) for v in y.flatten()] == [round(v, 12) for v in (2 * s0 + 20.0, 2 * s1 + 30.0, 2 * s2 + 50.0)] and abs(float(fin[0]) - s2) < 1e-12


def test_oracle_convolution_norms_and_gate_order():
    x = torch.arange(1.0, 5.0, dtype=torch.float64)[:, None]
    w, b = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64), torch.tensor([0.25], dtype=torch.float64)     # the last column is the current token's
    assert float((O.causal_conv(x, w, b) - O.silu(torch.tensor([[1.25], [12.25], [123.25], [234.25]], dtype=torch.float64))).abs().max()) < 1e-12
    y = O.centred_norm(torch.tensor([[3.0, 4.0]], dtype=torch.float64), torch.tensor([0.0, 1.0]), 0.0)
    assert float((y - torch.tensor([[3.0, 8.0]], dtype=torch.float64) / math.sqrt(12.5)).abs().max()) < 1e-12
    # the gate comes before the norm: scaling every gate's output of a group changes nothing
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    y, z, w = r(2, 6), r(2, 6), r(6)
    u = y * O.silu(z)
    want = torch.cat([u[:, :3] / u[:, :3].pow(2).mean(1, keepdim=True).sqrt(), u[:, 3:] / u[:, 3:].pow(2).mean(1, keepdim=True).sqrt()], 1) * w
    assert float((O.gate_then_group_norm(y, z, w, 2, 0.0) - want).abs().max()) < 1e-12
    assert float((O.softplus(torch.tensor([-800.0, 0.0, 800.0], dtype=torch.float64)) - torch.tensor([0.0, math.log(2.0), 800.0], dtype=torch.float64)).abs().max()) < 1e-12


def test_oracle_router_and_identity_experts():
    z = torch.tensor([[2.0, 1.0, 0.0, -1.0]], dtype=torch.float64)
    s = torch.softmax(z, -1)[0]
    idx, w = O.route(z, torch.tensor([0.0, 0.0, 0.0, 5.0], dtype=torch.float64), 2)
    assert idx[0].tolist() == [3, 0] and torch.equal(w[0], s[[3, 0]])       # chosen by the corrected score, weighted by the plain one
    h = torch.tensor([[1.0, -2.0]], dtype=torch.float64)
    W = {"router": torch.zeros(3, 2, dtype=torch.float64), "correction": torch.tensor([0.0, 1.0, 0.5], dtype=torch.float64)}
    for n in ("gate", "up", "down"):
        W[f"e0.{n}"] = torch.eye(2, dtype=torch.float64)
    out = O.mixture(h, W, {"router": {"experts": 1, "identity": 2, "top": 2}})
    assert float((out - h * (2.0 / 3.0)).abs().max()) < 1e-12               # both identity experts, a third of the weight each
    out = O.mixture(h, W, {"router": {"experts": 1, "identity": 2, "top": 3}})
    assert float((out - h * (2.0 / 3.0) - O.silu(h) * h / 3.0).abs().max()) < 1e-12
