"""Shared pieces of the Zaparax tests: small configurations (none of them a shipped model's sizes), float64 copies of seeded weights for
the oracle, a model builder (tests/hybrid_util.py has the engine and feeding helpers)."""
from __future__ import annotations

from typing import Dict, Optional

import torch


def attention(heads=4, kv_heads=2, dim=12, vdim=10, window: Optional[int] = 7, scale=0.5, softcap: Optional[float] = 4.0, q_temp=(0.4, 5)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if window is not None:
        m["mask"] = {"size": window}
    if q_temp is not None:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return m


def mamba(heads=4, vdim=10, state=9, groups=2, conv=3, norm_groups=2):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def moe(ff=20, experts=5, top=3, identity: Optional[int] = 2, shared: Optional[int] = 28):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    f = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, width=40, vocab=97, eps=1e-5, loop=None, bigram=(53, 7, 3), scale=1.5) -> dict:
    d = {"architecture": "Zaparax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if bigram is not None:
        d["embedding"]["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    if loop is not None:
        d["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return d


def small_config() -> dict:
    """Odd sizes throughout, both mixers on both sides of and inside the loop, layers without feed-forward, without a shared expert, without
    identity experts, an attention layer without window, cap and query temperature."""
    return config([
        layer("attention", attention(), moe()),
        layer("mamba2", mamba(), moe(ff=12, experts=6, top=2, identity=1)),
        layer("attention", attention(heads=3, kv_heads=3, dim=6, vdim=14, window=None, softcap=None, q_temp=None), None),
        layer("mamba2", mamba(heads=6, vdim=7, state=5, groups=3, conv=4, norm_groups=1), moe(ff=9, experts=4, top=4, identity=None, shared=None)),
        layer("attention", attention(heads=2, kv_heads=1, dim=10, vdim=10, window=16, softcap=1.5, q_temp=(0.2, 3)), moe(experts=3, top=5, identity=4)),
    ], loop=(1, 4, 3))


def aligned_config(width=128) -> dict:
    """Sizes the tensor-core products take (multiples of 8 and 32), for the bfloat16 path; the loop opens with the first layer."""
    return config([
        layer("attention", attention(heads=8, kv_heads=2, dim=32, vdim=32, window=24, scale=0.2, softcap=8.0, q_temp=(0.3, 16)), moe(ff=64, experts=6, top=2, identity=2, shared=96)),
        layer("mamba2", mamba(heads=4, vdim=32, state=16, groups=2, conv=4, norm_groups=2), moe(ff=48, experts=4, top=2, identity=1, shared=64)),
        layer("mamba2", mamba(heads=2, vdim=64, state=48, groups=1, conv=2, norm_groups=4), None),
    ], width=width, vocab=203, loop=(0, 2, 2), scale=1.0)


def many_heads_config() -> dict:
    """8 and 16 query heads over one key / value head: single tokens take the heads-as-rows attention with the keys split over CTAs; more
    heads than norm groups and more norm groups than a CTA has warps."""
    return config([
        layer("attention", attention(heads=8, kv_heads=1, dim=8, vdim=8, window=70), moe(ff=48)),
        layer("mamba2", mamba(heads=12, vdim=4, state=8, groups=1, conv=4, norm_groups=12), moe(ff=16)),
        layer("attention", attention(heads=16, kv_heads=1, dim=8, vdim=12, window=None), None),
        layer("mamba2", mamba(heads=5, vdim=12, state=6, groups=5, conv=2, norm_groups=3), None),
    ], width=48, vocab=101)


def f64(weights: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    return {k: v.double() for k, v in weights.items()}


def spread_corrections(weights: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    """The router corrections replaced by ones further apart than scores can be: every token chooses the same experts."""
    g = torch.Generator().manual_seed(99)
    return {k: (1.5 * torch.randperm(v.numel(), generator=g).float()).to(v.dtype) if k.endswith("mlp.correction") else v for k, v in weights.items()}


def build(cfg_dict: dict, dtype=torch.float32, seed=0, weights=None, **kw):
    """(model on the GPU, float64 weights); bfloat16 models get spread_corrections."""
    from vyomai_b200 import ZaparaxConfig, ZaparaxForCausalLM
    cfg = ZaparaxConfig(cfg_dict)
    w = weights if weights is not None else ZaparaxForCausalLM.random_weights(cfg, seed=seed)
    if weights is None and dtype == torch.bfloat16:
        w = spread_corrections(w)
    return ZaparaxForCausalLM(cfg, w, dtype=dtype, device="cuda", **kw), f64(w)


def random_config(seed: int) -> dict:
    """A configuration drawn from the design's whole space: 2-5 layers of the two mixers in any order, with and without a loop (also of one
    layer, of all layers, one pass), head counts from 1 to 16, unrelated channel counts, windows from 1 to longer than the sequence,
    1 to 6 taps, 1 to 12 experts with up to 3 identity outputs."""
    g = torch.Generator().manual_seed(seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]  # noqa: E731
    n = pick([2, 3, 4, 5])
    layers = []
    for _ in range(n):
        ex, ident = pick([1, 2, 5, 12]), pick([None, 1, 3])
        f = pick([None, moe(ff=pick([8, 24, 33]), experts=ex, top=pick([1, max(1, ex // 2), ex]), identity=ident, shared=pick([None, 16, 50]))])
        if pick([True, False]):
            kvh = pick([1, 2, 3])
            m = attention(heads=kvh * pick([1, 2, 4, 8]), kv_heads=kvh, dim=pick([4, 8, 16, 24, 40]), vdim=pick([4, 8, 20, 36]), window=pick([1, 3, 17, 50, 200, None]),
                          scale=pick([0.1, 0.5, 1.0]), softcap=pick([None, 0.7, 3.0, 50.0]), q_temp=pick([None, (0.1, 1), (0.5, 7), (1.0, 64)]))
            layers.append(layer("attention", m, f))
        else:
            gr, per, dv = pick([1, 2, 3]), pick([1, 2, 3]), pick([4, 6, 24, 40])
            m = mamba(heads=gr * per, vdim=dv, state=pick([1, 4, 8, 16, 33, 72]), groups=gr, conv=pick([1, 2, 4, 6]), norm_groups=pick([1, gr, gr * per, dv]))
            layers.append(layer("mamba2", m, f))
    loop = None
    if pick([True, True, False]):
        a = int(torch.randint(0, n, (1,), generator=g))
        b = int(torch.randint(a + 1, n + 1, (1,), generator=g))
        loop = (a, b, pick([1, 2, 3]))
    return config(layers, width=pick([37, 48, 64, 100, 160]), vocab=pick([50, 131, 256]), eps=pick([1e-6, 1e-5]), loop=loop,
                  bigram=pick([None, (1, 5, 9), (17, 31, 2), (211, 10 ** 12 + 39, 2 ** 40 + 1)]), scale=pick([1.0, 3.0, 0.5]))
