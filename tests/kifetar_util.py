"""Shared pieces of the Kifetar tests: small configurations (none of them a shipped model's sizes), float64 copies of seeded weights for
the oracle, a model builder (tests/hybrid_util.py has the engine and feeding helpers)."""
from __future__ import annotations

from typing import Dict, Optional

import torch

# original length below the test sequences and a base that spreads the wavelengths: every branch of the frequency rule comes up
LENGTHEN = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 40}


def attention(heads=4, kv_heads=2, dim=12, window: Optional[int] = 7, scale=0.35, base=300.0, rot_dims: Optional[int] = 8, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if rot_dims is not None:
        m["rot"] = {"base": base, "dims": rot_dims}
        if scaling:
            m["rot"]["scaling"] = dict(scaling)
    if window is not None:
        m["mask"] = {"size": window}
    return m


def delta(heads=4, kv_heads=2, dim=10, vdim=14, conv=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def dense(ff=44):
    return {"kind": "dense", "ff": ff}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, width=40, vocab=97, eps=1e-5, loop=None) -> dict:
    d = {"architecture": "Kifetar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        d["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return d


def small_config() -> dict:
    """Odd sizes throughout, both mixers on both sides of and inside the loop, a layer without feed-forward, scaled and plain
    frequencies, an attention layer without a window."""
    return config([
        layer("attention", attention(scaling=LENGTHEN), dense()),
        layer("delta", delta(), dense(ff=36)),
        layer("attention", attention(heads=3, kv_heads=3, dim=6, window=None, rot_dims=6, base=50.0), None),
        layer("delta", delta(heads=6, kv_heads=2, dim=7, vdim=9, conv=4), dense(ff=20)),
        layer("attention", attention(heads=2, kv_heads=1, dim=10, window=16, rot_dims=4), dense()),
    ], loop=(1, 4, 3))


def aligned_config(width=128) -> dict:
    """Sizes the tensor-core products take (multiples of 8 and 32), for the bfloat16 path; the loop opens with the first layer."""
    return config([
        layer("attention", attention(heads=8, kv_heads=2, dim=32, window=24, scale=0.18, base=1000.0, rot_dims=16, scaling=LENGTHEN), dense(ff=192)),
        layer("delta", delta(heads=4, kv_heads=2, dim=32, vdim=48, conv=4), dense(ff=160)),
        layer("delta", delta(heads=2, kv_heads=2, dim=40, vdim=32, conv=2), dense(ff=128)),
    ], width=width, vocab=203, loop=(0, 2, 2))


def many_heads_config() -> dict:
    """8 and 16 query heads over one key / value head: single tokens take the heads-as-rows attention with the keys split over CTAs."""
    return config([
        layer("attention", attention(heads=8, kv_heads=1, dim=8, window=70, rot_dims=4), dense(ff=48)),
        layer("delta", delta(heads=8, kv_heads=1, dim=8, vdim=12), dense(ff=48)),
        layer("attention", attention(heads=16, kv_heads=2, dim=8, window=None, rot_dims=8), None),
    ], width=48, vocab=101)


def f64(weights: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    return {k: v.double() for k, v in weights.items()}


def build(cfg_dict: dict, dtype=torch.float32, seed=0, weights=None, **kw):
    """(model on the GPU, float64 weights)."""
    from vyomai_b200 import KifetarConfig, KifetarForCausalLM
    cfg = KifetarConfig(cfg_dict)
    w = weights if weights is not None else KifetarForCausalLM.random_weights(cfg, seed=seed)
    return KifetarForCausalLM(cfg, w, dtype=dtype, device="cuda", **kw), f64(w)


def random_config(seed: int) -> dict:
    """A configuration drawn from the design's whole space: 2-5 layers of the two mixers in any order, with and without a loop (also of one
    layer, of all layers, one pass), head counts from 1 to 16, unrelated channel counts, windows from 1 to longer than the sequence,
    1 to 6 taps."""
    g = torch.Generator().manual_seed(seed)
    pick = lambda xs: xs[int(torch.randint(0, len(xs), (1,), generator=g))]  # noqa: E731
    n = pick([2, 3, 4, 5])
    layers = []
    for i in range(n):
        kvh = pick([1, 2, 3])
        if pick([True, False]):
            d = pick([4, 8, 16, 24, 40])
            sc = pick([None, {"factor": pick([2.0, 8.0]), "low": pick([0.5, 1.0]), "high": pick([2.0, 4.0]), "original": pick([16, 64, 1000])}])
            m = attention(heads=kvh * pick([1, 2, 4, 8]), kv_heads=kvh, dim=d, window=pick([1, 3, 17, 50, 200, None]), scale=pick([0.1, 0.25, 0.5]),
                          base=pick([10.0, 1000.0, 250000.0]), rot_dims=pick([None, 2, d // 2 // 2 * 2, d]), scaling=sc)
            layers.append(layer("attention", m, pick([None, dense(ff=pick([24, 64, 100]))])))
        else:
            m = delta(heads=kvh * pick([1, 2, 3]), kv_heads=kvh, dim=pick([4, 8, 16, 33, 72]), vdim=pick([4, 10, 24, 40]), conv=pick([1, 2, 4, 6]))
            layers.append(layer("delta", m, pick([None, dense(ff=pick([24, 64, 100]))])))
    loop = None
    if pick([True, True, False]):
        a = int(torch.randint(0, n, (1,), generator=g))
        b = int(torch.randint(a + 1, n + 1, (1,), generator=g))
        loop = (a, b, pick([1, 2, 3]))
    return config(layers, width=pick([48, 64, 96, 160]), vocab=pick([50, 131, 256]), eps=pick([1e-6, 1e-5]), loop=loop)
