"""Zaparax: a hybrid decoder-only language model whose layers RMS-norm a sublayer's input AND its result before adding it:
x += norm1b(mixer(norm1 x)), x += norm2b(ff(norm2 x)), all layer norms RMS norms with a weight stored around zero (1 + w). Layers are
listed in the configuration; two mixers:

  * `attention` (layers/mixers.py BiasedAttention): grouped-query softmax attention without rotation, unit-RMS queries and keys, a query
    factor that grows with the position, capped scores minus a per-head slope times the distance, sliding window, softmax sink.
  * `mamba2` (StateSpaceMixer): state-space recurrence with one decay per head and token, short convolutions, gated and group-normed
    read-out.

The feed-forward is a softmax-routed mixture of gated experts (MoEFeedForward): the choice is corrected by a bias, the weights are the
plain scores, some router outputs are identity experts, a gated shared expert runs for every token. The embedding of a token is its
scaled row plus a row of a hashed-pair table chosen by the token and the one before it, so the previous token is part of a sequence's
state. A run of layers may be looped: layers loop.start .. loop.stop - 1 run loop.times times in a row with the same weights, every pass
with pages and states of its own. The reference package has no such model; it is served by the same pieces as the other packed-step
decoders here (models/gelutar.py, models/zugunex.py, models/vazepel.py, models/fubinex.py, models/kifetar.py): a configuration object read
from config.json, weights loaded by tensor name, the cache manager's pages and state slots (vyomai_b200/paged.py), one `step` over a packed
batch that the batching engine, the CUDA-graph capture and the trace replayer all call, and greedy selection by vy_argmax_rows.

The residual stream, norms, attention scores and weights, router scores, decays, step sizes and recurrent state are fp32 in both dtypes;
with dtype=bfloat16 the projections read bf16 inputs on the tensor cores (fp32 results), with dtype=float32 they are fp32 FMA.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List, Optional, Tuple

import torch

from .. import _lib, ops
from ..layers.mixers import BiasedAttention, MoEFeedForward, Projection, StateSpaceMixer, pack_biases, pack_rows

MIXER_TYPES = ("attention", "mamba2")


class ZaparaxConfig:
    """config.json of the architecture: vocab, width, norm.eps, embedding ({scale, bigram?: {buckets, mul_prev, mul_cur}}), `loop`
    ({start, stop, times} or absent) and `layers`, a list of {"type": "attention", "mixer": {heads, kv_heads, dim, vdim, scale, softcap?,
    mask?: {size}, q_temp?: {coef, every}}} | {"type": "mamba2", "mixer": {heads, vdim, state, groups, conv, norm_groups}}, each with
    "mlp": null | {"kind": "moe", "expert": {ff}, "router": {experts, top, identity?}, "shared"?: {ff}}."""

    architecture = "Zaparax"

    def __init__(self, d: dict):
        if d.get("architecture") != self.architecture:
            raise ValueError(f"not a {self.architecture} configuration: {d.get('architecture')!r}")
        self.raw = d
        self.vocab, self.width = int(d["vocab"]), int(d["width"])
        self.eps = float(d["norm"]["eps"])
        e = d.get("embedding") or {}
        self.embedding_scale = float(e.get("scale", 1.0))
        b = e.get("bigram")
        self.bigram: Optional[Tuple[int, int, int]] = (int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None
        if self.bigram and self.bigram[0] < 1:
            raise ValueError("embedding.bigram: at least one bucket")
        self.layers = list(d["layers"])
        for i, L in enumerate(self.layers):
            if L["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
            m = L["mixer"]
            if L["type"] == "attention":
                if int(m["heads"]) % int(m["kv_heads"]):
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if m.get("q_temp") and int(m["q_temp"]["every"]) < 1:
                    raise ValueError(f"layer {i}: q_temp.every is at least 1")
            else:
                if int(m["heads"]) % int(m["groups"]):
                    raise ValueError(f"layer {i}: heads must be a multiple of groups")
                if int(m["heads"]) * int(m["vdim"]) % int(m["norm_groups"]):
                    raise ValueError(f"layer {i}: norm_groups must divide heads * vdim")
                if not 1 <= int(m["conv"]) <= 16:
                    raise ValueError(f"layer {i}: the convolution has 1 to 16 taps")
            f = L.get("mlp")
            if f:
                if f.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
                r = f["router"]
                if not 1 <= int(r["top"]) <= int(r["experts"]) + int(r.get("identity", 0)) or int(r["experts"]) < 1:
                    raise ValueError(f"layer {i}: router.top {r['top']} of {r['experts']} + {r.get('identity', 0)} experts")
        lp = d.get("loop")
        self.loop: Optional[Tuple[int, int, int]] = None
        if lp:
            self.loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"]))
            if not 0 <= self.loop[0] < self.loop[1] <= len(self.layers) or self.loop[2] < 1:
                raise ValueError(f"loop {lp}: layers start .. stop - 1 of {len(self.layers)} run at least once")

    @classmethod
    def from_dir(cls, path: str) -> "ZaparaxConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls(json.load(f))

    def runs(self) -> List[int]:
        """The layers in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Name -> shape of every weight the configuration implies (what a checkpoint must hold; also the recipe for random
        initialisation)."""
        W = self.width
        out: Dict[str, tuple] = {"embed": (self.vocab, W), "final.norm": (W,), "head": (self.vocab, W)}
        if self.bigram:
            out["bigram"] = (self.bigram[0] + 1, W)
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L["mixer"]
            for nm in ["norm1", "norm1b"] + (["norm2", "norm2b"] if L.get("mlp") else []):
                out[p + nm] = (W,)
            q = p + "mix."
            if L["type"] == "attention":
                H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
                out.update({q + "q": (H * dk, W), q + "q.b": (H * dk,), q + "k": (G * dk, W), q + "k.b": (G * dk,), q + "v": (G * dv, W), q + "v.b": (G * dv,),
                            q + "sink": (H,), q + "o": (W, H * dv)})
            else:
                H, dv, gn = m["heads"], m["vdim"], m["groups"] * m["state"]
                inner = H * dv
                out.update({q + "in": (2 * inner + 2 * gn + H, W), q + "conv": (inner + 2 * gn, m["conv"]), q + "conv.b": (inner + 2 * gn,), q + "dt_bias": (H,),
                            q + "A_log": (H,), q + "D": (H,), q + "norm": (inner,), q + "o": (W, inner)})
            f = L.get("mlp")
            if not f:
                continue
            r, q = f["router"], p + "mlp."
            gated = lambda pre, ff: {pre + "gate": (ff, W), pre + "up": (ff, W), pre + "down": (W, ff)}  # noqa: E731
            for e in range(r["experts"]):
                out.update(gated(q + f"e{e}.", f["expert"]["ff"]))
            n = r["experts"] + r.get("identity", 0)
            out.update({q + "router": (n, W), q + "correction": (n,)})
            if f.get("shared"):
                out.update(gated(q + "shared.", f["shared"]["ff"]))
                out[q + "shared.sg"] = (1, W)
        return out


class _Layer:
    """A layer's weights. `forward` takes the layer's normed input and returns the NEXT norm's output: closing a sublayer (its result
    normed and added to the residual) and the norm that follows are one launch, also across layers."""

    def __init__(self, idx: int, spec: dict, w: Dict[str, torch.Tensor], cfg: ZaparaxConfig, act_dtype, tensor_cores: bool, kv_dtype,
                 sorted_min_rows: int, force_sorted: bool):
        p = f"l{idx}."
        sub = lambda pre: {k[len(pre):]: v for k, v in w.items() if k.startswith(pre)}  # noqa: E731
        self.act_dtype = act_dtype
        self.close = dict(eps=cfg.eps, kind="rms_centred", out_dtype=act_dtype)
        self.norm1, self.norm1b = w[p + "norm1"].contiguous(), w[p + "norm1b"].contiguous()
        if spec["type"] == "attention":
            self.mixer = BiasedAttention(spec["mixer"], sub(p + "mix."), cfg.eps, act_dtype, tensor_cores, kv_dtype)
        else:
            self.mixer = StateSpaceMixer(spec["mixer"], sub(p + "mix."), cfg.eps, act_dtype, tensor_cores)
        packed, self.spans = pack_rows(self.mixer.input_weights())
        self.inp = Projection(packed, tensor_cores)   # every matrix that reads norm1(x), as one product
        self.inp_bias = pack_biases(self.spans, packed.shape[0], self.mixer.input_biases(), packed)
        self.mlp = None
        f = spec.get("mlp")
        if f:
            self.norm2, self.norm2b = w[p + "norm2"].contiguous(), w[p + "norm2b"].contiguous()
            r = f["router"]
            self.mlp = MoEFeedForward(sub(p + "mlp."), r["experts"], r["top"], 1.0, act_dtype, tensor_cores, shared=bool(f.get("shared")),
                                      sorted_min_rows=sorted_min_rows, force_sorted=force_sorted, router="softmax", normalize=False, form="swiglu",
                                      identity=int(r.get("identity", 0)))

    def forward(self, x: torch.Tensor, h: torch.Tensor, batch: ops.PackedBatch, cache, next_norm) -> Optional[torch.Tensor]:
        """x: the fp32 residual, updated in place; h = norm1(x). Returns next_norm(x) (None without one)."""
        P = self.inp(h, bias=self.inp_bias)
        y = self.mixer.forward([P[:, o:o + n] for o, n in self.spans], batch, cache)
        if self.mlp is None:
            return ops.sandwich_norm(x, y, self.norm1b, next_norm, x_out=x, **self.close)
        h2 = ops.sandwich_norm(x, y, self.norm1b, self.norm2, x_out=x, **self.close)
        y, ident = self.mlp.forward_parts(h2, batch)
        return ops.sandwich_norm(x, y, self.norm2b, next_norm, x_out=x, second=None if ident is None else (h2, ident), **self.close)


class ZaparaxForCausalLM:
    """The model: `step(ids, batch, caches, want_rows)` runs the step's packed tokens through every layer run, updating the
    sequences' pages and state slots in `caches` (one entry for the embedding, then one per layer RUN: a looped layer has one per
    pass), and returns fp32 logits [len(want_rows), vocab] of the requested rows."""

    config_class = ZaparaxConfig

    def __init__(self, config: ZaparaxConfig, weights: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16,
                 device: Optional[torch.device] = None, tensor_cores: bool = True, kv_dtype: torch.dtype = torch.float32,
                 sorted_min_rows: int = 128, force_sorted: bool = False):
        if dtype not in (torch.bfloat16, torch.float32):
            raise _lib.VyomError("ZaparaxForCausalLM runs in bfloat16 or float32")
        self.config, self.dtype = config, dtype
        self.device = torch.device(device or "cuda")
        need = config.tensor_shapes()
        missing = [k for k in need if k not in weights]
        if missing:
            raise KeyError(f"checkpoint lacks {missing[:5]}{' ...' if len(missing) > 5 else ''}")
        for k, shp in need.items():
            got = tuple(weights[k].shape)
            if got != tuple(shp):
                raise ValueError(f"{k}: shape {got}, the configuration implies {tuple(shp)}")
        w = {k: v.to(device=self.device, dtype=dtype) for k, v in weights.items() if k in need}
        self.embed = w["embed"].contiguous()
        self.pairs = w["bigram"].contiguous() if config.bigram else None
        self.head = Projection(w["head"], tensor_cores)
        self.final_norm = w["final.norm"].contiguous()
        self.layers = [_Layer(i, L, w, config, dtype, tensor_cores, kv_dtype, sorted_min_rows, force_sorted) for i, L in enumerate(config.layers)]
        self.runs = config.runs()
        self.debug_residuals: Optional[list] = None   # set to [] to collect the residual stream after every layer run

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device=None, **kw) -> "ZaparaxForCausalLM":
        from ..checkpoint import load_safetensors
        return cls(ZaparaxConfig.from_dir(path), load_safetensors(os.path.join(path, "model.safetensors")), dtype=dtype, device=device, **kw)

    @staticmethod
    def random_weights(config: ZaparaxConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
        """Seeded bf16 weights of the right shapes (tests, benchmarks): projections ~ N(0, 1/in), embeddings ~ N(0, 1), norm weights around
        what leaves a row as it is, sinks ~ N(0, 1), decays between ~0.5 and ~1, routers wide enough that softmax scores stay apart and
        corrections large enough to change some choices."""
        g = torch.Generator().manual_seed(seed)
        out = {}
        for k, shp in config.tensor_shapes().items():
            leaf = k.split(".")[-1]
            if leaf in ("embed", "bigram", "sink"):
                t = torch.randn(shp, generator=g)
            elif leaf == "conv":
                t = torch.randn(shp, generator=g) * 0.5
            elif leaf == "A_log":
                t = torch.rand(shp, generator=g) * 2.0 - 1.0
            elif leaf == "dt_bias":
                t = torch.rand(shp, generator=g) * 2.0 - 2.0
            elif leaf == "D":
                t = 0.5 + 0.5 * torch.randn(shp, generator=g)
            elif leaf == "router":
                t = torch.randn(shp, generator=g) * 2.0 / (shp[1] ** 0.5)
            elif leaf == "correction":
                t = 0.2 * torch.randn(shp, generator=g)
            elif len(shp) == 2:
                t = torch.randn(shp, generator=g) / (shp[1] ** 0.5)
            elif leaf == "norm" and ".mix." in k:
                t = 1.0 + 0.1 * torch.randn(shp, generator=g)
            else:   # layer norm weights (stored around zero) and biases
                t = 0.1 * torch.randn(shp, generator=g)
            out[k] = t.to(torch.bfloat16)
        return out

    def cache_specs(self):
        embedding = {"pages": None, "states": {"prev": (1,)} if self.pairs is not None else {}, "state_dtypes": {"prev": torch.int32}}
        return [[embedding]] + [[self.layers[i].mixer.cache_spec()] for i in self.runs]

    @torch.no_grad()
    def step(self, ids: torch.Tensor, batch: ops.PackedBatch, caches, want_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        cfg = self.config
        if self.pairs is None:
            x = ops.embed_rows(ids, self.embed, cfg.embedding_scale, torch.float32)
        else:
            _, mul_prev, mul_cur = cfg.bigram
            x = ops.pair_embed(batch, ids, self.embed, cfg.embedding_scale, self.pairs, caches[0][0].states["prev"], mul_prev=mul_prev, mul_cur=mul_cur)
        norms = [self.layers[i].norm1 for i in self.runs] + [None]
        close = dict(eps=cfg.eps, kind="rms_centred", out_dtype=self.dtype)
        h = ops.sandwich_norm(x, norm2=norms[0], **close) if self.runs else None
        for n, i in enumerate(self.runs):
            h = self.layers[i].forward(x, h, batch, caches[n + 1][0], norms[n + 1])
            if self.debug_residuals is not None:
                self.debug_residuals.append(x.clone())
        if want_rows is None or want_rows.numel() == 0:
            return None
        return self.head(ops.sandwich_norm(x, norm2=self.final_norm, row_index=want_rows, **close))
