"""Kifetar: a hybrid decoder-only language model whose layers norm a sublayer's input AND its result before adding it:
x += norm1b(mixer(norm1 x)), x += norm2b(ff(norm2 x)), all layer norms with weight and bias. Layers are listed in the configuration; two
mixers:

  * `attention` (layers/mixers.py SigmoidAttention): grouped-query attention over a sliding window whose key weights are sigmoids, not
    a softmax; the values are the keys as projected; RMS-normed, partly rotated queries and keys; per-head temperature, score bias and
    output gate.
  * `delta` (HeadDecayDeltaMixer): the gated delta rule with one decay per head, short convolutions, normed and gated read-out.

The feed-forward is W_down (silu(W_gate h) * (W_up h)). A run of layers may be looped: layers loop.start .. loop.stop - 1 run loop.times
times in a row with the same weights, and before each pass the stream is re-made from itself and the embedding output,
x <- W_in [x; x0]. Every pass owns its pages and states. The output head is the embedding table. The reference package has no such
model; it is served by the same pieces as the other packed-step decoders here (models/gelutar.py, models/zugunex.py, models/vazepel.py,
models/fubinex.py): a configuration object read from config.json, weights loaded by tensor name, the cache manager's pages and state
slots (vyomai_b200/paged.py), one `step` over a packed batch that the batching engine, the CUDA-graph capture and the trace replayer
all call, and greedy selection by vy_argmax_rows.

The residual stream, norms, rotation angles, attention scores and weights, decays and recurrent state are fp32 in both dtypes; with
dtype=bfloat16 the projections read bf16 inputs on the tensor cores (fp32 results), with dtype=float32 they are fp32 FMA.
"""
from __future__ import annotations

import json
import os
from typing import Dict, List, Optional, Tuple

import torch

from .. import _lib, ops
from ..layers.mixers import GatedMLP, HeadDecayDeltaMixer, Projection, SigmoidAttention, pack_biases, pack_rows

MIXER_TYPES = ("attention", "delta")


class KifetarConfig:
    """config.json of the architecture: vocab, width, norm.eps, `loop` ({start, stop, times} or absent) and `layers`, a list of
    {"type": "attention", "mixer": {heads, kv_heads, dim, vdim (= dim), scale, rot?: {base, dims, scaling?: {factor, low, high, original}},
    mask?: {size}}} | {"type": "delta", "mixer": {heads, kv_heads, dim, vdim, conv}}, each with "mlp": null | {"kind": "dense", "ff"}."""

    architecture = "Kifetar"

    def __init__(self, d: dict):
        if d.get("architecture") != self.architecture:
            raise ValueError(f"not a {self.architecture} configuration: {d.get('architecture')!r}")
        self.raw = d
        self.vocab, self.width = int(d["vocab"]), int(d["width"])
        self.eps = float(d["norm"]["eps"])
        self.layers = list(d["layers"])
        for i, L in enumerate(self.layers):
            if L["type"] not in MIXER_TYPES:
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
            m = L["mixer"]
            if int(m["heads"]) % int(m["kv_heads"]):
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if L["type"] == "attention":
                if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                    raise ValueError(f"layer {i}: the values are the keys, so vdim equals dim")
                rd = int((m.get("rot") or {}).get("dims", 0))
                if rd % 2 or rd > int(m["dim"]):
                    raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
            elif not 1 <= int(m["conv"]) <= 16:
                raise ValueError(f"layer {i}: the convolution has 1 to 16 taps")
            f = L.get("mlp")
            if f and f.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
        lp = d.get("loop")
        self.loop: Optional[Tuple[int, int, int]] = None
        if lp:
            self.loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"]))
            if not 0 <= self.loop[0] < self.loop[1] <= len(self.layers) or self.loop[2] < 1:
                raise ValueError(f"loop {lp}: layers start .. stop - 1 of {len(self.layers)} run at least once")

    @classmethod
    def from_dir(cls, path: str) -> "KifetarConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls(json.load(f))

    def runs(self) -> List[Tuple[int, bool]]:
        """The layers in the order they run: (layer, does a loop pass begin with it?)."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        a, b, times = self.loop
        return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(times) for i in range(a, b)] + [(i, False) for i in range(b, n)]

    def tensor_shapes(self) -> Dict[str, tuple]:
        """Name -> shape of every weight the configuration implies (what a checkpoint must hold; also the recipe for random
        initialisation)."""
        W = self.width
        out: Dict[str, tuple] = {"embed": (self.vocab, W), "final.norm": (W,), "final.norm.b": (W,)}
        if self.loop is not None:
            out["loop.in"] = (W, 2 * W)
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L["mixer"]
            norms = ["norm1", "norm1b"] + (["norm2", "norm2b"] if L.get("mlp") else [])
            for nm in norms:
                out.update({p + nm: (W,), p + nm + ".b": (W,)})
            H, G, dk = m["heads"], m["kv_heads"], m["dim"]
            q = p + "mix."
            if L["type"] == "attention":
                out.update({q + "q": (H * dk, W), q + "q.b": (H * dk,), q + "k": (G * dk, W), q + "k.b": (G * dk,), q + "q.norm": (dk,), q + "k.norm": (dk,),
                            q + "temp": (H,), q + "pb": (H,), q + "g": (H, W), q + "o": (W, H * dk)})
            else:
                dv, taps = m["vdim"], m["conv"]
                out.update({q + "q": (G * dk, W), q + "q.conv": (G * dk, taps), q + "k": (G * dk, W), q + "k.conv": (G * dk, taps), q + "v": (H * dv, W),
                            q + "v.conv": (H * dv, taps), q + "a": (H, W), q + "dt_bias": (H,), q + "A_log": (H,), q + "b": (H, W), q + "g": (H * dv, W),
                            q + "norm": (dv,), q + "o": (W, H * dv)})
            f = L.get("mlp")
            if f:
                out.update({p + "mlp.gate": (f["ff"], W), p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
        return out


class _Layer:
    """A layer's weights. `forward` takes the layer's normed input and returns the NEXT norm's output: closing a sublayer (its result
    normed and added to the residual) and the norm that follows are one launch, also across layers."""

    def __init__(self, idx: int, spec: dict, w: Dict[str, torch.Tensor], cfg: KifetarConfig, act_dtype, tensor_cores: bool, kv_dtype):
        p = f"l{idx}."
        sub = lambda pre: {k[len(pre):]: v for k, v in w.items() if k.startswith(pre)}  # noqa: E731
        norm = lambda name: (w[p + name].contiguous(), w[p + name + ".b"].contiguous())  # noqa: E731
        self.eps, self.act_dtype = cfg.eps, act_dtype
        self.norm1, self.norm1b = norm("norm1"), norm("norm1b")
        if spec["type"] == "attention":
            self.mixer = SigmoidAttention(spec["mixer"], sub(p + "mix."), cfg.eps, act_dtype, tensor_cores, kv_dtype)
        else:
            self.mixer = HeadDecayDeltaMixer(spec["mixer"], sub(p + "mix."), cfg.eps, act_dtype, tensor_cores)
        packed, self.spans = pack_rows(self.mixer.input_weights())
        self.inp = Projection(packed, tensor_cores)   # every matrix that reads norm1(x), as one product
        self.inp_bias = pack_biases(self.spans, packed.shape[0], self.mixer.input_biases(), packed)
        self.mlp = None
        if spec.get("mlp"):
            self.norm2, self.norm2b = norm("norm2"), norm("norm2b")
            self.mlp = GatedMLP(sub(p + "mlp."), act_dtype, tensor_cores)

    def forward(self, x: torch.Tensor, h: torch.Tensor, batch: ops.PackedBatch, cache, next_norm, copy_out: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """x: the fp32 residual, updated in place; h = norm1(x). Returns next_norm(x) (None without one); copy_out also receives x."""
        P = self.inp(h, bias=self.inp_bias)
        y = self.mixer.forward([P[:, o:o + n] for o, n in self.spans], batch, cache)
        last = dict(norm2=next_norm, copy_out=copy_out)
        if self.mlp is None:
            return ops.sandwich_norm(x, y, self.norm1b, eps=self.eps, x_out=x, out_dtype=self.act_dtype, **last)
        h2 = ops.sandwich_norm(x, y, self.norm1b, self.norm2, eps=self.eps, x_out=x, out_dtype=self.act_dtype)
        return ops.sandwich_norm(x, self.mlp.forward(h2), self.norm2b, eps=self.eps, x_out=x, out_dtype=self.act_dtype, **last)


class KifetarForCausalLM:
    """The model: `step(ids, batch, caches, want_rows)` runs the step's packed tokens through every layer run, updating the
    sequences' pages and state slots in `caches` (one entry per layer RUN: a looped layer has one per pass), and returns fp32 logits
    [len(want_rows), vocab] of the requested rows."""

    config_class = KifetarConfig

    def __init__(self, config: KifetarConfig, weights: Dict[str, torch.Tensor], dtype: torch.dtype = torch.bfloat16,
                 device: Optional[torch.device] = None, tensor_cores: bool = True, kv_dtype: torch.dtype = torch.float32):
        if dtype not in (torch.bfloat16, torch.float32):
            raise _lib.VyomError("KifetarForCausalLM runs in bfloat16 or float32")
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
        self.head = Projection(self.embed, tensor_cores)   # tied
        self.final_norm = (w["final.norm"].contiguous(), w["final.norm.b"].contiguous())
        self.loop_in = Projection(w["loop.in"], tensor_cores) if config.loop is not None else None
        self.layers = [_Layer(i, L, w, config, dtype, tensor_cores, kv_dtype) for i, L in enumerate(config.layers)]
        self.runs = config.runs()
        self.debug_residuals: Optional[list] = None   # set to [] to collect the residual stream after every layer run

    @classmethod
    def from_pretrained(cls, path: str, dtype: torch.dtype = torch.bfloat16, device=None, **kw) -> "KifetarForCausalLM":
        from ..checkpoint import load_safetensors
        return cls(KifetarConfig.from_dir(path), load_safetensors(os.path.join(path, "model.safetensors")), dtype=dtype, device=device, **kw)

    @staticmethod
    def random_weights(config: KifetarConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
        """Seeded bf16 weights of the right shapes (tests, benchmarks): projections ~ N(0, 1/in), embeddings ~ N(0, 1), norm weights
        around 1, temperatures of order 2, score biases around -2 (a few keys per window stand out), decays between ~0.5 and ~1."""
        g = torch.Generator().manual_seed(seed)
        out = {}
        for k, shp in config.tensor_shapes().items():
            leaf = k.split(".")[-1]
            if leaf == "embed":
                t = torch.randn(shp, generator=g)
            elif leaf == "conv":
                t = torch.randn(shp, generator=g) * 0.5
            elif leaf == "A_log":
                t = torch.rand(shp, generator=g) * 2.0 - 2.0
            elif leaf == "dt_bias":
                t = torch.rand(shp, generator=g) * 2.0 - 3.0
            elif leaf == "temp":
                t = 2.0 + 0.5 * torch.randn(shp, generator=g)
            elif leaf == "pb":
                t = torch.randn(shp, generator=g) * 0.5 - 2.0
            elif len(shp) == 2:
                t = torch.randn(shp, generator=g) / (shp[1] ** 0.5)
            elif leaf == "b":   # norm and projection biases
                t = 0.1 * torch.randn(shp, generator=g)
            else:               # norm weights
                t = 1.0 + 0.1 * torch.randn(shp, generator=g)
            out[k] = t.to(torch.bfloat16)
        return out

    def cache_specs(self):
        return [[self.layers[i].mixer.cache_spec()] for i, _ in self.runs]

    @torch.no_grad()
    def step(self, ids: torch.Tensor, batch: ops.PackedBatch, caches, want_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        eps, W = self.config.eps, self.config.width
        x = ops.embed_rows(ids, self.embed, 1.0, torch.float32)
        both = None
        if self.loop_in is not None:   # [x; x0] in the products' dtype: x0 stays in the right half, x is written beside it by the layer before a pass
            both = torch.empty((x.shape[0], 2 * W), device=x.device, dtype=self.dtype)
            ops.embed_rows(ids, self.embed, 1.0, self.dtype, out=both[:, W:])
        h = None
        for n, ((i, opens), c) in enumerate(zip(self.runs, caches)):
            L = self.layers[i]
            if opens:
                if n == 0:
                    ops.embed_rows(ids, self.embed, 1.0, self.dtype, out=both[:, :W])
                self.loop_in(both, out=x)
            if h is None:
                h = ops.sandwich_norm(x, norm2=L.norm1, eps=eps, out_dtype=self.dtype)
            nxt = self.runs[n + 1] if n + 1 < len(self.runs) else None
            to_pass = nxt is not None and nxt[1]   # a loop pass follows: it needs x itself, not a norm of it
            h = L.forward(x, h, batch, c[0], None if nxt is None or to_pass else self.layers[nxt[0]].norm1, both[:, :W] if to_pass else None)
            if self.debug_residuals is not None:
                self.debug_residuals.append(x.clone())
        if want_rows is None or want_rows.numel() == 0:
            return None
        hn = ops.sandwich_norm(x, norm2=self.final_norm, eps=eps, row_index=want_rows, out_dtype=self.dtype)
        return self.head(hn)
