"""Plain, slow float64 statement of the Kifetar decoder's mechanisms, one function per mechanism, written from the equations and
sharing no code with vyomai_b200. Every function takes a WHOLE sequence from position 0 (time along dim 0) and loops over tokens where
the mechanism is a recurrence; the tests compare the CUDA path (whole prompts, portions, single-token decoding, mixed batches) against
these.

The mixers and `forward` take `rnd`, a function applied to the input of every product with a weight matrix (default: none): with a
rounding to bf16 there, the difference from the unrounded result says how far rounding alone moves a model's logits.

Notation: T tokens, H heads, G key / value heads, dk / dv per-head key and value sizes.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def layer_norm(x, w, b, eps):
    m = x.mean(-1, keepdim=True)
    d = x - m
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def unit(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def frequencies(rot: dict) -> List[float]:
    """Angle per position of pair i: base^(-2i / dims); with a scaling block, by wavelength against the original length: short waves
    keep their frequency, long ones are divided by the factor, the ones between are blended."""
    dims, base, out = rot["dims"], float(rot["base"]), []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave < sc["original"] / sc["high"]:
                pass
            elif wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            else:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_half(x, rot: Optional[dict]):
    """x [T, n, d], row t at position t: entry i of the first rot.dims turns with entry i + rot.dims / 2."""
    if not rot or not rot.get("dims"):
        return x
    half, freqs = rot["dims"] // 2, frequencies(rot)
    y = x.clone()
    for t in range(x.shape[0]):
        for i, f in enumerate(freqs):
            c, s = math.cos(t * f), math.sin(t * f)
            u, v = x[t, :, i], x[t, :, i + half]
            y[t, :, i] = u * c - v * s
            y[t, :, i + half] = v * c + u * s
    return y


def sigmoid_attention(q, k, v, *, scale: float, window: int, temp, bias, gate_logits):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]: weight of a visible key = sigmoid(q.k scale temp_h + bias_h), the weights
    are not normalised; query i sees j with 0 <= i - j < window (window 0: every j <= i); head outputs times sigmoid(gate_logits[t, h])."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale * temp[h] + bias[h]
        i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
        seen = (j <= i) & ((i - j < window) if window > 0 else (j <= i))
        out[:, h] = torch.where(seen, torch.sigmoid(s), torch.zeros_like(s)) @ v[:, g]
    return out * torch.sigmoid(gate_logits)[:, :, None]


def causal_conv(x, w):
    """x [T, C], w [C, taps], LAST column = the current token; zeros before the start; then silu."""
    T, C = x.shape
    taps = w.shape[1]
    y = torch.zeros(T, C, dtype=F64)
    for t in range(T):
        for d in range(taps):
            if t - d >= 0:
                y[t] += w[:, taps - 1 - d] * x[t - d]
    return silu(y)


def gated_delta_rule(q, k, v, g, beta, state=None):
    """q, k [T, G, dk] (unit vectors, q scaled), v [T, H, dv], decay g [T, H], strength beta [T, H]:
    S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, G, dk = q.shape
    H, dv = v.shape[1], v.shape[2]
    out = torch.zeros(T, H, dv, dtype=F64)
    for h in range(H):
        c = h // (H // G)
        S = torch.zeros(dk, dv, dtype=F64)
        for t in range(T):
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, c])
            S = S + torch.outer(k[t, c], u)
            out[t, h] = S.T @ q[t, c]
        if state is not None:
            state.append(S)
    return out


def exact(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(F64)


def gated_mlp(h, gate, up, down, rnd=exact):
    h = rnd(h)
    return rnd(silu(h @ gate.T) * (h @ up.T)) @ down.T


# ---- mixers and the model ----
def attention_mixer(h, W: Dict[str, torch.Tensor], m: dict, eps: float, rnd=exact):
    T, h = h.shape[0], rnd(h)
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W["q"].T + W["q.b"]).view(T, H, d)
    k = (h @ W["k"].T + W["k.b"]).view(T, G, d)
    v = k                                           # the keys as projected are the values
    q = rotate_half(rms(q, eps) * W["q.norm"], m.get("rot"))
    k = rotate_half(rms(k, eps) * W["k.norm"], m.get("rot"))
    o = sigmoid_attention(q, k, v, scale=m["scale"], window=(m.get("mask") or {}).get("size", 0), temp=W["temp"], bias=W["pb"],
                          gate_logits=h @ W["g"].T)
    return rnd(o.reshape(T, H * d)) @ W["o"].T


def delta_mixer(h, W, m, eps, rnd=exact):
    T, h = h.shape[0], rnd(h)
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = causal_conv(h @ W["q"].T, W["q.conv"]).view(T, G, dk)
    k = causal_conv(h @ W["k"].T, W["k.conv"]).view(T, G, dk)
    v = causal_conv(h @ W["v"].T, W["v.conv"]).view(T, H, dv)
    q, k = unit(q) * dk ** -0.5, unit(k)
    beta = torch.sigmoid(h @ W["b"].T)
    g = torch.exp(-torch.exp(W["A_log"]) * torch.nn.functional.softplus(h @ W["a"].T + W["dt_bias"], threshold=1e9))
    o = gated_delta_rule(q, k, v, g, beta)
    o = rms(o, eps) * W["norm"] * silu(h @ W["g"].T).view(T, H, dv)
    return rnd(o.reshape(T, H * dv)) @ W["o"].T


def _sub(W, pre):
    return {k[len(pre):]: v for k, v in W.items() if k.startswith(pre)}


def layer_runs(cfg: dict):
    """The layers in the order they run, as (layer index, first of a loop pass?)."""
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    out = [(i, False) for i in range(lp["start"])]
    for _ in range(lp["times"]):
        out += [(i, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
    return out + [(i, False) for i in range(lp["stop"], n)]


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None, rnd=exact) -> torch.Tensor:
    """Logits [T, vocab] of one sequence. W: name -> float64 tensor. residuals: receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    ln = lambda x, name: layer_norm(x, W[name], W[name + ".b"], eps)  # noqa: E731
    x0 = W["embed"][torch.tensor(tokens)]
    x = x0
    for i, opens in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if opens:
            x = rnd(torch.cat([x, x0], 1)) @ W["loop.in"].T
        mixer = attention_mixer if L["type"] == "attention" else delta_mixer
        x = x + ln(mixer(ln(x, p + "norm1"), _sub(W, p + "mix."), L["mixer"], eps, rnd), p + "norm1b")
        if L.get("mlp"):
            y = gated_mlp(ln(x, p + "norm2"), W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"], rnd)
            x = x + ln(y, p + "norm2b")
        if residuals is not None:
            residuals.append(x.clone())
    return rnd(ln(x, "final.norm")) @ W["embed"].T


def greedy(cfg, W, prompt: List[int], n_new: int):
    """Greedy continuation by re-running the whole sequence; also returns each step's top-1 / top-2 margin."""
    toks, margins = list(prompt), []
    for _ in range(n_new):
        lg = forward(cfg, W, toks)[-1]
        top = lg.topk(2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(lg.argmax()))
    return toks, margins
