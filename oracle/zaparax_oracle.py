"""Plain, slow float64 statement of the Zaparax decoder's mechanisms, one function per mechanism, written from the equations and
sharing no code with vyomai_b200. Every function takes a WHOLE sequence from position 0 (time along dim 0) and loops over tokens where
the mechanism is a recurrence; the tests compare the CUDA path (whole prompts, portions, single-token decoding, mixed batches) against
these.

The mixers, the feed-forward and `forward` take `rnd`, a function applied to the input of every product with a weight matrix (default:
none): with a rounding to bf16 there, the difference from the unrounded result says how far rounding alone moves a model's logits.

Notation: T tokens, H heads, G key / value heads (attention) or B / C groups (state space), dk / dv per-head key and value sizes,
N the state size.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def exact(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(F64)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


# ---- embedding ----
def bigram_rows(tokens: List[int], mul_prev: int, mul_cur: int, buckets: int) -> List[int]:
    """Row of the bigram table for every token: hashed pair of the previous token and this one, the extra last row for the first."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + tokens[i] * mul_cur) % buckets for i in range(len(tokens))]


def embedding(tokens: List[int], table, scale: float, bigram=None, hashing: Optional[dict] = None):
    x = table[torch.tensor(tokens)] * scale
    if hashing:
        rows = bigram_rows(tokens, int(hashing["mul_prev"]), int(hashing["mul_cur"]), int(hashing["buckets"]))
        x = x + bigram[torch.tensor(rows)]
    return x


# ---- attention ----
def query_temperature(T: int, coef: float, every: int):
    """Factor of the query at each position: 1 + coef ln(floor((p + 1) / every) + 1)."""
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1.0) for p in range(T)], dtype=F64)


def head_slopes(H: int):
    return [2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]


def biased_attention(q, k, v, *, scale: float, softcap: float, window: int, slopes, sink=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]: score = cap tanh(q.k scale / cap) - slope_h (i - j), query i sees j with
    0 <= i - j < window (0: every j <= i), softmax whose denominator also holds exp(sink_h)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & ((i - j < window) if window > 0 else (j <= i))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        s = torch.where(seen, s - slopes[h] * (i - j), torch.full_like(s, -math.inf))
        m = s.max(-1, keepdim=True).values
        if sink is not None:
            m = torch.clamp(m, min=float(sink[h]))
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - m)
        out[:, h] = (e / den) @ v[:, g]
    return out


def attention_mixer(h, W: Dict[str, torch.Tensor], m: dict, eps: float, rnd=exact):
    T, h = h.shape[0], rnd(h)
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ W["q"].T + W["q.b"]).view(T, H, d), eps)
    k = rms((h @ W["k"].T + W["k.b"]).view(T, G, d), eps)
    v = (h @ W["v"].T + W["v.b"]).view(T, G, dv)
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    o = biased_attention(q, k, v, scale=m["scale"], softcap=m.get("softcap") or 0.0, window=(m.get("mask") or {}).get("size", 0), slopes=head_slopes(H),
                         sink=W["sink"])
    return rnd(o.reshape(T, H * dv)) @ W["o"].T


# ---- state space ----
def causal_conv(x, w, b):
    """x [T, C], w [C, taps], LAST column = the current token, bias b [C]; zeros before the start; then silu."""
    T, C = x.shape
    taps = w.shape[1]
    y = b.repeat(T, 1).clone()
    for t in range(T):
        for d in range(taps):
            if t - d >= 0:
                y[t] += w[:, taps - 1 - d] * x[t - d]
    return silu(y)


def state_space(x, B, C, dt, a_log, D, state: Optional[list] = None):
    """x [T, H, dv], B / C [T, G, N], dt [T, H] (after softplus): S <- exp(-exp(a_log) dt) S + dt B x^T (S is N x dv), y = S^T C + D x."""
    T, H, dv = x.shape
    G, N = B.shape[1], B.shape[2]
    y = torch.zeros(T, H, dv, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(N, dv, dtype=F64)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + D[h] * x[t, h]
        if state is not None:
            state.append(S)
    return y


def gate_then_group_norm(y, z, w, groups: int, eps: float):
    """y [T, inner] times silu(z), then `groups` equal runs of columns each divided by its own root mean square, times w [inner]."""
    T, n = y.shape
    u = (y * silu(z)).view(T, groups, n // groups)
    return rms(u, eps).reshape(T, n) * w


def mamba_mixer(h, W, m, eps, rnd=exact):
    T, h = h.shape[0], rnd(h)
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    p = h @ W["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = causal_conv(xbc, W["conv"], W["conv.b"])
    x, B, C = xbc[:, :inner].reshape(T, H, dv), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    y = state_space(x, B, C, softplus(dt + W["dt_bias"]), W["A_log"], W["D"]).reshape(T, inner)
    return rnd(gate_then_group_norm(y, z, W["norm"], m["norm_groups"], eps)) @ W["o"].T


# ---- feed-forward ----
def gated_mlp(h, gate, up, down, rnd=exact):
    h = rnd(h)
    return rnd(silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(z, correction, top: int):
    """(chosen [T, top], weights [T, top]) of router logits z [T, E]: softmax scores, chosen by score + correction, weighted by the
    score alone, not renormalised."""
    s = torch.softmax(z, -1)
    idx = (s + correction).topk(top, -1).indices
    return idx, s.gather(-1, idx)


def mixture(h, W, f: dict, rnd=exact):
    """Routed experts, identity experts behind them (weight times h itself), a gated shared expert for every token."""
    E, ident = f["router"]["experts"], f["router"].get("identity", 0)
    idx, wt = route(rnd(h) @ W["router"].T, W["correction"], f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(E + ident):
        w = (wt * (idx == e)).sum(-1, keepdim=True)
        out = out + w * (gated_mlp(h, W[f"e{e}.gate"], W[f"e{e}.up"], W[f"e{e}.down"], rnd) if e < E else h)
    if f.get("shared"):
        out = out + torch.sigmoid(rnd(h) @ W["shared.sg"].T) * gated_mlp(h, W["shared.gate"], W["shared.up"], W["shared.down"], rnd)
    return out


# ---- the model ----
def _sub(W, pre):
    return {k[len(pre):]: v for k, v in W.items() if k.startswith(pre)}


def layer_runs(cfg: dict) -> List[int]:
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None, rnd=exact) -> torch.Tensor:
    """Logits [T, vocab] of one sequence. W: name -> float64 tensor. residuals: receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    nm = lambda x, name: centred_norm(x, W[name], eps)  # noqa: E731
    e = cfg.get("embedding") or {}
    x = embedding(tokens, W["embed"], e.get("scale", 1.0), W.get("bigram"), e.get("bigram"))
    for i in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        mixer = attention_mixer if L["type"] == "attention" else mamba_mixer
        x = x + nm(mixer(nm(x, p + "norm1"), _sub(W, p + "mix."), L["mixer"], eps, rnd), p + "norm1b")
        if L.get("mlp"):
            x = x + nm(mixture(nm(x, p + "norm2"), _sub(W, p + "mlp."), L["mlp"], rnd), p + "norm2b")
        if residuals is not None:
            residuals.append(x.clone())
    return rnd(nm(x, "final.norm")) @ W["head"].T


def greedy(cfg, W, prompt: List[int], n_new: int):
    """Greedy continuation by re-running the whole sequence; also returns each step's top-1 / top-2 margin."""
    toks, margins = list(prompt), []
    for _ in range(n_new):
        lg = forward(cfg, W, toks)[-1]
        top = lg.topk(2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(lg.argmax()))
    return toks, margins
