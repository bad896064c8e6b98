"""A plain, slow implementation of the Gumodra design in float64 (or float32), one function per mechanism, written from the
design's equations and sharing no code with the package.  It runs whole sequences at once on the CPU and is what the
framework's kernels, cache, state slots and batching are compared with.

Notation: T tokens at positions 0..T-1, W the model width, x the residual [T, W], h = n1(x).

    layer      x <- x + mixer(h) * s(R1 h + b1) + ff(h) * s(R2 h + b2)   s the sigmoid; one norm for both sublayers and gates
    norm       n(x) = x / sqrt(mean(x^2) + eps) * g with ONE number g
    attention  q = W_q h + b, u = W_k h + b; keys: u normed per head and turned, values: u itself; scores over the last
               ``size`` tokens and the first ``keep_first``, a learned sink in the denominator; W_o(.) + b
    mlstm      S_t = e^(f + m' - m) S' + e^(i - m) k v^T with m = max(f + m', i), n likewise; S^T q / (max(|n q|, e^-m) + 1e-6)
    ff         down(silu(gate h) * up h); or the chosen experts' weighted sum plus s(w h) times a shared expert
    output     head n(x), the embedding times a constant at the start
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

_ROUND = [None]     # set by forward(round_inputs=True): what an engine that computes in 16 bits rounds ahead of a product


def lin(x, w, b=None):
    """W x + b for rows x; the rows are rounded first when forward() asks for it."""
    if _ROUND[0] is not None:
        x = _ROUND[0](x)
    y = x @ w.T
    return y if b is None else y + b


def rms(x, eps: float):
    return torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def one_number_norm(x, g, eps: float):
    return x / rms(x, eps) * g


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------ attention
def turn_halves(x, positions, dims: int, base: float):
    """x [T, H, D]: element i < dims/2 turns with element i + dims/2; elements beyond dims pass."""
    half = dims // 2
    rates = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    ang = (positions.to(x.dtype)[:, None] * rates[None, :])[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * torch.cos(ang) - b * torch.sin(ang), b * torch.cos(ang) + a * torch.sin(ang), x[..., dims:]], dim=-1)


def seen_keys(positions, size: int, keep: int):
    """[T, T]: j is seen from i if j <= i and (i - j < size, or j is one of the first ``keep``); size 0: no window."""
    i, j = positions[:, None], positions[None, :]
    near = (i - j < size) | (j < keep) if size > 0 else torch.ones_like(i - j, dtype=torch.bool)
    return (j <= i) & near


def sink_softmax(scores, seen, sink):
    """Weights of the seen keys; exp(sink) joins the denominator."""
    s = scores.masked_fill(~seen, float("-inf"))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def attention_mixer(h, positions, w, p: str, m: dict, eps: float):
    T, H, G, D = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = lin(h, w[p + ".q"], w[p + ".q.b"]).reshape(T, H, D)
    u = lin(h, w[p + ".k"], w[p + ".k.b"]).reshape(T, G, D)
    q = turn_halves(q / rms(q, eps) * w[p + ".q.norm"], positions, int(rot["dims"]), float(rot["base"]))
    k = turn_halves(u / rms(u, eps) * w[p + ".k.norm"], positions, int(rot["dims"]), float(rot["base"]))
    mask = m.get("mask") or {}
    seen = seen_keys(positions, int(mask.get("size", 0)), int(mask.get("keep_first", 0)))
    heads = []
    for a in range(H):
        g = a // (H // G)
        heads.append(sink_softmax(q[:, a] @ k[:, g].T * float(m["scale"]), seen, w[p + ".sink"][a]) @ u[:, g])
    return lin(torch.cat(heads, dim=-1), w[p + ".o"], w[p + ".o.b"])


# ------------------------------------------------------------------------------------------------ mlstm
def capped(z, cap: float):
    return cap * torch.tanh(z / cap)


def mlstm_recurrence(q, k, v, i, f, state=None):
    """One head: q, k [T, D], v [T, V], i and f [T] (log gates): (o [T, V], (S, n, m) behind the last token)."""
    if state is None:
        S, n = torch.zeros((k.shape[1], v.shape[1]), dtype=q.dtype), torch.zeros(k.shape[1], dtype=q.dtype)
        m = torch.zeros((), dtype=q.dtype)
    else:
        S, n, m = state
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S, n, m = keep * S + take * torch.outer(k[t], v[t]), keep * n + take * k[t], new
        out.append((S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out), (S, n, m)


def mlstm_mixer(h, w, p: str, m: dict, eps: float, states: Optional[list] = None):
    T, H, D, V, cap = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
    q = (lin(h, w[p + ".q"]) * D ** -0.5).reshape(T, H, D)
    k = lin(h, w[p + ".k"]).reshape(T, H, D)
    v = lin(h, w[p + ".v"]).reshape(T, H, V)
    i = capped(lin(h, w[p + ".i"], w[p + ".i.b"]), cap)
    f = torch.nn.functional.logsigmoid(capped(lin(h, w[p + ".f"], w[p + ".f.b"]), cap))
    heads = []
    for a in range(H):
        o, last = mlstm_recurrence(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a])
        heads.append(o / rms(o, eps))
        if states is not None:
            states.append(last)
    return lin(torch.cat(heads, dim=-1) * w[p + ".norm"] * torch.sigmoid(lin(h, w[p + ".g"])), w[p + ".o"])


# ------------------------------------------------------------------------------------------------ feed-forwards
def gated_ff(h, w, p: str):
    return lin(silu(lin(h, w[p + ".gate"])) * lin(h, w[p + ".up"]), w[p + ".down"])


def choose(s, correction, groups, top: int):
    """[T, top] experts: the largest s + correction among the members of the best groups (a group counts as its best)."""
    c = s + correction
    T, E = c.shape
    count, keep = groups
    if count > 1:
        best = c.reshape(T, count, E // count).max(dim=-1).values.argsort(dim=-1, descending=True, stable=True)[:, :keep]
        open_ = torch.zeros((T, count), dtype=torch.bool)
        open_[torch.arange(T)[:, None], best] = True
        c = c.masked_fill(~open_.repeat_interleave(E // count, dim=1), float("-inf"))
    return c.argsort(dim=-1, descending=True, stable=True)[:, :top]


def expert_ff(h, w, p: str, mlp: dict):
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(lin(h, w[p + ".router"]), dim=-1)
    chosen = choose(s, w[p + ".correction"], (int(g["count"]), int(g["keep"])), int(r["top"]))
    part = s.gather(1, chosen)
    part = part / (part.sum(dim=-1, keepdim=True) + 1e-20)
    out = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        t, slot = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            out.index_add_(0, t, gated_ff(h[t], w, f"{p}.e{e}") * part[t, slot][:, None])
    if mlp.get("shared"):
        out = out + torch.sigmoid(lin(h, w[p + ".shared.sg"])) * gated_ff(h, w, p + ".shared")
    return out


# ------------------------------------------------------------------------------------------------ the model
def forward(config: dict, weights: Dict[str, torch.Tensor], tokens, dtype=torch.float64, layers_out: Optional[list] = None,
            round_inputs: bool = False):
    """Logits [T, vocab] of a whole sequence.  ``layers_out`` collects the residual after every layer.  With ``round_inputs``
    the rows that enter a product with a weight matrix are rounded to bfloat16 first, as an engine that computes in 16 bits
    rounds them: how far that alone moves a position says how well conditioned the position is."""
    _ROUND[0] = (lambda t: t.to(torch.bfloat16).to(t.dtype)) if round_inputs else None
    try:
        return _forward(config, weights, tokens, dtype, layers_out)
    finally:
        _ROUND[0] = None


def _forward(config, weights, tokens, dtype, layers_out):
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(tokens.shape[0])
    x = w["embed"][tokens] * float(config["embedding"]["scale"])
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        h = one_number_norm(x, w[p + ".norm1"], eps)
        if layer["type"] == "attention":
            y = attention_mixer(h, positions, w, p + ".mix", layer["mixer"], eps)
        elif layer["type"] == "mlstm":
            y = mlstm_mixer(h, w, p + ".mix", layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        add = y * torch.sigmoid(lin(h, w[p + ".rg1"], w[p + ".rg1.b"]))
        mlp = layer.get("mlp")
        if mlp is not None:
            z = gated_ff(h, w, p + ".mlp") if mlp["kind"] == "dense" else expert_ff(h, w, p + ".mlp", mlp)
            add = add + z * torch.sigmoid(lin(h, w[p + ".rg2"], w[p + ".rg2.b"]))
        x = x + add
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(one_number_norm(x, w["final.norm"], eps), w["head"])


def greedy(config: dict, weights, prompt, new_tokens: int, dtype=torch.float64):
    toks = list(prompt)
    for _ in range(new_tokens):
        toks.append(int(torch.argmax(forward(config, weights, toks, dtype)[-1])))
    return toks[len(prompt):]
