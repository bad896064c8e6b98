"""A plain, slow implementation of the Kadodra design in float64 (or float32), one function per mechanism, written from
the design's equations and sharing no code with the package.  It runs whole sequences at once on the CPU and is what the
framework's kernels, cache, state slots and batching are compared with.

Notation: T tokens at positions 0..T-1, W the model width, x the residual [T, W], x0 the embedding output, h = n(x).

    layer      x <- x + ( mixer(h) + ff(h) ),  h = n1(x), n(x) = x / sqrt(mean(x^2) + eps) * w: one norm for both sublayers
    lightning  q, k, v = silu of their projections,  S_t = g S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t per head (g a constant),
               W_o( n(concat o) * sigmoid(W_g h) )
    latent     scores (q_u . W_uk c_j + q_r . r_j) * scale over the last ``size`` tokens, a learned sink in the denominator
    ff         down(relu(up h)^2), or the mean of the experts that a table gives the token's id
    loop       layers start .. stop-1 run ``times`` times; ahead of every pass but the first, x <- x + x0
    output     s E n(x), E the embedding table
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------ small pieces
_ROUND = [None]     # set by forward(round_inputs=True): what an engine that computes in 16 bits rounds ahead of a product


def lin(x, w):
    """W x for rows x; the rows are rounded first when forward() asks for it."""
    if _ROUND[0] is not None:
        x = _ROUND[0](x)
    return x @ w.T


def rms_norm(x, w, eps: float):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def clipped_gate(gate, up, limit: float):
    """g sigmoid(1.702 g) (u + 1) with g = min(gate, limit) and u held within -limit .. limit."""
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def turn_rates(rot: dict):
    """(angle per position of every pair, factor on cos and sin)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    rates = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return rates, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def crossing(turns):          # the (fractional) pair index that makes ``turns`` turns over ``original`` positions
        return dims * math.log(original / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))

    low = max(math.floor(crossing(float(sc["fast"]))), 0)
    high = min(math.ceil(crossing(float(sc["slow"]))), dims - 1)
    span = max(high - low, 0.001)
    mixed = []
    for i, f in enumerate(rates):
        share = min(max((i - low) / span, 0.0), 1.0)
        mixed.append(share * f / factor + (1.0 - share) * f)
    return mixed, 1.0 + 0.1 * math.log(factor)


def rotate_halves(x, positions, rot: dict):
    """x [T, ..., D]: element i < dims/2 and element i + dims/2 turn as a pair; elements beyond dims pass unchanged."""
    dims = int(rot["dims"])
    half = dims // 2
    rates, mag = turn_rates(rot)
    ang = positions.to(x.dtype)[:, None] * torch.tensor(rates, dtype=x.dtype)[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c, s = (mag * torch.cos(ang)).reshape(shape), (mag * torch.sin(ang)).reshape(shape)
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., dims:]], dim=-1)


def window_mask(positions, size: int):
    """[T, T]: key j is seen from i if 0 <= i - j < size (size 0: every earlier key)."""
    gap = positions[:, None] - positions[None, :]
    return (gap >= 0) & ((gap < size) if size > 0 else torch.ones_like(gap, dtype=torch.bool))


def softmax_with_sink(scores, seen, sink):
    """Rows of weights; exp(sink) joins the denominator and gets no weight of its own (sink None: plain softmax)."""
    s = scores.masked_fill(~seen, float("-inf"))
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return e / total


# ------------------------------------------------------------------------------------------------ mixers
def constant_decay_recurrence(q, k, v, decay: float, state=None):
    """One head, q and k [T, D], v [T, V]: (o [T, V], the last state [D, V])."""
    S = torch.zeros((k.shape[1], v.shape[1]), dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def lightning_mixer(h, w: Dict[str, torch.Tensor], p: str, m: dict, eps: float, states: Optional[list] = None):
    T, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(lin(h, w[p + ".q"])).reshape(T, H, D)
    k = silu(lin(h, w[p + ".k"])).reshape(T, H, D)
    v = silu(lin(h, w[p + ".v"])).reshape(T, H, V)
    heads = []
    for i in range(H):
        o, S = constant_decay_recurrence(q[:, i], k[:, i], v[:, i], float(m["decay"][i]))
        heads.append(o)
        if states is not None:
            states.append(S)
    o = rms_norm(torch.cat(heads, dim=-1), w[p + ".norm"], eps)
    return lin(o * torch.sigmoid(lin(h, w[p + ".g"])), w[p + ".o"])


def latent_mixer(h, positions, w, p: str, m: dict, eps: float):
    T, H = h.shape[0], int(m["heads"])
    D, R, V, C = int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    q = lin(h, w[p + ".q"]).reshape(T, H, D + R)
    q_u, q_r = q[..., :D], rotate_halves(q[..., D:], positions, m["rot"])
    down = lin(h, w[p + ".dkv"])
    c, r = rms_norm(down[:, :C], w[p + ".dkv.norm"], eps), rotate_halves(down[:, C:], positions, m["rot"])
    keys, vals = lin(c, w[p + ".uk"]).reshape(T, H, D), lin(c, w[p + ".uv"]).reshape(T, H, V)
    seen = window_mask(positions, int((m.get("mask") or {}).get("size", 0)))
    heads = []
    for i in range(H):
        scores = (q_u[:, i] @ keys[:, i].T + q_r[:, i] @ r.T) * float(m["scale"])
        heads.append(softmax_with_sink(scores, seen, w[p + ".sink"][i]) @ vals[:, i])
    return lin(torch.cat(heads, dim=-1), w[p + ".o"])


# ------------------------------------------------------------------------------------------------ feed-forwards
def dense_ff(h, w, p: str):
    return lin(relu_squared(lin(h, w[p + ".up"])), w[p + ".down"])


def tabled_experts(h, tokens, w, p: str, mlp: dict):
    """Every token goes through the experts its id has in the table, each with weight 1/top."""
    top, limit = int(mlp["router"]["top"]), float(mlp["expert"]["limit"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        row = h[t:t + 1]
        for e in w[p + ".table"][int(tokens[t])].tolist():
            y = clipped_gate(lin(row, w[f"{p}.e{e}.gate"]), lin(row, w[f"{p}.e{e}.up"]), limit)
            out[t] += lin(y, w[f"{p}.e{e}.down"])[0] / top
    return out


# ------------------------------------------------------------------------------------------------ the model
def order_of_runs(config: dict) -> List[tuple]:
    """[(layer, whether x0 is added ahead of it)] in the order the layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, False) for i in range(a)]
    for t in range(times):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens, dtype=torch.float64, layers_out: Optional[list] = None,
            round_inputs: bool = False):
    """Logits [T, vocab] of a whole sequence.  ``layers_out`` collects the residual after every layer run.  With
    ``round_inputs`` the rows that enter a product with a weight matrix are rounded to bfloat16 first, as an engine that
    computes in 16 bits rounds them: how far that alone moves a position says how well conditioned the position is."""
    _ROUND[0] = (lambda t: t.to(torch.bfloat16).to(t.dtype)) if round_inputs else None
    try:
        return _forward(config, weights, tokens, dtype, layers_out)
    finally:
        _ROUND[0] = None


def _forward(config, weights, tokens, dtype, layers_out):
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(tokens.shape[0])
    x0 = w["embed"][tokens]
    x = x0.clone()
    for i, again in order_of_runs(config):
        layer, p = config["layers"][i], f"l{i}"
        if again:
            x = x + x0
        h = rms_norm(x, w[p + ".norm1"], eps)
        if layer["type"] == "lightning":
            y = lightning_mixer(h, w, p + ".mix", layer["mixer"], eps)
        elif layer["type"] == "latent_attention":
            y = latent_mixer(h, positions, w, p + ".mix", layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        mlp = layer.get("mlp")
        if mlp is not None:
            y = y + (dense_ff(h, w, p + ".mlp") if mlp["kind"] == "dense" else tabled_experts(h, tokens, w, p + ".mlp", mlp))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return float(config.get("logit_scale", 1.0)) * lin(rms_norm(x, w["final.norm"], eps), w["embed"])


def greedy(config: dict, weights, prompt, new_tokens: int, dtype=torch.float64):
    toks = list(prompt)
    for _ in range(new_tokens):
        toks.append(int(torch.argmax(forward(config, weights, toks, dtype)[-1])))
    return toks[len(prompt):]
