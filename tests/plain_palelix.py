"""Palelix written out plainly: every mechanism as one float64 function, no cache, no batching, no kernels.

The yardstick of the Palelix tests. A model is (config dict as in ``config.json``, dict of float64 tensors by
checkpoint name); ``forward`` runs one whole sequence and returns logits at every position (and, on request, the
stream after every layer run). Nothing here is shared with the engine.

Notation: T tokens, positions p = 0 .. T-1; a matrix W is stored [out, in] and applied as ``x @ W.T``.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6          # under the root of a unit vector


def over_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def over_length(x):
    """x over its length along the last axis."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ---------------------------------------------------------------------- positions
def rotate(x, positions, rot):
    """Rotates the first ``rot["dims"]`` entries of the last axis of x [T, heads, D], entry i with entry i + dims/2."""
    if not rot or rot["dims"] == 0:
        return x
    dims = rot["dims"]
    half = dims // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    angle = positions.to(F64)[:, None, None] * f
    cos, sin = torch.cos(angle), torch.sin(angle)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


# ---------------------------------------------------------------------- convolution, softmax
def causal_conv(u, w):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) for every channel of u [T, C]; zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))


def attend(q, k, v, scale):
    """Causal softmax attention of q [T, H, D] over k [T, G, D] and v [T, G, V] -> [T, H, V]; query head h reads
    key/value head h // (H / G)."""
    T, H = q.shape[0], q.shape[1]
    kv_of = torch.arange(H) // (H // k.shape[1])
    scores = torch.einsum("ihd,jhd->hij", q, k[:, kv_of]) * scale
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    weights = torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)
    return torch.einsum("hij,jhv->ihv", weights, v[:, kv_of])


# ---------------------------------------------------------------------- recurrences
def decaying_sum(q, k, v, decay):
    """o_t = S_t^T q_t with S_t = decay_h S_(t-1) + k_t v_t^T, per head."""
    state = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=F64)
    out = []
    for t in range(q.shape[0]):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out)


def delta_rule(q, k, v, g, beta):
    """q, k [T, H, D], v [T, H, V], g [T, H, D] (a factor per row of the state), beta [T, H]: the state forgets, the
    value it holds under k is moved towards v by beta, then it is read with q."""
    state = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=F64)
    out = []
    for t in range(q.shape[0]):
        state = g[t][:, :, None] * state
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", state, k[t]))
        state = state + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out)


# ---------------------------------------------------------------------- mixers
def lightning(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = silu(h @ w[p + "q"].T).view(T, H, D), silu(h @ w[p + "k"].T).view(T, H, D)
    v = silu(h @ w[p + "v"].T).view(T, H, V)
    o = decaying_sum(q, k, v, torch.tensor(m["decay"], dtype=F64)).reshape(T, H * V)
    return (over_rms(o, eps) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def delta_operands(h, w, p, m):
    """(q, k, v) per value head: convolved, activated, q and k of unit length, q times dim^(-1/2)."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    kv_of = torch.arange(H) // (H // G)
    q = over_length(q.view(T, G, D)) * D ** -0.5
    return q[:, kv_of], over_length(k.view(T, G, D))[:, kv_of], v.view(T, H, V)


def gated_delta(h, w, p, m, eps):
    """One decay per head."""
    T, H = h.shape[0], m["heads"]
    q, k, v = delta_operands(h, w, p, m)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = delta_rule(q, k, v, g[:, :, None].expand(-1, -1, m["dim"]), torch.sigmoid(h @ w[p + "b"].T))
    o = over_rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, m["vdim"])
    return o.reshape(T, -1) @ w[p + "o"].T


def channel_delta(h, w, p, m, eps):
    """One decay per head and key channel; decay and gate through low-rank maps."""
    T, H, D = h.shape[0], m["heads"], m["dim"]
    q, k, v = delta_operands(h, w, p, m)
    z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * softplus(z))
    o = delta_rule(q, k, v, g, torch.sigmoid(h @ w[p + "b"].T))
    o = over_rms(o, eps) * w[p + "norm"] * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, m["vdim"])
    return o.reshape(T, -1) @ w[p + "o"].T


def softmax_attention(h, w, p, m):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    pos = torch.arange(T)
    q = rotate((h @ w[p + "q"].T).view(T, H, m["dim"]), pos, m.get("rot"))
    k = rotate((h @ w[p + "k"].T).view(T, G, m["dim"]), pos, m.get("rot"))
    return attend(q, k, (h @ w[p + "v"].T).view(T, G, m["vdim"]), m["scale"]).reshape(T, -1) @ w[p + "o"].T


def mixer(layer, h, w, p, eps):
    m = layer["mixer"]
    if layer["type"] == "lightning":
        return lightning(h, w, p, m, eps)
    if layer["type"] == "delta":
        return gated_delta(h, w, p, m, eps)
    if layer["type"] == "parallel":
        return (m["left_scale"] * softmax_attention(h, w, p + "left.", m["left"])
                + m["right_scale"] * channel_delta(h, w, p + "right.", m["right"], eps))
    raise ValueError(layer["type"])


# ---------------------------------------------------------------------- feed-forwards
def eligible(scores, groups):
    """[T, experts] bool: the experts of the ``keep`` groups of neighbours whose best score is largest."""
    T, E = scores.shape
    if not groups:
        return torch.ones(T, E, dtype=torch.bool)
    best = scores.view(T, groups["count"], -1).max(dim=-1).values
    kept = torch.argsort(best, dim=-1, descending=True, stable=True)[:, :groups["keep"]]
    open_groups = torch.zeros(T, groups["count"], dtype=torch.bool).scatter_(1, kept, True)
    return open_groups.repeat_interleave(E // groups["count"], dim=1)


def route(h, router, r):
    """(chosen experts [T, top], margin): the margin is the smallest difference of logits that decided anything (between
    the last chosen and the best eligible unchosen expert, and between the last kept and the best dropped group)."""
    z = h @ router.T
    scores = torch.softmax(z, dim=-1)
    groups = r.get("groups")
    allowed = eligible(scores, groups)
    order = torch.argsort(scores.masked_fill(~allowed, -1.0), dim=-1, descending=True, stable=True)
    top = r["top"]
    margin = torch.full((h.shape[0],), math.inf, dtype=F64)
    open_z = z.masked_fill(~allowed, -math.inf)
    if z.shape[1] > top:
        margin = torch.gather(z, 1, order[:, top - 1:top])[:, 0] - torch.gather(open_z, 1, order[:, top:top + 1])[:, 0]
    if groups and groups["keep"] < groups["count"]:
        best = z.view(z.shape[0], groups["count"], -1).max(dim=-1).values.sort(dim=-1, descending=True).values
        margin = torch.minimum(margin, best[:, groups["keep"] - 1] - best[:, groups["keep"]])
    return order[:, :top], margin


def expert(h, gate, up, down, limit):
    g, u = h @ gate.T, h @ up.T
    if limit is not None:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def feed_forward(h, w, p, f, forced=None, heard=None):
    """``forced`` [T, top]: expert choices to use instead of the router's own (the weights are those experts'
    scores). ``heard``: a list that receives (the router's own choice, its margin) of a routed layer."""
    if f["kind"] == "dense":
        return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T
    own, margin = route(h, w[p + "router"], f["router"])
    if heard is not None:
        heard.append((own, margin))
    chosen = own if forced is None else torch.as_tensor(forced).long()
    scores = torch.gather(torch.softmax(h @ w[p + "router"].T, dim=-1), 1, chosen)
    weights = scores / (scores.sum(dim=-1, keepdim=True) + 1e-20)
    out = torch.zeros_like(h)
    for e in range(w[p + "router"].shape[0]):
        rows, slots = (chosen == e).nonzero(as_tuple=True)
        if rows.numel():
            q = f"{p}e{e}."
            y = expert(h[rows], w[q + "gate"], w[q + "up"], w[q + "down"], f["expert"].get("limit"))
            out.index_add_(0, rows, weights[rows, slots][:, None] * y)
    return out


# ---------------------------------------------------------------------- the model
def layer_runs(config):
    """[(layer, number of the pass it opens or None)] in order."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(start)]
    for t in range(loop["times"]):
        runs += [(i, t if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, n)]


def routed_runs(config):
    """The numbers of the layer runs that route."""
    return [run for run, (i, _) in enumerate(layer_runs(config)) if (config["layers"][i].get("mlp") or {}).get("kind") == "moe"]


def forward(config, w, tokens, return_layers=False, forced=None, heard=None):
    """Logits [T, vocab] of one sequence. ``forced``: {number of the layer run: [T, top] expert choices}; ``heard``: a
    list that receives (own choice, margin) of every routed layer run."""
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)].to(F64)
    taps = []
    for run, (i, opens) in enumerate(layer_runs(config)):
        layer, p = config["layers"][i], f"l{i}."
        if opens is not None:
            x = x + w["loop.step"][opens]
        h = over_rms(x, eps) * w[p + "norm1"]
        y = mixer(layer, h, w, p + "mix.", eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, w, p + "mlp.", layer["mlp"], None if forced is None else forced.get(run), heard)
        x = x + y
        taps.append(x.clone())
    logits = (over_rms(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, torch.stack(taps)) if return_layers else logits
