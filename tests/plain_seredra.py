"""Seredra written out plainly: every mechanism as one float64 function, no cache, no batching, no kernels.

The yardstick of the Seredra tests. A model is (config dict as in ``config.json``, dict of float64 tensors by
checkpoint name); ``forward`` runs one whole sequence and returns logits at every position (and, on request, the
stream after every layer). Nothing here is shared with the engine.

Notation: T tokens, positions p = 0 .. T-1; a matrix W is stored [out, in] and applied as ``x @ W.T``.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def unit(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


# ---------------------------------------------------------------------- positions
def frequencies(dims, base, scaling=None):
    """([dims/2] radians per position, factor on cos and sin). ``scaling``: {factor, original, fast, slow} blends
    every plain frequency f with f / factor along a ramp over the pair's index."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    if not scaling:
        return f, 1.0

    def pair_at(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_at(scaling["fast"])), 0)
    hi = min(math.ceil(pair_at(scaling["slow"])), dims - 1)
    ramp = ((torch.arange(half, dtype=F64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """Rotates the first ``rot["dims"]`` entries of the last axis of x [T, heads, D], entry i with entry i + dims/2."""
    if not rot or rot["dims"] == 0:
        return x
    dims = rot["dims"]
    half = dims // 2
    f, amplitude = frequencies(dims, rot["base"], rot.get("scaling"))
    angle = positions.to(F64)[:, None, None] * f
    cos, sin = torch.cos(angle) * amplitude, torch.sin(angle) * amplitude
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def temperature(positions, coef, every):
    return 1.0 + coef * torch.log(torch.floor((positions.to(F64) + 1.0) / every) + 1.0)


def distance_bias(n, r1, r2):
    """[H, n, n]: r1_h ln(1 + r2_h (i - j)) for j <= i, zero above the diagonal."""
    d = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).clamp(min=0).to(F64)
    return r1[:, None, None] * torch.log(1.0 + r2[:, None, None] * d)


# ---------------------------------------------------------------------- convolution, softmax
def causal_conv(u, w, bias=None):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) for every channel of u [T, C]; zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    y = sum(w[:, j] * padded[j:j + u.shape[0]] for j in range(taps))
    return y if bias is None else y + bias


def attend(q, k, v, scale, softcap=None, bias=None):
    """Causal softmax attention of q [T, H, D] over k [T, G, D] and v [T, G, V] -> [T, H, V]; query head h reads
    key/value head h // (H / G)."""
    T, H = q.shape[0], q.shape[1]
    kv_of = torch.arange(H) // (H // k.shape[1])
    scores = torch.einsum("ihd,jhd->hij", q, k[:, kv_of]) * scale
    if softcap is not None:
        scores = softcap * torch.tanh(scores / softcap)
    if bias is not None:
        scores = scores - bias
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    weights = torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)
    return torch.einsum("hij,jhv->ihv", weights, v[:, kv_of])


# ---------------------------------------------------------------------- mixers
def keys_values(h, w, p, m, eps):
    """The keys and values an ``attention`` layer stores: projected, convolved, keys normalised over all heads."""
    T, G = h.shape[0], m["kv_heads"]
    k = causal_conv(h @ w[p + "k"].T + w[p + "k.b"], w[p + "k.conv"])
    v = causal_conv(h @ w[p + "v"].T + w[p + "v.b"], w[p + "v.conv"])
    return (unit(k, eps) * w[p + "k.norm"]).view(T, G, m["dim"]), v.view(T, G, m["vdim"])


def attention(h, w, p, m, eps, kv):
    T, H = h.shape[0], m["heads"]
    q = causal_conv(h @ w[p + "q"].T + w[p + "q.b"], w[p + "q.conv"])
    q = unit(q, eps) * w[p + "q.norm"]
    q = q * temperature(torch.arange(T), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
    o = attend(q.view(T, H, m["dim"]), *kv, m["scale"], bias=distance_bias(T, w[p + "r1"], w[p + "r2"]))
    return o.reshape(T, -1) @ w[p + "o"].T + w[p + "o.b"]


def capped_attention(h, w, p, m, eps):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = (h @ w[p + "q"].T).view(T, H, D), (h @ w[p + "k"].T).view(T, G, D)
    pos = torch.arange(T)
    qn = rotate(unit(q, eps) * w[p + "q.norm"], pos, m.get("rot"))
    kn = rotate(unit(k, eps) * w[p + "k.norm"], pos, m.get("rot"))
    return attend(qn, kn, k, m["scale"], softcap=m["softcap"]).reshape(T, -1) @ w[p + "o"].T


def selective_scan(x, dt, b, c, a, d):
    """y [T, C] of S[c, n] <- exp(dt_c a[c, n]) S[c, n] + dt_c x_c b_n, y_c = sum_n S[c, n] c_n + d_c x_c."""
    state = torch.zeros_like(a)
    out = []
    for t in range(x.shape[0]):
        state = torch.exp(dt[t][:, None] * a) * state + (dt[t] * x[t])[:, None] * b[t][None, :]
        out.append(state @ c[t] + d * x[t])
    return torch.stack(out)


def mamba(h, w, p, m):
    inner, rank, n = m["inner"], m["dt_rank"], m["state"]
    xz = h @ w[p + "in"].T
    x = silu(causal_conv(xz[:, :inner], w[p + "conv"], w[p + "conv.b"]))
    z = xz[:, inner:]
    low = x @ w[p + "x"].T
    dt = torch.nn.functional.softplus(low[:, :rank] @ w[p + "dt"].T + w[p + "dt.b"], threshold=1e9)
    y = selective_scan(x, dt, low[:, rank:rank + n], low[:, rank + n:], -torch.exp(w[p + "A_log"]), w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


def linear_recurrence(q, k, v, decay):
    """o_t = S_t^T q_t with S_t = decay_h S_(t-1) + k_t v_t^T, per head."""
    state = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=F64)
    out = []
    for t in range(q.shape[0]):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out)


def retention(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rotate((h @ w[p + "q"].T).view(T, H, D), pos, m.get("rot"))
    k = rotate((h @ w[p + "k"].T).view(T, H, D), pos, m.get("rot")) * D ** -0.5
    o = linear_recurrence(q, k, (h @ w[p + "v"].T).view(T, H, V), torch.tensor(m["decay"], dtype=F64))
    return (unit(o, eps).reshape(T, H * V) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixer(layer, h, w, p, eps, stored):
    """``stored``: {layer index: keys and values}, read by layers that attend over another layer's."""
    m = layer["mixer"]
    if layer["type"] == "attention":
        return attention(h, w, p, m, eps, stored)
    if layer["type"] == "retention":
        return retention(h, w, p, m, eps)
    if layer["type"] == "parallel":
        return (m["left_scale"] * capped_attention(h, w, p + "left.", m["left"], eps)
                + m["right_scale"] * mamba(h, w, p + "right.", m["right"]))
    raise ValueError(layer["type"])


# ---------------------------------------------------------------------- feed-forwards
def route(h, router, top):
    """(chosen experts [T, top], their scores, margin between the last chosen and the first unchosen logit)."""
    z = h @ router.T
    order = torch.argsort(z, dim=-1, descending=True, stable=True)
    chosen = order[:, :top]
    if z.shape[1] > top:
        margin = torch.gather(z, 1, order[:, top - 1:top])[:, 0] - torch.gather(z, 1, order[:, top:top + 1])[:, 0]
    else:
        margin = torch.full((h.shape[0],), math.inf, dtype=F64)
    return chosen, torch.sigmoid(torch.gather(z, 1, chosen)), margin


def gated(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def feed_forward(h, w, p, f, forced=None, heard=None):
    """``forced`` [T, top]: expert choices to use instead of the router's own (the weights are those experts'
    scores). ``heard``: a list that receives (the router's own choice, its margin) of a routed layer."""
    if f["kind"] == "dense":
        return relu_squared(h @ w[p + "up"].T) @ w[p + "down"].T
    own, _, margin = route(h, w[p + "router"], f["router"]["top"])
    if heard is not None:
        heard.append((own, margin))
    chosen = own if forced is None else torch.as_tensor(forced).long()
    score = torch.sigmoid(torch.gather(h @ w[p + "router"].T, 1, chosen))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for slot in range(chosen.shape[1]):
            q = f"{p}e{int(chosen[t, slot])}."
            out[t] += gated(score[t, slot] * h[t:t + 1], w[q + "gate"], w[q + "up"], w[q + "down"])[0]
    return out


def routed_layers(config):
    return [i for i, layer in enumerate(config["layers"]) if (layer.get("mlp") or {}).get("kind") == "moe"]


def forward(config, w, tokens, return_layers=False, forced=None, heard=None):
    """Logits [T, vocab] of one sequence. ``forced``: {layer index: [T, top] expert choices}; ``heard``: a list that
    receives (own choice, margin) of every routed layer."""
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)].to(F64) * config["embedding"]["scale"]
    stored, taps = {}, []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = unit(x, eps) * w[p + "norm1"]
        kv = None
        if layer["type"] == "attention":
            source = layer["mixer"].get("kv_from")
            if source is None:
                stored[i] = keys_values(h, w, p + "mix.", layer["mixer"], eps)
            kv = stored[i if source is None else source]
        x = x + mixer(layer, h, w, p + "mix.", eps, kv)
        if layer.get("mlp") is not None:
            x = x + feed_forward(unit(x, eps) * w[p + "norm2"], w, p + "mlp.", layer["mlp"],
                                 None if forced is None else forced.get(i), heard)
        taps.append(x.clone())
    logits = (unit(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, torch.stack(taps)) if return_layers else logits
