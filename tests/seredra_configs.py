"""Small Seredra configurations of the tests (sizes, orders and constants of their own) and helpers that draw their
weights. Where random weights would hide a fault the weights are moved: distance biases whose numbers differ from head to
head and are large enough to change the softmax, steps of the recurrence between slow and fast, decays near and far from
one, routers whose logits lie apart."""

from __future__ import annotations

import copy

import torch

from matricxon_b200.config.registry import config_from_dict
from matricxon_b200.weights.random_init import RandomInit, random_tensors


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def conv_attention(heads, kv_heads, dim, vdim, scale, conv, temp, kv_from=None, mlp=None):
    """``temp`` = (coef, every)."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv,
             "q_temp": {"coef": temp[0], "every": temp[1]}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def parallel(left, right, left_scale, right_scale, mlp=None):
    """``left`` = (heads, kv_heads, dim, scale, softcap, rot or None), ``right`` = (inner, state, dt_rank, conv)."""
    heads, kv_heads, dim, scale, softcap, rot = left
    inner, state, dt_rank, conv = right
    side = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": softcap}
    if rot is not None:
        side["rot"] = rot
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": side, "left_scale": left_scale, "right_scale": right_scale,
                      "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}}


def retention(heads, dim, vdim, decay, rot, mlp=None):
    """``rot`` = (dims, base) or None."""
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot is not None:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "retention", "mixer": mixer, "mlp": mlp}


def turned(dims, base, scaling=None):
    rot = {"dims": dims, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return rot


def model(width, vocab, embedding_scale, layers, eps=1e-5):
    return {"architecture": "Seredra", "width": width, "vocab": vocab, "embedding": {"scale": embedding_scale},
            "norm": {"eps": eps}, "layers": layers}


# odd head sizes with keys wider and narrower than values, convolutions of four and two taps, a layer without a
# feed-forward, a shared cache with another layer in between, fewer rotated entries than the head has, thirteen
# states, a step rank that is a multiple of nothing, top 2 of 5 experts
MODEL_A = model(96, 211, 3.0, [
    conv_attention(6, 3, 24, 40, 0.2, 4, (0.4, 19)),
    retention(3, 20, 28, [0.9, 0.99, 0.5], (12, 900.0), mlp=moe(40, 5, 2)),
    parallel((4, 1, 40, 0.25, 4.0, turned(24, 5000.0, (4.0, 64, 8.0, 1.0))), (72, 13, 9, 3), 0.7, 1.4, mlp=dense(72)),
    conv_attention(3, 3, 24, 40, 0.3, 2, (0.9, 7), kv_from=0, mlp=moe(24, 3, 1)),
])

# head sizes that the tensor-core attention kernels take (64 and 128), groups of four, two and one query heads, states
# of 16 and 40, the parallel layer first and last, two layers that share the same source
MODEL_B = model(128, 257, 1.0, [
    parallel((8, 2, 64, 0.12, 20.0, turned(64, 10000.0)), (160, 16, 8, 4), 1.0, 1.0, mlp=moe(96, 4, 2)),
    conv_attention(8, 2, 64, 64, 0.15, 3, (0.2, 32), mlp=dense(160)),
    conv_attention(8, 2, 64, 64, 0.1, 5, (0.6, 50), kv_from=1),
    retention(2, 64, 128, [0.97, 0.999], (64, 10000.0), mlp=moe(64, 9, 3)),
    conv_attention(2, 2, 64, 64, 0.1, 3, (0.3, 64), kv_from=1, mlp=dense(96)),
    parallel((2, 1, 128, 0.08, 30.0, turned(96, 300.0, (16.0, 32, 4.0, 1.0))), (96, 40, 12, 2), -0.6, 0.8),
])

# sizes that are multiples of nothing useful: width 100, odd vocabulary, heads of 12 and 20, one state per channel, a
# step rank of one, a convolution of one tap, no rotation, one expert, a period of one position
MODEL_C = model(100, 131, 0.5, [
    retention(5, 12, 20, [0.8, 0.95, 0.0, 1.0, 0.6], None, mlp=moe(52, 10, 3)),
    parallel((5, 5, 12, 0.4, 1.5, None), (60, 1, 1, 1), 1.3, 0.9, mlp=moe(36, 2, 2)),
    conv_attention(5, 1, 20, 12, 0.3, 1, (1.1, 1), mlp=moe(20, 1, 1)),
])
# recurrent layers only: no paged cache at all in the model
MODEL_D = model(64, 97, 2.0, [
    retention(1, 96, 24, [0.995], (2, 50.0), mlp=dense(48)),
    retention(9, 8, 8, [0.5 + 0.05 * i for i in range(9)], (8, 100.0), mlp=moe(40, 6, 2)),
])

# a middle size for long prompts: products of more than a thousand rows, many key chunks, heads of 64 in a group of four
# and of 128 in a group of two, 288 channels of 24 states
MODEL_L = model(256, 512, 4.0, [
    parallel((8, 2, 64, 0.12, 15.0, turned(48, 500000.0, (8.0, 512, 16.0, 1.0))), (288, 24, 16, 4), 0.9, 1.1,
             mlp=moe(128, 8, 2)),
    conv_attention(4, 2, 128, 128, 0.08, 4, (0.3, 100), mlp=dense(384)),
    retention(4, 128, 64, [0.9, 0.97, 0.99, 0.998], (128, 1000000.0), mlp=moe(64, 6, 3)),
    conv_attention(8, 2, 128, 128, 0.06, 3, (0.5, 33), kv_from=1),
])

MODELS = {"A": MODEL_A, "B": MODEL_B, "C": MODEL_C, "D": MODEL_D, "L": MODEL_L}
INIT = RandomInit(weight_std=0.08, bias_std=0.05, norm_weight_std=0.2, norm_bias_std=0.1)


def single_layer(layer: dict, width=64, vocab=120, embedding_scale=1.5) -> dict:
    return model(width, vocab, embedding_scale, [copy.deepcopy(layer)])


def draw(raw: dict, seed: int, store_dtype=torch.float32, router_gain: float = 1.0) -> dict[str, torch.Tensor]:
    """Random weights with the tensors away from the values that hide them (see above). ``router_gain`` sharpens the
    routers: with a large one, few tokens have two experts so close that 16-bit rounding decides between them."""
    tensors = random_tensors(config_from_dict(copy.deepcopy(raw)), seed, INIT, store_dtype)
    generator = torch.Generator().manual_seed(seed + 1)
    for name in tensors:
        shape = tensors[name].shape

        def put(values):
            tensors[name] = values.to(store_dtype)

        last = name.rsplit(".", 1)[-1]
        if name.endswith(".mlp.router"):
            put(tensors[name].float() * 4.0 * router_gain)
        elif name.endswith(".conv"):
            put(torch.randn(shape, generator=generator) * 0.5)
        elif last == "r1":
            put(torch.rand(shape, generator=generator) * 2.5 - 0.4)
        elif last == "r2":
            put(torch.rand(shape, generator=generator) * 0.8 + 0.05)
        elif last == "A_log":
            put(torch.rand(shape, generator=generator) * 3.0 - 1.0)
        elif name.endswith(".dt.b"):
            put(torch.rand(shape, generator=generator) * 5.0 - 4.0)
        elif name.endswith(".right.in") or name.endswith(".right.dt"):
            put(tensors[name].float() * 1.5)
        elif name.endswith(".right.o"):
            put(tensors[name].float() * 0.7)
        elif name == "embed":
            put(tensors[name].float() * 6.0)
        elif last in ("gate", "up"):
            put(tensors[name].float() * 1.5)
        elif ".mix." in name and last in ("q", "k", "v", "g"):
            put(tensors[name].float() * 2.0)
    return tensors


def ids(count: int, vocab: int, seed: int) -> list[int]:
    generator = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (count,), generator=generator).tolist()
