"""Small Palelix configurations of the tests (sizes, orders and constants of their own) and helpers that draw their weights.
Where random weights would hide a fault the weights are moved: decays between slow and fast that differ from head to head and
channel to channel, convolutions whose taps all matter, expert activations that reach their limit, step vectors as large
as the stream, routers whose logits lie apart."""

from __future__ import annotations

import copy

import torch

from matricxon_b200.config.registry import config_from_dict
from matricxon_b200.weights.random_init import RandomInit, random_tensors


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, limit=0.8):
    """``groups`` = (count, keep) or None, ``limit`` may be None."""
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff} if limit is None else {"ff": ff, "limit": limit}, "router": router}


def lightning(heads, dim, vdim, decay, mlp=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": _delta(heads, kv_heads, dim, vdim, conv), "mlp": mlp}


def parallel(left, right, left_scale, right_scale, mlp=None):
    """``left`` = (heads, kv_heads, dim, vdim, scale, (dims, base) or None), ``right`` = (heads, kv_heads, dim, vdim, conv)."""
    heads, kv_heads, dim, vdim, scale, rot = left
    side = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if rot is not None:
        side["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": side, "left_scale": left_scale, "right": _delta(*right), "right_scale": right_scale}}


def model(width, vocab, layers, eps=1e-5, loop=None):
    out = {"architecture": "Palelix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# sizes that are multiples of four at best, keys wider and narrower than values, half the heads rotated, the run of repeated
# layers at the end with three passes, groups of which one is kept, a layer without a feed-forward
MODEL_A = model(96, 211, [
    parallel((6, 3, 24, 40, 0.3, (12, 500.0)), (4, 2, 20, 28, 3), 0.7, 1.4, mlp=dense(72)),
    lightning(3, 20, 28, [0.9, 0.99, 0.5]),
    delta(6, 2, 12, 20, 5, mlp=moe(40, 6, 2, (3, 1))),
    lightning(2, 24, 16, [0.97, 0.7], mlp=moe(24, 8, 3, (2, 2))),
], loop=(2, 4, 3))

# head sizes that the tensor-core attention kernels take, recurrent heads of 64 and 128, a repeated run in the middle, the
# delta layer first and the parallel one last, groups of one expert each
MODEL_B = model(128, 257, [
    delta(4, 4, 64, 64, 4, mlp=moe(96, 4, 2, (4, 2), limit=None)),
    parallel((8, 2, 64, 64, 0.15, (64, 10000.0)), (2, 1, 128, 64, 4), 1.0, 1.0, mlp=moe(64, 9, 2, (3, 2))),
    lightning(2, 64, 128, [0.97, 0.999], mlp=dense(160)),
    parallel((2, 1, 128, 128, 0.1, (96, 300.0)), (4, 4, 32, 32, 2), -0.6, 0.8),
], loop=(1, 3, 2))

# sizes that are multiples of nothing useful: width 100, an odd vocabulary, recurrent heads of 13 x 7 and 5 x 9, a convolution
# of one tap and one of nine, no rotation, one expert, no repeated run; an eps that keeps the norms of such small heads from
# magnifying 16-bit rounding where a read-out is nearly zero
MODEL_C = model(100, 131, [
    lightning(5, 13, 7, [0.8, 0.95, 0.0, 1.0, 0.6], mlp=moe(52, 10, 3)),
    parallel((5, 5, 12, 20, 0.4, None), (3, 1, 13, 7, 1), 1.3, 0.9, mlp=moe(36, 2, 2)),
    delta(5, 5, 5, 9, 9, mlp=moe(20, 1, 1)),
    parallel((3, 1, 17, 11, 0.5, (2, 50.0)), (2, 2, 6, 30, 2), 0.5, -1.1, mlp=dense(33)),
], eps=0.01)

# recurrent layers only, so no paged cache at all, the whole model repeated
MODEL_D = model(64, 97, [
    delta(1, 1, 96, 24, 3, mlp=dense(48)),
    lightning(9, 8, 8, [0.5 + 0.05 * i for i in range(9)], mlp=moe(40, 6, 2, (2, 1))),
], loop=(0, 2, 2))

# a middle size for long prompts: products of more than a thousand rows, many key tiles, many groups of the recurrences
MODEL_L = model(256, 512, [
    parallel((4, 2, 128, 128, 0.08, (128, 1000000.0)), (4, 2, 64, 128, 4), 0.9, 1.1, mlp=moe(128, 8, 2, (4, 2))),
    lightning(4, 128, 64, [0.9, 0.97, 0.99, 0.998], mlp=dense(384)),
    delta(4, 2, 128, 64, 3, mlp=moe(64, 6, 3, (2, 1))),
    parallel((8, 2, 64, 64, 0.12, (48, 500000.0)), (2, 2, 160, 40, 4), 0.8, 1.0),
], loop=(1, 2, 2))

MODELS = {"A": MODEL_A, "B": MODEL_B, "C": MODEL_C, "D": MODEL_D, "L": MODEL_L}
INIT = RandomInit(weight_std=0.08, bias_std=0.05, norm_weight_std=0.2, norm_bias_std=0.1)
RANKS = {"a1": 7, "g1": 10}          # of the low-rank maps, unlike each other and multiples of nothing


def single_layer(layer: dict, width=64, vocab=120) -> dict:
    return model(width, vocab, [copy.deepcopy(layer)])


def config_of(raw: dict, tensors: dict | None = None):
    """The configuration with the ranks of ``tensors`` (None: of ``RANKS``)."""
    config = config_from_dict(copy.deepcopy(raw))
    if tensors is None:
        return config.with_tensor_shapes(lambda name: (RANKS[name.rsplit(".", 1)[-1]], raw["width"]))
    return config.with_tensor_shapes(lambda name: tuple(tensors[name].shape) if name in tensors else None)


def draw(raw: dict, seed: int, store_dtype=torch.float32, router_gain: float = 1.0) -> dict[str, torch.Tensor]:
    """Random weights with the tensors away from the values that hide them (see above). ``router_gain`` sharpens the
    routers: with a large one, few tokens have two experts so close that 16-bit rounding decides between them."""
    tensors = random_tensors(config_of(raw), seed, INIT, store_dtype)
    generator = torch.Generator().manual_seed(seed + 1)
    for name in tensors:
        shape = tensors[name].shape

        def put(values):
            tensors[name] = values.to(store_dtype)

        last = name.rsplit(".", 1)[-1]
        if name.endswith(".mlp.router"):
            put(tensors[name].float() * 4.0 * router_gain)
        elif last == "conv":
            put(torch.randn(shape, generator=generator) * 0.6)
        elif last == "A_log":
            put(torch.rand(shape, generator=generator) * 3.0 - 2.0)
        elif last == "dt_bias":
            put(torch.rand(shape, generator=generator) * 5.0 - 4.0)
        elif name == "loop.step":
            put(torch.randn(shape, generator=generator))
        elif name == "embed":
            put(tensors[name].float() * 12.0)
        elif last in ("gate", "up"):
            put(tensors[name].float() * 2.0)
        elif last in ("a", "b", "a1", "a2", "g1", "g2"):
            put(tensors[name].float() * 3.0)
        elif ".mix." in name and last in ("q", "k", "v", "g"):
            put(tensors[name].float() * 2.0)
    return tensors


def ids(count: int, vocab: int, seed: int) -> list[int]:
    generator = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (count,), generator=generator).tolist()
