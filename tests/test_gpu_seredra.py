"""Seredra through the engine against the plain implementation (tests/plain_seredra.py): every mechanism alone, then whole
models cut and batched every way, in float32 and bfloat16, with pools so small that pages and slots are used again. Sizes,
orders and constants are the tests' own."""

import copy
import json
import math
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_seredra as plain
from matricxon_b200.config.registry import config_from_dict
from matricxon_b200.engine.core import model_from_tensors
from matricxon_b200.engine.replay import TraceReplayer
from matricxon_b200.ops import kernels
from matricxon_b200.ops.linear import EPILOGUE_RELU2, linear
from seredra_configs import (MODELS, conv_attention, dense, draw, ids, model, moe, parallel, retention, single_layer,
                             turned)
from trace_utils import ROOT

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
CHUNKS = [7, 2, 5, 3, 11, 2, 4, 13, 2, 9]
F64 = torch.float64


def limit_for(dtype: str, reference: np.ndarray) -> float:
    scale = max(1.0, float(np.abs(reference).max()))
    return (2e-4 if dtype == "float32" else 0.06) * scale


def rounded(tensors: dict, dtype: str) -> dict:
    """What the engine holds: a bfloat16 engine reads bfloat16 matrices, so the plain side gets the same."""
    if dtype == "float32":
        return tensors
    return {name: value.to(torch.bfloat16).float() for name, value in tensors.items()}


def doubles(tensors: dict) -> dict:
    return {name: value.double() for name, value in tensors.items()}


class Run:
    """One engine over one model: requests fed in portions, logits kept per (request, position).

    A bfloat16 engine may send a token to another expert than the plain model does when two router logits lie
    closer than 16-bit rounding resolves, and the positions that attend to such a token differ then too. That is no
    fault, so the bfloat16 runs listen to the engine's choices (``StepRunner.taps``; such steps run launch by launch)
    and hand them to the plain model, which is then compared at every position; where the plain model's own choice is
    clear, the engine's is the same but for one in fifty. float32 runs listen to nothing, replay captured steps and
    are compared with the plain model's own routing."""

    clear = unclear = 0

    def __init__(self, raw: dict, tensors: dict, dtype: str, max_tokens: int, max_requests: int = 4,
                 page_size: int = 16) -> None:
        self.raw, self.dtype = raw, dtype
        self.weights = rounded(tensors, dtype)
        self.plain_weights = doubles(self.weights)
        config = config_from_dict(copy.deepcopy(raw))
        model = model_from_tensors(config, self.weights, dtype=dtype, device=DEVICE, page_size=page_size)
        self.replayer = TraceReplayer(None, dtype, max_tokens, page_size=page_size, device=DEVICE,
                                      max_requests=max_requests, model=model, poison_cache=True)
        self.routed = plain.routed_layers(raw)
        self.listens = dtype == "bfloat16" and bool(self.routed)
        if self.listens:
            self.replayer.core.runner.taps = ("expert_choices",)
        self.logits: dict[tuple[str, int], np.ndarray] = {}
        self.choices: dict[tuple[str, int], list] = {}
        self.progress: dict[str, int] = {}
        self.slots_seen: dict[str, int] = {}

    def step(self, portions: list[tuple[str, list[int]]], end=()) -> None:
        entries, keys = [], []
        for request, tokens in portions:
            start = self.progress.get(request, 0)
            entries.append({"id": request, "tokens": tokens, "want": list(range(len(tokens)))})
            keys.extend((request, start + i) for i in range(len(tokens)))
            self.progress[request] = start + len(tokens)
        out = self.replayer.step(entries, [])
        rows = list(self.replayer.last_rows)
        if self.listens:
            heard = [layer.cpu() for layer in self.replayer.core.runner.last_taps["expert_choices"]]
            assert len(heard) == len(self.routed)
            for row, key in enumerate(keys):
                self.choices[key] = [layer[row].tolist() for layer in heard]
        for request, _ in portions:
            self.slots_seen[request] = self.replayer.core.cache.record(request).state_slot
        if end:
            self.replayer.step([], list(end))
            for request in end:
                self.progress.pop(request, None)
        assert rows == keys
        for key, row in zip(keys, out.numpy()):
            self.logits[key] = row
        self.replayer.core.cache.check_invariants()

    def feed(self, request: str, tokens: list[int], sizes, end: bool = True) -> None:
        """One request alone, cut into portions of the given sizes (a list, then one by one; or a function of
        the turn)."""
        start, turn = 0, 0
        while start < len(tokens):
            if isinstance(sizes, list):
                size = sizes[turn] if turn < len(sizes) else 1
            else:
                size = sizes(turn)
            size = min(size, len(tokens) - start)
            turn += 1
            last = start + size == len(tokens)
            self.step([(request, tokens[start:start + size])], end=[request] if last and end else [])
            start += size

    def check(self, request: str, tokens: list[int], first: int = 0) -> None:
        forced, heard = None, []
        if self.listens:
            forced = {layer: [self.choices[(request, i)][k] for i in range(len(tokens))]
                      for k, layer in enumerate(self.routed)}
        want = plain.forward(self.raw, self.plain_weights, tokens, forced=forced, heard=heard).numpy()
        if self.listens:
            # under the engine's routing the plain model's stream is the engine's: where its own choice there is
            # clear, it is the engine's
            for k, (own, margin) in enumerate(heard):
                clear = np.nonzero(margin.numpy() > 0.6)[0]
                Run.clear += len(clear)
                Run.unclear += len(tokens) - len(clear)
                theirs = forced[self.routed[k]]
                same = sum(sorted(own[t].tolist()) == sorted(theirs[t]) for t in clear)
                assert same >= len(clear) - max(1, len(clear) // 50), (request, k, same, len(clear))
        got = np.stack([self.logits[(request, i)] for i in range(first, len(tokens))])
        worst = np.abs(got - want[first:]).max(axis=1)
        limit = limit_for(self.dtype, want)
        bad = np.nonzero(~(worst <= limit))[0]
        # float32 is strict. In bfloat16 a model of several layers with sharp softmaxes magnifies a rounding
        # difference of one layer in the next at a few positions (one layer alone, fed the engine's own input, stays
        # far inside the limit): of a long prompt one position in a hundred may pass the limit, none by half
        allowed = len(tokens) // 100 if self.dtype == "bfloat16" else 0
        assert bad.size <= allowed and (bad.size == 0 or worst[bad].max() <= 1.5 * limit), (
            f"{request}: first wrong position {first + bad[0]} of {len(tokens)}, "
            f"error {worst[bad[0]]:.3e} > {limit:.1e}; {bad.size} positions over")


def cycle(turn: int) -> int:
    return CHUNKS[turn % len(CHUNKS)]


def ints(values) -> torch.Tensor:
    return torch.tensor(values, dtype=torch.int32, device=DEVICE)


def word() -> torch.Tensor:
    return torch.zeros(1, dtype=torch.int32, device=DEVICE)


class Batch:
    """Sequences that bring ``q_lens`` tokens each after ``contexts`` earlier ones, in the slots given."""

    def __init__(self, q_lens, contexts, slots):
        self.q_lens, self.contexts = q_lens, contexts
        self.cu = [0] + [int(x) for x in np.cumsum(q_lens)]
        self.tok_seq = ints([s for s, n in enumerate(q_lens) for _ in range(n)])
        self.positions = ints([c + i for c, n in zip(contexts, q_lens) for i in range(n)])
        self.cu_q, self.slots, self.n = ints(self.cu), ints(slots), self.cu[-1]

    def rows(self, s):
        return slice(self.cu[s], self.cu[s + 1])


def batches_of(cuts, slots):
    """The steps that bring sequence s in portions ``cuts[s]`` (0: it sits a step out)."""
    done = [0] * len(cuts)
    for step in range(max(len(c) for c in cuts)):
        live = [s for s in range(len(cuts)) if step < len(cuts[s]) and cuts[s][step] > 0]
        yield live, Batch([cuts[s][step] for s in live], [done[s] for s in live], [slots[s] for s in live])
        for s in live:
            done[s] += cuts[s][step]


# ---------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("backend, dtype, m, n, k", [
    ("simt", torch.float32, 37, 70, 50), ("simt", torch.bfloat16, 19, 33, 64), ("skinny", torch.bfloat16, 5, 100, 96),
    ("skinny", torch.bfloat16, 16, 64, 128), ("stream", torch.bfloat16, 100, 300, 256), ("library", torch.bfloat16, 40, 72, 80),
    ("library", torch.bfloat16, 33, 63, 40), ("tcgen05", torch.bfloat16, 100, 96, 72), ("tcgen05", torch.bfloat16, 700, 260, 200),
    ("tcgen05", torch.bfloat16, 2100, 520, 256)])
def test_squared_relu_in_the_epilogue_of_every_product(backend, dtype, m, n, k):
    gen = torch.Generator().manual_seed(m + n)
    x, w, b = torch.randn(m, k, generator=gen), torch.randn(n, k, generator=gen) * 0.2, torch.randn(n, generator=gen)
    x, w = x.to(dtype), w.to(dtype)
    want = plain.relu_squared(x.double() @ w.double().T + b.double())
    got = linear(x.to(DEVICE), w.to(DEVICE), b.to(DEVICE), EPILOGUE_RELU2, backend=backend)
    assert got.dtype == dtype
    tol = 1e-4 if dtype == torch.float32 else 2e-2
    assert torch.allclose(got.double().cpu(), want, rtol=tol, atol=tol * float(want.max()) * 0.1)
    assert float((got == 0).float().mean()) > 0.2                       # the negative half is exactly zero


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden, rows", [(40, 9), (96, 3), (1002, 70), (4100, 5), (2048, 300), (33000, 2)])
@pytest.mark.parametrize("biased", [True, False])
def test_norm_that_forms_the_sum_before_it(dtype, hidden, rows, biased):
    torch.manual_seed(hidden)
    x, acc = torch.randn(rows, hidden, device=DEVICE) * 3, torch.randn(rows, hidden, device=DEVICE) * 2
    bias = torch.randn(hidden, device=DEVICE) if biased else None
    weight = torch.randn(hidden, device=DEVICE)
    want_x = x.double() + acc.double() + (bias.double() if biased else 0.0)
    stream, out = x.clone(), torch.empty(rows, hidden, dtype=dtype, device=DEVICE)
    kernels.rmsnorm_pending(stream, acc, bias, weight, 0.0, 1e-3, out)
    assert torch.allclose(stream.double(), want_x, rtol=1e-6, atol=1e-5)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(out.double(), plain.unit(want_x, 1e-3) * weight.double(), rtol=tol, atol=tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv, dim, rot, scaling", [(6, 3, 24, 12, None), (4, 1, 40, 40, (4.0, 64, 8.0, 1.0)),
                                                          (2, 2, 128, 64, (16.0, 32, 4.0, 1.0)), (5, 5, 12, 0, None)])
def test_values_that_are_the_projected_keys_and_an_amplitude_on_the_angles(dtype, heads, kv, dim, rot, scaling):
    gen = torch.Generator().manual_seed(dim)
    n, page, value_scale = 9, 4, 1.7
    hd = -(-dim // 16) * 16
    proj = torch.randn(n, (heads + kv) * dim + 3, generator=gen) * 2
    positions = torch.tensor([0, 1, 2, 3, 50, 51, 1000, 7, 8], dtype=torch.int32)
    wq, wk = torch.randn(dim, generator=gen), torch.randn(dim, generator=gen)
    spec = turned(rot, 700.0, scaling) if rot else None
    freq, amplitude = plain.frequencies(rot, 700.0, spec.get("scaling")) if rot else (torch.empty(0), 1.0)
    slots = torch.randperm(5 * page, generator=gen)[:n].to(torch.int32)
    cache = torch.full((5, 2, kv, page, hd), 7.0, dtype=dtype, device=DEVICE)
    q_out, status = torch.empty(n, heads * hd, dtype=dtype, device=DEVICE), word()
    kernels.norm_rotate_kv_write(proj.to(DEVICE), positions.to(DEVICE), freq.float().to(DEVICE), rot, False, wq.to(DEVICE),
                                 wk.to(DEVICE), 1e-4, slots.to(DEVICE), cache, q_out, heads, kv, dim, dim, status,
                                 amplitude=amplitude, values_are_keys=True, value_scale=value_scale)
    assert int(status.item()) == 0
    p64 = proj.double()
    k = p64[:, heads * dim:(heads + kv) * dim].view(n, kv, dim)
    want_q = plain.rotate(plain.unit(p64[:, :heads * dim].view(n, heads, dim), 1e-4) * wq.double(), positions, spec)
    want_k = plain.rotate(plain.unit(k, 1e-4) * wk.double(), positions, spec)
    tol = 2e-3 if dtype == torch.float32 else 3e-2
    assert torch.allclose(q_out.double().cpu().view(n, heads, hd)[:, :, :dim], want_q, rtol=tol, atol=tol)
    host = cache.double().cpu()
    for t in range(n):
        pg, off = int(slots[t]) // page, int(slots[t]) % page
        assert torch.allclose(host[pg, 0, :, off, :dim], want_k[t], rtol=tol, atol=tol)
        stored = host[pg, 1].view(kv, hd, page)
        assert torch.allclose(stored[:, :dim, off], k[t] * value_scale, rtol=1e-2, atol=1e-5)
        assert hd == dim or float(stored[:, dim:, off].abs().max()) == 0.0


def _paged_case(dtype, n_heads, n_kv, hd, page_size, contexts, q_lens, seed, spikes=()):
    """Queries and keys of unit root mean square in a paged cache with shuffled pages. ``spikes`` = (sequence, key
    position): that key equals the sequence's last query's first head of each group."""
    gen = torch.Generator().manual_seed(seed)
    n_seqs, n_tok = len(contexts), sum(q_lens)
    totals = [c + q for c, q in zip(contexts, q_lens)]
    pages_of = [-(-t // page_size) for t in totals]
    n_pages = sum(pages_of) + 3
    order = torch.randperm(n_pages, generator=gen).tolist()
    tables = torch.full((n_seqs, max(pages_of)), -1, dtype=torch.int32)
    cache = torch.zeros((n_pages, 2, n_kv, page_size, hd))
    unit = lambda x: x / x.pow(2).mean(-1, keepdim=True).sqrt()
    q = unit(torch.randn(n_tok, n_heads, hd, generator=gen)).reshape(n_tok, n_heads * hd)
    keys, values, group, row = [], [], n_heads // n_kv, 0
    for s in range(n_seqs):
        k = unit(torch.randn(totals[s], n_kv, hd, generator=gen))
        v = torch.randn(totals[s], n_kv, hd, generator=gen)
        last = row + q_lens[s] - 1
        for seq, where in spikes:
            if seq == s:
                for g in range(n_kv):
                    k[where, g] = q[last].view(n_heads, hd)[g * group]
        keys.append(k)
        values.append(v)
        for lp in range(pages_of[s]):
            page = order.pop()
            tables[s, lp] = page
            lo, hi = lp * page_size, min((lp + 1) * page_size, totals[s])
            cache[page, 0, :, :hi - lo] = k[lo:hi].transpose(0, 1)
            cache[page, 1].view(n_kv, hd, page_size)[:, :, :hi - lo] = v[lo:hi].permute(1, 2, 0)
        row += q_lens[s]
    return q.to(dtype).to(DEVICE), cache.to(dtype).to(DEVICE), tables.to(DEVICE), keys, values


def _attend_with_distance(q, keys, values, contexts, q_lens, n_heads, n_kv, hd, scale, distance, softcap):
    out = torch.zeros(q.shape[0], n_heads, hd, dtype=F64)
    group, row = n_heads // n_kv, 0
    for s, (c, n) in enumerate(zip(contexts, q_lens)):
        kv_of = torch.arange(n_heads) // group
        k, v = keys[s].double()[:, kv_of], values[s].double()[:, kv_of]
        scores = torch.einsum("ihd,jhd->hij", q[row:row + n].double().view(n, n_heads, hd), k) * scale
        if softcap:
            scores = softcap * torch.tanh(scores / softcap)
        if distance is not None:
            scores = scores - plain.distance_bias(c + n, distance[0].double(), distance[1].double())[:, c:]
        seen = torch.arange(c + n)[None, :] <= torch.arange(c, c + n)[:, None]
        out[row:row + n] = torch.einsum("hij,jhv->ihv", torch.softmax(scores.masked_fill(~seen, -math.inf), -1), v)
        row += n
    return out.view(q.shape[0], n_heads * hd)


@pytest.mark.parametrize("kernel, dtype, hd, group", [
    ("simt", torch.float32, 48, 3), ("simt", torch.float32, 128, 2), ("simt", torch.bfloat16, 32, 1),
    ("simt", torch.float32, 256, 20), ("mma", torch.bfloat16, 64, 4), ("mma", torch.bfloat16, 128, 2),
    ("mma", torch.bfloat16, 64, 1), ("mma", torch.bfloat16, 128, 8), ("tc", torch.bfloat16, 128, 2),
    ("tc", torch.bfloat16, 128, 4), ("tc", torch.bfloat16, 128, 1)])
@pytest.mark.parametrize("softcap", [None, 6.0])
def test_attention_kernels_with_a_distance_bias(kernel, dtype, hd, group, softcap):
    """Prompt portions and single tokens in one launch, shuffled pages, key splits. The last query of every sequence meets
    keys equal to itself nearby and far away: without the bias they would share the softmax, with it the heads whose
    numbers are large hardly see the far one."""
    n_kv, n_heads, page = 2, 2 * group, 16
    contexts, q_lens = [70, 5, 300, 0, 131], [1, 37, 1, 45, 2]
    if kernel == "tc":                     # prompt portions only
        contexts, q_lens = [70, 5, 130, 600, 0], [40, 37, 64, 150, 300]
    spikes = [(s, j) for s, (c, n) in enumerate(zip(contexts, q_lens)) for j in (0, c + n - 3) if 0 <= j < c + n - 1]
    q, cache, tables, keys, values = _paged_case(dtype, n_heads, n_kv, hd, page, contexts, q_lens, seed=hd + group,
                                                 spikes=spikes)
    batch = Batch(q_lens, contexts, [0] * len(q_lens))
    gen = torch.Generator().manual_seed(3)
    distance = torch.stack([torch.rand(n_heads, generator=gen) * 2.4 - 0.3, torch.rand(n_heads, generator=gen) * 0.7 + 0.02])
    distance[:, 0] = torch.tensor([2.5, 0.9])
    scale, n_tok, status = 8.0 / hd, batch.n, word()
    rounded_keys, rounded_values = [k.to(dtype).float() for k in keys], [v.to(dtype).float() for v in values]
    arguments = (q.cpu().float(), rounded_keys, rounded_values, contexts, q_lens, n_heads, n_kv, hd, scale)
    want = _attend_with_distance(*arguments, distance, softcap)
    meta = batch.cu_q, ints(contexts)
    for n_splits in (1, 3):
        # columns of wider rows: the kernels' output may lie beside another branch's
        wide = torch.zeros(n_tok, n_heads * hd + 64, dtype=dtype, device=DEVICE)
        out = wide[:, 32:32 + n_heads * hd]
        scratch = None
        if n_splits > 1:
            scratch = torch.empty(kernels.attention_scratch_bytes(n_tok, n_heads, hd, n_splits) // 4 + 4,
                                  dtype=torch.float32, device=DEVICE)
        common = dict(n_splits=n_splits, scratch=scratch, distance=distance.to(DEVICE), softcap=softcap)
        if kernel == "simt":
            kernels.paged_attention(q, q.stride(0), cache, tables, batch.tok_seq, batch.positions, n_tok, n_heads, n_kv, hd,
                                    None, scale, out, status, **common)
        elif kernel == "tc":
            _, tiles = kernels.attention_tile_lists([max(n, 17) for n in q_lens], group, True)
            kernels.paged_attention_tc(q, q.stride(0), cache, tables, *meta, ints(tiles), len(tiles) // 2, n_tok, n_heads,
                                       n_kv, hd, None, scale, out, status, **common)
        else:
            narrow, tiles = kernels.attention_tile_lists(q_lens, group, False)
            if n_splits > 1:        # key splits need a launch that covers every token: all tiles wide
                narrow, tiles = [], [x for s, n in enumerate(q_lens) for r in range(0, n * group, 64) for x in (s, r)]
            for some, is_narrow in ((narrow, True), (tiles, False)):
                if some:
                    kernels.paged_attention_mma(q, q.stride(0), cache, tables, *meta, ints(some), len(some) // 2, is_narrow,
                                                n_tok, n_heads, n_kv, hd, None, scale, out, status, **common)
        tol = 2e-5 if dtype == torch.float32 else 0.03
        got = out.double().cpu()
        assert torch.allclose(got, want, rtol=tol, atol=tol), (n_splits, (got - want).abs().max())
        assert float(wide[:, :32].abs().max()) == 0.0 and float(wide[:, 32 + n_heads * hd:].abs().max()) == 0.0
        assert int(status.item()) == 0
    without = _attend_with_distance(*arguments, None, softcap)
    assert float((without - want)[batch.cu[1] - 1, :hd].abs().max()) > 0.05          # head 0 of the first sequence
    # the far key matters too: a head that loses it for the bias's sake keeps it when the numbers are small
    assert float((without - want).abs().max()) > 0.3


CONV_CUTS = [[1, 1, 5, 1, 9], [17], [2, 2, 2, 2, 9], [0, 3, 1, 1, 12], [1, 0, 1, 0, 1]]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, kv, dim, vdim, taps, own", [(6, 3, 24, 40, 4, True), (4, 4, 64, 64, 2, True),
                                                             (2, 1, 20, 12, 5, True), (3, 3, 24, 40, 3, False),
                                                             (5, 1, 16, 16, 1, True), (8, 2, 128, 128, 4, False)])
def test_convolved_normalised_operands_and_their_memory(dtype, heads, kv, dim, vdim, taps, own):
    """Five sequences cut every way (shorter portions than the convolution is long among them): biases, convolution,
    the norm over all heads at once, the temperature, the pages and the memory, against the whole sequences."""
    gen = torch.Generator().manual_seed(dim + taps)
    page, hd = 8, -(-max(dim, vdim) // 16) * 16
    channels = heads * dim + (kv * (dim + vdim) if own else 0)
    coef, every, eps = 0.7, 5.0, 1e-4
    bias, conv = torch.randn(channels, generator=gen), torch.randn(channels, taps, generator=gen)
    wq, wk = torch.randn(heads * dim, generator=gen), torch.randn(kv * dim, generator=gen)
    sequences = [torch.randn(sum(c), channels, generator=gen) for c in CONV_CUTS]
    slots = [3, 0, 4, 1, 2]
    state = torch.zeros(5, taps - 1, channels, device=DEVICE) if taps > 1 else None
    cache = torch.zeros(20, 2, kv, page, hd, dtype=dtype, device=DEVICE) if own else None
    status = word()
    place, got_q = {}, [[] for _ in sequences]
    free = torch.randperm(20 * page, generator=gen).tolist()
    done = [0] * len(sequences)
    for live, batch in batches_of(CONV_CUTS, slots):
        proj = torch.cat([sequences[s][done[s]:done[s] + n] for s, n in zip(live, batch.q_lens)])
        wide = torch.cat([proj, torch.full((batch.n, 3), 9.0)], 1).to(DEVICE)
        where = [free.pop() for _ in range(batch.n)]
        for s, n, first in zip(live, batch.q_lens, batch.cu):
            for i in range(n):
                place[(s, done[s] + i)] = where[first + i]
        q_out = torch.empty(batch.n, heads * hd, dtype=dtype, device=DEVICE)
        kernels.conv_norm_kv_write(wide, bias.to(DEVICE), conv.t().contiguous().to(DEVICE), wq.to(DEVICE),
                                   wk.to(DEVICE) if own else None, eps, (coef, every), state, batch.positions,
                                   batch.tok_seq, batch.cu_q, batch.slots, ints(where) if own else None, cache, q_out,
                                   heads, kv, dim, vdim, status)
        if taps > 1 and max(batch.q_lens) > 1:
            kernels.conv_state_update(wide, bias.to(DEVICE), state.flatten(1), batch.cu_q, batch.slots, len(live), channels,
                                      taps)
        for i, s in enumerate(live):
            got_q[s].append(q_out[batch.rows(i)].double().cpu())
            done[s] += batch.q_lens[i]
    assert int(status.item()) == 0
    tol = 1e-4 if dtype == torch.float32 else 2e-2
    for s, sequence in enumerate(sequences):
        u = sequence.double() + bias.double()
        y = plain.causal_conv(u, conv.double())
        q = plain.unit(y[:, :heads * dim], eps) * wq.double()
        q = q * plain.temperature(torch.arange(len(u)), coef, every)[:, None]
        got = torch.cat(got_q[s]).view(len(u), heads, hd)
        assert torch.allclose(got[:, :, :dim], q.view(len(u), heads, dim), rtol=tol, atol=tol)
        assert hd == dim or float(got[:, :, dim:].abs().max()) == 0.0
        if taps > 1:
            kept = torch.cat([torch.zeros(taps - 1, channels, dtype=F64), u])[-(taps - 1):]
            assert torch.allclose(state[slots[s]].double().cpu(), kept, atol=1e-5)
        if own:
            k = (plain.unit(y[:, heads * dim:(heads + kv) * dim], eps) * wk.double()).view(-1, kv, dim)
            v = y[:, (heads + kv) * dim:].view(-1, kv, vdim)
            host = cache.double().cpu()
            for i in range(len(u)):
                pg, off = place[(s, i)] // page, place[(s, i)] % page
                assert torch.allclose(host[pg, 0, :, off, :dim], k[i], rtol=tol, atol=tol)
                assert torch.allclose(host[pg, 1].view(kv, hd, page)[:, :vdim, off], v[i], rtol=tol, atol=tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("channels, n, rank, taps", [(72, 13, 9, 3), (160, 16, 8, 4), (60, 1, 1, 1), (96, 40, 12, 2),
                                                     (33, 100, 5, 6), (256, 24, 16, 4), (130, 4, 128, 4), (64, 64, 20, 3)])
def test_selective_recurrence_kernels(dtype, channels, n, rank, taps):
    """Convolution with silu, then the recurrence: portions through the scan, steps of single tokens through the kernel that
    folds the step product in, from and to one state vector a slot; gates and inputs lie in columns of wider rows."""
    gen = torch.Generator().manual_seed(channels + n)
    conv, conv_bias = torch.randn(channels, taps, generator=gen), torch.randn(channels, generator=gen)
    dt_weight = torch.randn(channels, rank, generator=gen) * rank ** -0.5
    dt_bias = torch.rand(channels, generator=gen) * 5 - 4
    a = -torch.exp(torch.rand(channels, n, generator=gen) * 4 - 2)
    d, out_scale = torch.randn(channels, generator=gen), 1.3
    cuts = [[1, 1, 5, 1, 40], [37], [2, 2, 2, 1, 9], [0, 3, 1, 1, 70], [1, 1, 1, 1, 1]]
    slots = [3, 0, 4, 1, 2]
    x = [torch.randn(sum(c), channels, generator=gen) for c in cuts]
    z = [torch.randn(sum(c), channels, generator=gen) for c in cuts]
    # the low-rank rows are given, not computed, so that the two sides see the same ones
    low = [torch.randn(sum(c), rank + 2 * n, generator=gen) for c in cuts]
    dt_weight = dt_weight.to(dtype)
    state = torch.zeros(5, channels * (taps - 1 + n), device=DEVICE)
    recurrent = channels * (taps - 1)
    done, got = [0] * len(cuts), [[] for _ in cuts]
    a_log2 = (a.double() * math.log2(math.e)).float().to(DEVICE)
    constants = dt_bias.to(DEVICE), a_log2, d.to(DEVICE)
    got_u = [[] for _ in cuts]
    kinds = set()
    for live, batch in batches_of(cuts, slots):
        def rows(of):
            return torch.cat([of[s][done[s]:done[s] + k] for s, k in zip(live, batch.q_lens)]).to(DEVICE)
        wide = torch.cat([rows(x), rows(z)], 1)
        u = torch.empty(batch.n, channels, dtype=dtype, device=DEVICE)
        kernels.conv_silu(wide[:, :channels], conv.t().contiguous().to(DEVICE), conv_bias.to(DEVICE), state, batch.tok_seq,
                          batch.cu_q, batch.slots, u)
        single = max(batch.q_lens) == 1
        kinds.add(single)
        out = torch.zeros(batch.n, channels + 16, dtype=dtype, device=DEVICE)
        low_rows = rows(low)
        common = (wide[:, channels:], state, recurrent, batch.cu_q, batch.slots, len(live), out[:, 8:8 + channels], n, rank,
                  out_scale)
        if single:
            kernels.selective_step(u, low_rows, dt_weight.to(DEVICE), *constants, *common)
        else:
            kernels.conv_state_update(wide, None, state, batch.cu_q, batch.slots, len(live), channels, taps)
            raw = low_rows[:, :rank] @ dt_weight.float().to(DEVICE).T
            kernels.selective_scan(u, raw, low_rows, *constants, *common)
        assert float(out[:, :8].abs().max()) == 0.0 and float(out[:, 8 + channels:].abs().max()) == 0.0
        for i, s in enumerate(live):
            got[s].append(out[batch.rows(i), 8:8 + channels].double().cpu())
            got_u[s].append(u[batch.rows(i)].double().cpu())
            done[s] += batch.q_lens[i]
    assert kinds == {False} or kinds == {True, False}
    tol = 3e-4 if dtype == torch.float32 else 2e-2
    for s in range(len(cuts)):
        u = plain.silu(plain.causal_conv(x[s].double(), conv.double(), conv_bias.double()))
        mine = torch.cat(got_u[s])
        assert torch.allclose(mine, u, rtol=tol, atol=tol)
        dt = torch.nn.functional.softplus(low[s][:, :rank].double() @ dt_weight.double().T + dt_bias.double())
        # the recurrence on the kernel's own (rounded) inputs: what is left is the recurrence's error alone
        y = plain.selective_scan(mine, dt, low[s][:, rank:rank + n].double(), low[s][:, rank + n:].double(), a.double(),
                                 d.double())
        want = y * plain.silu(z[s].double()) * out_scale
        error = (torch.cat(got[s]) - want).abs()
        assert float((error / (want.abs() + 1.0)).max()) < (2e-4 if dtype == torch.float32 else 1e-2)
        if taps > 1:
            kept = torch.cat([torch.zeros(taps - 1, channels, dtype=F64), x[s].double()])[-(taps - 1):]
            assert torch.allclose(state[slots[s], :recurrent].view(taps - 1, channels).double().cpu(), kept, atol=1e-6)


def test_single_token_steps_of_the_selective_recurrence_alone():
    """Every step is the folded kernel: 60 tokens of three sequences, one of them with the fixed-size batch's padding
    rows behind it, against the scan over whole portions."""
    gen = torch.Generator().manual_seed(2)
    channels, n, rank = 40, 6, 8
    w, a_log2 = torch.randn(channels, rank, generator=gen), -torch.rand(channels, n, generator=gen)
    dt_bias, d = torch.randn(channels, generator=gen) - 2, torch.randn(channels, generator=gen)
    u, z, low = (torch.randn(3, 60, k, generator=gen).to(DEVICE) for k in (channels, channels, rank + 2 * n))
    w, a_log2, dt_bias, d = (t.to(DEVICE) for t in (w, a_log2, dt_bias, d))
    state = torch.zeros(3, channels * n, device=DEVICE)
    outs = []
    for t in range(60):
        out = torch.full((5, channels), 3.0, device=DEVICE)
        pad = lambda rows: torch.cat([rows, torch.full((2, rows.shape[1]), float("nan"), device=DEVICE)])
        kernels.selective_step(pad(u[:, t]), pad(low[:, t]), w, dt_bias, a_log2, d, pad(z[:, t]), state, 0,
                               ints([0, 1, 2, 3, 3, 3]), ints([2, 0, 1, 0, 0]), 5, out, n, rank)
        assert float(out[3:].abs().max()) == 0.0                        # padding rows: zeros, and no state moved
        outs.append(out[:3])
    whole = torch.zeros(3, channels * n, device=DEVICE)
    flat = [t.reshape(180, -1).contiguous() for t in (u, low, z)]
    out = torch.empty(180, channels, device=DEVICE)
    kernels.selective_scan(flat[0], flat[1][:, :rank] @ w.T, flat[1], dt_bias, a_log2, d, flat[2], whole, 0,
                           ints([0, 60, 120, 180]), ints([2, 0, 1]), 3, out, n, rank)
    assert torch.allclose(torch.stack(outs, 1).reshape(180, channels), out, rtol=1e-4, atol=1e-4)
    assert torch.allclose(state, whole, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("heads, dim, vdim, rot", [(3, 20, 28, 12), (2, 64, 128, 64), (4, 128, 64, 128), (1, 96, 24, 2),
                                                   (9, 8, 8, 0), (2, 200, 40, 100), (1, 256, 16, 256)])
def test_retention_kernels(heads, dim, vdim, rot):
    """Constant decays (zero and one among them), q and k rotated by a pass of their own or on their way in, portions and
    single tokens from and to a slot."""
    gen = torch.Generator().manual_seed(dim)
    decay = torch.tensor([0.0, 1.0, 0.97, 0.5, 0.9, 0.999, 0.2, 0.8, 0.99])[-heads:] if heads < 9 else \
        torch.tensor([0.0, 1.0, 0.97, 0.5, 0.9, 0.999, 0.2, 0.8, 0.99])
    cuts, slots = [[1, 1, 5, 1, 40], [37], [2, 2, 2, 1, 9], [0, 3, 1, 1, 20]], [3, 0, 2, 1]
    rows_of = [torch.randn(sum(c), heads * (2 * dim + vdim) + 4, generator=gen) for c in cuts]
    spec = turned(rot, 400.0) if rot else None
    freq = plain.frequencies(rot, 400.0)[0].float().to(DEVICE) if rot else None
    for in_kernel in (False, True):
        state = torch.zeros(4, heads, dim, vdim, device=DEVICE)
        done, got = [0] * len(cuts), [[] for _ in cuts]
        for live, batch in batches_of(cuts, slots):
            proj = torch.cat([rows_of[s][done[s]:done[s] + k] for s, k in zip(live, batch.q_lens)]).to(DEVICE)
            rotation = {}
            if rot and in_kernel:
                rotation = dict(positions=batch.positions, freq=freq, rot=rot)
            elif rot:
                kernels.rotate_heads(proj, 0, 2 * heads, dim, rot, batch.positions, freq)
            out = torch.empty(batch.n, heads * vdim, device=DEVICE)
            kernels.retention_scan(proj, 0, heads * dim, 2 * heads * dim, decay.to(DEVICE), dim ** -0.5, state, batch.cu_q,
                                   batch.slots, len(live), out, heads, dim, vdim, **rotation)
            for i, s in enumerate(live):
                got[s].append(out[batch.rows(i)].double().cpu())
                done[s] += batch.q_lens[i]
        for s, rows in enumerate(rows_of):
            p64, pos = rows.double(), torch.arange(len(rows))
            q = plain.rotate(p64[:, :heads * dim].view(-1, heads, dim), pos, spec)
            k = plain.rotate(p64[:, heads * dim:2 * heads * dim].view(-1, heads, dim), pos, spec) * dim ** -0.5
            v = p64[:, 2 * heads * dim:2 * heads * dim + heads * vdim].view(-1, heads, vdim)
            want = plain.linear_recurrence(q, k, v, decay.double()).reshape(len(rows), -1)
            mine = torch.cat(got[s])
            assert torch.allclose(mine, want, rtol=1e-4, atol=1e-4 * float(want.abs().max())), (in_kernel, s)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, dim, vdim, rot", [(3, 20, 28, 12), (2, 64, 128, 64), (4, 128, 64, 128), (1, 96, 24, 2),
                                                   (5, 13, 7, 6), (2, 128, 128, 0), (3, 64, 64, 32)])
def test_retention_in_chunks(dtype, heads, dim, vdim, rot):
    """Long and short portions in one launch (whole chunks, one token more and less, single tokens), the norm and the gate
    in the same kernels, from and to the slots, against the plain recurrence over the whole sequences."""
    gen = torch.Generator().manual_seed(dim + rot)
    decay = torch.tensor([0.0, 1.0, 0.97, 0.5, 0.9])[-heads:]
    cuts, slots = [[64, 1, 130], [63, 65, 64], [200, 128, 1], [0, 1, 7]], [3, 0, 2, 1]
    width = heads * (2 * dim + 2 * vdim)
    rows_of = [torch.randn(sum(c), width, generator=gen) for c in cuts]
    spec, freq = (turned(rot, 400.0), plain.frequencies(rot, 400.0)[0].float().to(DEVICE)) if rot else (None, None)
    state = torch.zeros(4, heads, dim, vdim, device=DEVICE)
    size, eps = kernels.retention_chunk_tokens(), 1e-4
    done, got = [0] * len(cuts), [[] for _ in cuts]
    for live, batch in batches_of(cuts, slots):
        rows = torch.cat([rows_of[s][done[s]:done[s] + k] for s, k in zip(live, batch.q_lens)])
        proj = torch.cat([rows, torch.full((batch.n, 4), 9.0)], 1).to(DEVICE)
        chunks, first = kernels.scan_chunk_lists(batch.q_lens, size)
        wide = torch.zeros(batch.n, heads * vdim + 16, dtype=dtype, device=DEVICE)
        rotation = dict(positions=batch.positions, freq=freq, rot=rot) if rot else {}
        kernels.retention_chunked(proj, 0, heads * dim, 2 * heads * dim, heads * (2 * dim + vdim), decay.to(DEVICE),
                                  dim ** -0.5, eps, state, batch.cu_q, batch.slots, len(live), ints(chunks), ints(first),
                                  len(chunks) // 2, wide[:, 8:8 + heads * vdim], heads, dim, vdim, **rotation)
        assert float(wide[:, :8].abs().max()) == 0.0 and float(wide[:, 8 + heads * vdim:].abs().max()) == 0.0
        for i, s in enumerate(live):
            got[s].append(wide[batch.rows(i), 8:8 + heads * vdim].double().cpu())
            done[s] += batch.q_lens[i]
    tol = 2e-4 if dtype == torch.float32 else 1e-2
    for s, rows in enumerate(rows_of):
        p64, pos = rows.double(), torch.arange(len(rows))
        q = plain.rotate(p64[:, :heads * dim].view(-1, heads, dim), pos, spec)
        k = plain.rotate(p64[:, heads * dim:2 * heads * dim].view(-1, heads, dim), pos, spec) * dim ** -0.5
        v = p64[:, 2 * heads * dim:heads * (2 * dim + vdim)].view(-1, heads, vdim)
        o = plain.linear_recurrence(q, k, v, decay.double())
        want = plain.unit(o, eps).reshape(len(rows), -1) * plain.silu(p64[:, heads * (2 * dim + vdim):])
        mine = torch.cat(got[s])
        # a head whose o is nearly zero for all its values is ill-conditioned under its own norm: rounding shows there
        hard = (o.pow(2).mean(-1).sqrt() < 1e-2)[:, :, None].expand(-1, -1, vdim).reshape(len(rows), -1)
        error = ((mine - want).abs() / (want.abs() + 1.0)).masked_fill(hard, 0.0)
        assert float(error.max()) < tol, (s, float(error.max()))
        assert float(hard.double().mean()) < 0.05


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("channels, n, rank, size", [(72, 13, 9, 32), (160, 16, 8, 128), (33, 100, 5, 7), (40, 1, 3, 50)])
def test_selective_recurrence_in_chunks(dtype, channels, n, rank, size):
    """The three-launch form beside the walk it replaces, over several steps and unequal portions, from and to the slots."""
    gen = torch.Generator().manual_seed(channels * n)
    dt_bias, d = torch.rand(channels, generator=gen) * 5 - 4, torch.randn(channels, generator=gen)
    a_log2 = -torch.exp(torch.rand(channels, n, generator=gen) * 4 - 2)
    constants = dt_bias.to(DEVICE), a_log2.to(DEVICE), d.to(DEVICE)
    state = torch.randn(4, 24 + channels * n, generator=gen).to(DEVICE)
    whole = state.clone()
    for q_lens in ([300, 1, size, 64], [2, size + 1, 90], [1, 1, 1, 3 * size]):
        batch = Batch(q_lens, [0] * len(q_lens), [2, 0, 3, 1][:len(q_lens)])
        u, z = (torch.randn(batch.n, channels, generator=gen).to(dtype).to(DEVICE) for _ in range(2))
        raw, low = torch.randn(batch.n, channels, generator=gen).to(DEVICE), torch.randn(batch.n, rank + 2 * n, generator=gen).to(DEVICE)
        chunks, first = kernels.scan_chunk_lists(q_lens, size)
        outs = []
        for kept, chunked in ((whole, None), (state, (ints(chunks), ints(first), len(chunks) // 2, size))):
            out = torch.empty(batch.n, channels, dtype=dtype, device=DEVICE)
            kernels.selective_scan(u, raw, low, *constants, z, kept, 24, batch.cu_q, batch.slots, len(q_lens), out, n, rank,
                                   0.7, chunked=chunked)
            outs.append(out.double())
        tol = 1e-4 if dtype == torch.float32 else 1e-2
        assert torch.allclose(*outs, rtol=tol, atol=tol) and torch.allclose(state, whole, rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, vdim", [(3, 28), (2, 128), (1, 300)])
def test_heads_normalised_without_a_weight_and_gated(dtype, heads, vdim):
    gen = torch.Generator().manual_seed(vdim)
    o, gate = torch.randn(21, heads * vdim, generator=gen) * 5, torch.randn(21, heads * vdim + 7, generator=gen)
    out = torch.empty(21, heads * vdim, dtype=dtype, device=DEVICE)
    kernels.gla_norm_gate(o.to(DEVICE), gate.to(DEVICE)[:, 3:3 + heads * vdim], None, 1e-3, out, heads, vdim)
    want = plain.unit(o.double().view(21, heads, vdim), 1e-3).reshape(21, -1) * plain.silu(gate.double()[:, 3:3 + heads * vdim])
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(out.double().cpu(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts, top", [(5, 2), (3, 1), (16, 2), (40, 5), (2, 2), (1, 1), (70, 40)])
def test_router_kernel_leaves_the_scores_as_weights(dtype, experts, top):
    gen = torch.Generator().manual_seed(experts * 7 + top)
    n, width = 50, 72
    h, router = torch.randn(n, width, generator=gen).to(dtype), torch.randn(experts, width, generator=gen) * 0.3
    chosen, place = ints([0] * n * top), ints([0] * n * top)
    counts, weights = ints([0] * experts), torch.empty(n * top, dtype=torch.float32, device=DEVICE)
    kernels.moe_route(h.to(DEVICE), router.to(DEVICE), top, 1, 1, 1.0, chosen, weights, counts, place, normalize=False)
    want, scores, margin = plain.route(h.double(), router.double(), top)
    got_ids, got = chosen.view(n, top).cpu().long(), weights.view(n, top).cpu().double()
    clear = margin > 1e-3
    assert torch.equal(torch.sort(got_ids[clear], 1).values, torch.sort(want[clear], 1).values)
    own = torch.sigmoid(torch.gather(h.double() @ router.double().T, 1, got_ids))
    assert torch.allclose(got, own, atol=1e-5)
    assert int(counts.sum()) == n * top
    assert top == 1 or float((got.sum(1) - 1).abs().max()) > 0.05       # they are not shares of one


def test_a_router_that_sees_no_numbers_stays_inside_its_arrays():
    """Rows of a fixed-size batch beyond its requests hold anything; their choice is an expert that exists."""
    h = torch.full((3, 40), float("nan"), device=DEVICE)
    router = torch.randn(6, 40, device=DEVICE)
    chosen, place, counts = ints([-1] * 6), ints([0] * 6), ints([0] * 6)
    weights = torch.empty(6, dtype=torch.float32, device=DEVICE)
    for groups, keep in ((1, 1), (3, 2)):
        counts.zero_()
        kernels.moe_route(h, router, 2, groups, keep, 1.0, chosen, weights, counts, place)
        assert int(chosen.min()) >= 0 and int(chosen.max()) < 6 and int(counts.sum()) == 6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_activation_of_weighted_rows(dtype):
    gen = torch.Generator().manual_seed(4)
    for ff in (40, 37):
        gu = torch.randn(30, 2 * ff, generator=gen).to(dtype)
        weight, order = torch.rand(30, generator=gen), torch.randperm(30, generator=gen).to(torch.int32)
        out = torch.empty(30, ff, dtype=dtype, device=DEVICE)
        kernels.glu(gu.to(DEVICE), out, "silu", pair_weight=weight.to(DEVICE), order=order.to(DEVICE))
        scaled = gu.double() * weight.double()[order.long()][:, None]
        want = plain.silu(scaled[:, :ff]) * scaled[:, ff:]
        tol = 1e-5 if dtype == torch.float32 else 1e-2
        assert torch.allclose(out.double().cpu(), want, rtol=tol, atol=tol)


# ---------------------------------------------------------------------- single layers
BASE = retention(2, 16, 16, [0.9, 0.99], (8, 100.0))
LAYERS_ALONE = {
    "convolved": conv_attention(6, 3, 24, 40, 0.3, 4, (0.4, 19)),
    "convolved_tensor_core_head": conv_attention(4, 1, 64, 64, 0.2, 3, (0.5, 32)),
    "convolved_head_128": conv_attention(2, 2, 128, 128, 0.12, 2, (0.2, 9)),
    "convolved_keys_wider_than_values": conv_attention(2, 1, 64, 32, 0.2, 4, (0.5, 16)),
    "one_tap_one_period": conv_attention(5, 1, 20, 12, 0.3, 1, (1.1, 1)),
    "seven_taps": conv_attention(2, 1, 16, 16, 0.3, 7, (0.0, 3)),
    "parallel": parallel((4, 1, 40, 0.25, 4.0, turned(24, 5000.0, (4.0, 64, 8.0, 1.0))), (72, 13, 9, 3), 0.7, 1.4),
    "parallel_tensor_core_head": parallel((4, 2, 64, 0.2, 2.0, turned(64, 100.0, (8.0, 64, 16.0, 2.0))), (64, 16, 8, 4), 1.2,
                                          0.9),
    "parallel_left_only_in_weight": parallel((2, 2, 16, 0.4, 20.0, turned(16, 300.0)), (40, 8, 4, 2), 2.0, 0.01),
    "parallel_right_only_in_weight": parallel((2, 2, 16, 0.4, 20.0, turned(8, 300.0)), (200, 20, 7, 4), 0.01, 2.0),
    "parallel_unrotated_one_state": parallel((5, 5, 12, 0.4, 1.5, None), (60, 1, 1, 1), 1.3, 0.9),
    "parallel_many_states": parallel((2, 1, 32, 0.3, 5.0, turned(2, 50.0)), (48, 128, 33, 5), -0.8, 1.0),
    "retention": retention(3, 20, 28, [0.9, 0.99, 0.5], (12, 900.0)),
    "retention_without_rotation_or_memory": retention(2, 16, 40, [0.0, 1.0], None),
    "retention_wide": retention(2, 64, 128, [0.97, 0.999], (64, 10000.0)),
    "retention_wider": retention(1, 144, 48, [0.995], (144, 10000.0)),
    "dense_feed_forward": dict(BASE, mlp=dense(72)),
    "experts_top_two": dict(BASE, mlp=moe(40, 5, 2)),
    "experts_top_one": dict(BASE, mlp=moe(24, 3, 1)),
    "all_experts_chosen": dict(BASE, mlp=moe(32, 3, 3)),
    "one_expert": dict(BASE, mlp=moe(36, 1, 1)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(LAYERS_ALONE))
def test_one_layer_models(name, dtype):
    """Whole, then one token at a time, then in portions: the three must agree with the plain model."""
    raw = single_layer(LAYERS_ALONE[name])
    run = Run(raw, draw(raw, seed=len(name), router_gain=3.0), dtype, max_tokens=4 * 256)
    tokens = ids(75, raw["vocab"], seed=1)
    run.feed("whole", tokens, [75])
    run.check("whole", tokens)
    run.feed("single", tokens[:60], [])
    run.check("single", tokens[:60])
    run.feed("cut", tokens, cycle)
    run.check("cut", tokens)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_that_share_one_cache(dtype):
    """Two layers read a third one's keys and values with queries, convolutions, temperatures and biases of their own;
    the source's cache is written once, and one more attention layer keeps its own."""
    raw = model(64, 120, 1.5, [conv_attention(4, 2, 24, 32, 0.3, 3, (0.4, 11), mlp=dense(48)),
                               conv_attention(4, 2, 24, 32, 0.3, 2, (0.8, 5)),
                               conv_attention(2, 2, 24, 32, 0.25, 5, (0.1, 40), kv_from=0),
                               conv_attention(4, 2, 24, 32, 0.35, 4, (0.6, 3), kv_from=0)])
    run = Run(raw, draw(raw, seed=31), dtype, max_tokens=4 * 128)
    assert [len(g.entries) for g in run.replayer.model.cache_plan.groups] == [2]
    tokens = ids(90, raw["vocab"], seed=6)
    run.feed("whole", tokens, [90])
    run.check("whole", tokens)
    run.feed("cut", tokens, cycle)
    run.check("cut", tokens)
    run.feed("decoded", tokens, [20])
    run.check("decoded", tokens)


# ---------------------------------------------------------------------- planted tokens
def _align_convolved(raw, tensors):
    """The last query (token 89) points at the key of token 88 in every head; identity convolutions, no biases."""
    m = raw["layers"][0]["mixer"]
    eps, g = raw["norm"]["eps"], tensors["l0.norm1"]
    h88, h89 = (plain.unit(tensors["embed"][t] * raw["embedding"]["scale"], eps) * g for t in (88, 89))
    for name in ("q", "k", "v"):
        tensors[f"l0.mix.{name}.conv"].zero_()
        tensors[f"l0.mix.{name}.conv"][:, -1] = 1.0
        tensors[f"l0.mix.{name}.b"].zero_()
    k88 = (tensors["l0.mix.k"] @ h88).view(m["kv_heads"], m["dim"])
    group = m["heads"] // m["kv_heads"]
    target = torch.cat([k88[h // group] for h in range(m["heads"])])
    tensors["l0.mix.q"] = (torch.outer(target, h89) / (h89 @ h89)).contiguous()
    tensors["l0.mix.q.norm"], tensors["l0.mix.k.norm"] = torch.ones(m["heads"] * m["dim"]), torch.ones(m["kv_heads"] * m["dim"])
    tensors["l0.mix.r1"].fill_(0.05)


def _align_capped(raw, tensors):
    m = raw["layers"][0]["mixer"]["left"]
    eps, g = raw["norm"]["eps"], tensors["l0.norm1"]
    h88, h89 = (plain.unit(tensors["embed"][t] * raw["embedding"]["scale"], eps) * g for t in (88, 89))
    k88 = (tensors["l0.mix.left.k"] @ h88).view(m["kv_heads"], m["dim"])
    group = m["heads"] // m["kv_heads"]
    target = torch.cat([k88[h // group] for h in range(m["heads"])])
    tensors["l0.mix.left.q"] = (torch.outer(target, h89) / (h89 @ h89)).contiguous()
    tensors["l0.mix.left.q.norm"], tensors["l0.mix.left.k.norm"] = torch.ones(m["dim"]), torch.ones(m["dim"])


PLANTED = {
    "convolved": (conv_attention(2, 1, 32, 32, 0.5, 3, (0.3, 100)), _align_convolved, 430),
    "convolved_tensor_core_head": (conv_attention(4, 2, 64, 64, 0.35, 4, (0.2, 64)), _align_convolved, 430),
    "capped": (parallel((2, 1, 32, 0.5, 30.0, None), (32, 8, 4, 3), 1.5, 0.3), _align_capped, 430),
    "capped_tensor_core_head": (parallel((4, 2, 128, 0.15, 25.0, None), (32, 8, 4, 3), 1.5, 0.3), _align_capped, 200),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [0, 50])
@pytest.mark.parametrize("name", list(PLANTED))
def test_one_token_decides_wherever_it_stands(name, decode, dtype):
    """The asked-for token among hundreds: the sequence's first ones, both sides of page borders, the place just before
    the last; in a whole prompt and with the tail decoded token by token."""
    layer, align, length = PLANTED[name]
    raw = single_layer(layer, vocab=90)
    tensors = draw(raw, seed=9)
    align(raw, tensors)
    tokens = [t % 86 for t in ids(length, 86, seed=2)]
    tokens[-1] = 89
    run = Run(raw, tensors, dtype, max_tokens=2 * (length + 64))
    last, base = length - 1, None
    for turn, place in enumerate([None, 0, 1, 15, 16, 17, 31, 32, length - 51, length - 50, length - 49, last - 1]):
        planted = list(tokens)
        if place is not None:
            planted[place] = 88
        run.feed(f"p{turn}", planted, [length - decode] if decode else [length])
        run.check(f"p{turn}", planted)
        row = run.logits[(f"p{turn}", last)]
        if place is None:
            base = row
        else:
            assert float(np.abs(row - base).max()) > 0.3, place


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer", [retention(2, 16, 16, [1.0, 0.999], (8, 100.0)),
                                   parallel((2, 2, 16, 0.1, 5.0, None), (48, 8, 4, 3), 0.02, 1.5)], ids=["retention", "scan"])
def test_an_early_token_stays_in_the_state(layer, dtype):
    """One changed token at the start moves the last logits through the state alone (no layer looks back otherwise), in
    every cut; a state that a portion drops, or a slot that keeps what it held, shows."""
    raw = single_layer(layer, vocab=90)
    tensors = draw(raw, seed=3)
    if layer["type"] == "parallel":
        tensors["l0.mix.right.A_log"].fill_(-6.0)                 # hardly any decay
        tensors["l0.mix.right.dt.b"].fill_(-1.0)
    tokens = [t % 80 for t in ids(150, 90, seed=4)]
    other = list(tokens)
    other[2] = 85
    run = Run(raw, tensors, dtype, max_tokens=2 * 192, max_requests=2)
    for turn, sizes in enumerate(([150], [], cycle, lambda turn: 2)):
        run.feed(f"a{turn}", tokens, sizes)
        run.check(f"a{turn}", tokens)
        run.feed(f"b{turn}", other, sizes)
        run.check(f"b{turn}", other)
        moved = np.abs(run.logits[(f"a{turn}", 149)] - run.logits[(f"b{turn}", 149)]).max()
        assert moved > (1e-3 if dtype == "float32" else 5e-3), moved


# ---------------------------------------------------------------------- whole models
@pytest.fixture(scope="module", params=[(n, d) for n in ("A", "B", "C", "D") for d in ("float32", "bfloat16")],
                ids=lambda p: f"{p[0]}-{p[1]}")
def run(request):
    name, dtype = request.param
    raw = MODELS[name]
    # four live requests of at most 128 tokens: pages and slots must come back to be used again
    made = Run(raw, draw(raw, seed=11 + ord(name), router_gain=2.0), dtype, max_tokens=4 * 128, max_requests=4)
    yield made


LENGTHS = [1, 2, 17, 40, 65, 100, 128]


def prompts_of(run):
    # a sequence's first token gives a retention head (q . k) v over its root mean square: where q . k is near zero, 16-bit
    # rounding decides the head's sign (these first tokens have none so near)
    return {f"r{n}": ids(n, run.raw["vocab"], seed=300 + n) for n in LENGTHS}


def test_whole_prompts(run):
    for request, tokens in prompts_of(run).items():
        run.feed(request + "w", tokens, [len(tokens)])
        run.check(request + "w", tokens)


def test_prefill_then_token_by_token(run):
    for request, tokens in prompts_of(run).items():
        head = max(len(tokens) - 70, 0)
        run.feed(request + "d", tokens, [head] if head else [])
        run.check(request + "d", tokens)


def test_portions_down_to_two_tokens(run):
    for shift, (request, tokens) in enumerate(prompts_of(run).items()):
        run.feed(request + "c", tokens, lambda turn: cycle(turn + shift))
        run.check(request + "c", tokens)
    tokens = prompts_of(run)["r65"]
    run.feed("pairs", tokens, lambda turn: 2)
    run.check("pairs", tokens)


def test_unequal_requests_batched_with_pages_and_slots_used_again(run):
    prompts = prompts_of(run)
    waiting = [(f"{request}m{again}", tokens) for again in range(2) for request, tokens in prompts.items()]
    tokens_of = dict(waiting)
    live: dict[str, int] = {}
    cache = run.replayer.core.cache
    turn = 0
    while waiting or live:
        while waiting and len(live) < 4:
            live[waiting.pop(0)[0]] = 0
        portions, ended = [], []
        for place, (request, done) in enumerate(list(live.items())):
            tokens = tokens_of[request]
            if (turn + place) % 5 == 4 and len(live) > 1:
                continue                                          # sits this step out
            remaining = len(tokens) - done
            size = 1 if (turn + place) % 3 == 0 else min(cycle(turn + place), remaining)
            portions.append((request, tokens[done:done + size]))
            live[request] = done + size
            if done + size == len(tokens):
                ended.append(request)
        turn += 1
        if portions:
            run.step(portions, end=ended)
        for request in ended:
            del live[request]
    for request, tokens in tokens_of.items():
        run.check(request, tokens)
    assert cache.pages_reused > 0 or not cache.rules
    assert len(set(run.slots_seen[r] for r in tokens_of)) <= 4 < len(tokens_of)


def test_long_decoding(run):
    """Hundreds of single-token steps (the captured decode step replayed) after a short prompt, two requests
    side by side, one of them starting later."""
    a = ids(260, run.raw["vocab"], seed=7)
    b = ids(150, run.raw["vocab"], seed=8)
    run.step([("la", a[:6])])
    for i in range(6, len(a)):
        portions = [("la", a[i:i + 1])]
        j = i - 100
        if 0 <= j < len(b):
            portions.append(("lb", b[j:j + 1]))
        ended = [name for name, k, seq in (("la", i, a), ("lb", j, b)) if k == len(seq) - 1]
        run.step(portions, end=ended)
    run.check("la", a)
    run.check("lb", b)


def test_routing_was_mostly_clear():
    assert Run.clear >= 2 * Run.unclear, "most choices must have been clear enough to be compared"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts(dtype):
    """A prompt long enough for the prompt-sized product kernels, many attention tiles and many rounds of the recurrences:
    whole, then in uneven portions with the tail decoded."""
    raw, length = MODELS["L"], 1100
    run = Run(raw, draw(raw, seed=21, router_gain=2.0), dtype, max_tokens=2 * (length + 64))
    tokens = ids(length, raw["vocab"], seed=5)
    run.feed("whole", tokens, [length])
    run.check("whole", tokens)
    run.feed("cut", tokens, [length // 3 + 1, 2, length // 2, length - 40 - (length // 3 + 3 + length // 2)])
    run.check("cut", tokens)


def test_greedy_generation_through_the_engine_entry_point():
    from matricxon_b200 import ChatEngine, GenerationRequest, SamplingConfig

    for name in ("A", "D"):
        raw = MODELS[name]
        tensors = draw(raw, seed=11)
        model_ = model_from_tensors(config_from_dict(copy.deepcopy(raw)), tensors, dtype="float32", device=DEVICE)
        # a pool that the five requests do not fit together: some give way, and their state is computed again
        engine = ChatEngine(model_, max_cache_tokens=2 * 96, max_active=3, max_batched_tokens=64, prefill_chunk=24,
                            max_model_len=128)
        prompts = [ids(n, raw["vocab"], seed=40 + n) for n in (5, 33, 70, 12, 50)]
        sampling = SamplingConfig(temperature=0.0, repeat_penalty=1.0, num_predict=24, num_ctx=128, seed=0)
        results = engine.generate_batch([GenerationRequest(input_ids=p, sampling=sampling) for p in prompts])
        weights = doubles(tensors)
        for prompt, result in zip(prompts, results):
            assert result.finish_reason == "length" and len(result.token_ids) == 24
            logits = plain.forward(raw, weights, prompt + result.token_ids[:-1]).numpy()
            for k, token in enumerate(result.token_ids):
                row = logits[len(prompt) - 1 + k]
                assert row[token] >= row.max() - 2e-3, (name, k, token, int(row.argmax()))


def test_trace_program_and_command_line(tmp_path):
    """The replay program itself on a model folder (bfloat16 file, both dtypes), and the generation command."""
    from matricxon_b200.weights.safetensors_io import write_safetensors

    raw = copy.deepcopy(MODELS["C"])
    tensors = draw(raw, seed=12, store_dtype=torch.bfloat16, router_gain=3.0)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(raw))
    write_safetensors(folder / "model.safetensors", tensors.items())
    tokens = ids(50, raw["vocab"], seed=3)
    want = plain.forward(raw, {k: v.double() for k, v in tensors.items()}, tokens).numpy()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:31], "want": [0, 30]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[31:33], "want": []},
                                     {"id": "b", "tokens": tokens[:9], "want": [8]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[33:], "want": [16]}], "end": ["a"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        done = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype",
                               dtype, "--out", str(out), "--max-tokens", "128"],
                              input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                              timeout=600)
        assert done.returncode == 0, done.stderr[-2000:]
        assert [line for line in done.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
        got = {s: np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, raw["vocab"]) for s in (0, 1, 2)}
        limit = limit_for(dtype, want) * (1 if dtype == "float32" else 2)
        assert np.abs(got[0] - want[[0, 30]]).max() <= limit
        assert np.abs(got[1] - want[[8]]).max() <= limit
        assert np.abs(got[2] - want[[49]]).max() <= limit
    config_path = tmp_path / "config.json"
    config_path.write_text(json.dumps(MODELS["B"]))
    done = subprocess.run([sys.executable, "-m", "matricxon_b200.generate", "--random-config", str(config_path),
                           "--prompt-len", "20", "--num-predict", "12"], capture_output=True, text=True,
                          timeout=600, cwd=str(ROOT))
    assert done.returncode == 0, done.stderr[-2000:]
    assert "finish_reason:  length" in done.stdout and "Seredra" in done.stdout
