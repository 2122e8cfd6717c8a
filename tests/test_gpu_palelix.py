"""Palelix through the engine against the plain implementation (tests/plain_palelix.py): every mechanism alone, then whole
models cut and batched every way, in float32 and bfloat16, with pools so small that pages and slots are used again. Sizes,
orders and constants are the tests' own."""

import copy
import json
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_palelix as plain
from matricxon_b200.engine.core import model_from_tensors
from matricxon_b200.engine.replay import TraceReplayer
from matricxon_b200.ops import kernels
from matricxon_b200.ops.linear import PendingSum
from palelix_configs import MODELS, config_of, delta, dense, draw, ids, lightning, model, moe, parallel, single_layer
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
        model = model_from_tensors(config_of(raw, tensors), self.weights, dtype=dtype, device=DEVICE, page_size=page_size)
        self.replayer = TraceReplayer(None, dtype, max_tokens, page_size=page_size, device=DEVICE,
                                      max_requests=max_requests, model=model, poison_cache=True)
        self.routed = plain.routed_runs(raw)
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
            forced = {number: [self.choices[(request, i)][k] for i in range(len(tokens))]
                      for k, number in enumerate(self.routed)}
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
CUTS = [[1, 1, 5, 1, 40], [37], [2, 2, 2, 1, 9], [0, 3, 1, 1, 20], [16, 8, 24, 7, 17]]
SLOTS = [3, 0, 4, 1, 2]


def delta_rows(s, heads, kv, dim, vdim, channel, gen):
    """(qkv with unit q and k, beta, g) of sequence s; decays from nearly zero to one, writes from none to full."""
    n = sum(CUTS[s])
    q, k = (plain.over_length(torch.randn(n, kv, dim, generator=gen, dtype=F64)) for _ in range(2))
    k[n // 2] = k[0]                                                  # a key that comes back
    qkv = torch.cat([(q * dim ** -0.5).reshape(n, -1), k.reshape(n, -1), torch.randn(n, heads * vdim, generator=gen, dtype=F64)], 1)
    beta = torch.rand(n, heads, generator=gen, dtype=F64)
    beta[::5] = 1.0
    g = torch.rand((n, heads, dim) if channel else (n, heads), generator=gen, dtype=F64) ** 0.2
    g[::7] = 1e-20
    g[3::7] = 1.0
    return qkv.float(), beta.float(), g.float()


def plain_delta(qkv, beta, g, heads, kv, dim, vdim):
    n, of = len(qkv), torch.arange(heads) // (heads // kv)
    q, k = (qkv.double()[:, i * kv * dim:(i + 1) * kv * dim].view(n, kv, dim)[:, of] for i in range(2))
    g = g.double() if g.dim() == 3 else g.double()[:, :, None].expand(-1, -1, dim)
    return plain.delta_rule(q, k, qkv.double()[:, 2 * kv * dim:].view(n, heads, vdim), g, beta.double())


@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("heads, kv, dim, vdim", [(3, 3, 20, 28), (4, 2, 64, 128), (2, 1, 128, 64), (6, 2, 12, 20), (1, 1, 96, 24),
                                                  (2, 2, 160, 40), (4, 1, 256, 16), (5, 5, 8, 8), (16, 4, 128, 128), (8, 8, 256, 64)])
def test_delta_rule_kernels(heads, kv, dim, vdim, channel):
    """Portions through the groups of eight (whole groups, one token more and less, single tokens among them), from and to
    slots, then single tokens through the step kernel, which ends in norm, weight and gate."""
    gen = torch.Generator().manual_seed(dim + heads)
    rows = [delta_rows(s, heads, kv, dim, vdim, channel, gen) for s in range(len(CUTS))]
    want = [plain_delta(*r, heads, kv, dim, vdim) for r in rows]
    for stepwise in (False, True):
        state = torch.zeros(5, 12 + heads * vdim * dim, device=DEVICE)
        done, cuts = [0] * len(CUTS), [[1] * sum(c) for c in CUTS] if stepwise else CUTS
        eps, scale, weight = 1e-5, 1.3, torch.rand(vdim, generator=gen) + 0.5
        for live, batch in batches_of(cuts, SLOTS):
            qkv, beta, g = (torch.cat([rows[s][i][done[s]:done[s] + n] for s, n in zip(live, batch.q_lens)]).to(DEVICE)
                            for i in range(3))
            if stepwise:
                gate = torch.randn(batch.n, heads * vdim + 5, generator=gen)
                wide = torch.zeros(batch.n, heads * vdim + 8, device=DEVICE)
                sigmoid = channel
                kernels.delta_step(qkv, beta, g, state, 12, batch.cu_q, batch.slots, len(live), gate.to(DEVICE)[:, 2:2 + heads * vdim],
                                   sigmoid, weight.to(DEVICE), eps, wide[:, 4:4 + heads * vdim], kv, heads, dim, vdim,
                                   out_scale=scale)
                out = wide[:, 4:4 + heads * vdim].double().cpu()
                assert float(wide[:, :4].abs().max()) == 0.0 and float(wide[:, 4 + heads * vdim:].abs().max()) == 0.0
                z = gate.double()[:, 2:2 + heads * vdim]
                act = torch.sigmoid(z) if sigmoid else plain.silu(z)
            else:
                out = torch.empty(batch.n, heads * vdim, device=DEVICE)
                kernels.delta_scan(qkv, beta, g, state, 12, batch.tok_seq, batch.cu_q, batch.slots, len(live), out, kv, heads, dim,
                                   vdim)
                out = out.double().cpu()
            for i, s in enumerate(live):
                o = want[s][done[s]:done[s] + batch.q_lens[i]]
                mine = out[batch.rows(i)]
                if stepwise:
                    o = scale * plain.over_rms(o, eps) * weight.double()
                    o = o.reshape(len(o), -1) * act[batch.rows(i)]
                o = o.reshape(len(mine), -1)
                assert torch.allclose(mine, o, rtol=2e-4, atol=2e-5 * max(1.0, float(o.abs().max()))), (stepwise, s, done[s])
                done[s] += batch.q_lens[i]
        assert float(state[:, :12].abs().max()) == 0.0                 # what lies ahead of S is somebody else's


def test_delta_rule_padding_rows():
    """A fixed-size batch of four rows with two requests: the rows beyond them hold no numbers, get zeros, move no state."""
    heads, kv, dim, vdim = 2, 1, 16, 12
    for channel in (False, True):
        bad = lambda *shape: torch.full(shape, float("nan"), device=DEVICE)
        qkv, beta = bad(4, 2 * kv * dim + heads * vdim), bad(4, heads)
        g = bad(4, heads, dim) if channel else bad(4, heads)
        for tensor in (qkv, beta, g):
            tensor[:2] = torch.rand(2, *tensor.shape[1:], device=DEVICE) * 0.5
        state = torch.zeros(3, heads * vdim * dim, device=DEVICE)
        out = torch.full((4, heads * vdim), 7.0, device=DEVICE)
        kernels.delta_step(qkv, beta, g, state, 0, ints([0, 1, 2, 2, 2]), ints([2, 1, 0, 0]), 4, torch.zeros(4, heads * vdim, device=DEVICE),
                           True, torch.ones(vdim, device=DEVICE), 1e-5, out, kv, heads, dim, vdim)
        assert float(out[2:].abs().max()) == 0.0 and bool(torch.isfinite(out).all()) and float(state[0].abs().max()) == 0.0
        assert float(state[1].abs().max()) > 0.0 and float(state[2].abs().max()) > 0.0


@pytest.mark.parametrize("heads, kv, dim, vdim, taps", [(4, 2, 20, 28, 3), (2, 1, 128, 64, 4), (3, 3, 12, 40, 2), (2, 2, 160, 8, 4),
                                                        (1, 1, 36, 200, 8), (2, 1, 8, 12, 16)])
def test_convolved_unit_operands_and_their_memory(heads, kv, dim, vdim, taps):
    """Sequences cut every way (shorter portions than the convolution is long among them; a long batch takes the walk over
    eight tokens): convolution, silu, unit length, steps, decays and the memory, against the whole sequences."""
    gen = torch.Generator().manual_seed(dim + taps)
    channels = 2 * kv * dim + heads * vdim
    conv, rate = torch.randn(channels, taps, generator=gen), -torch.rand(heads, generator=gen) * 3
    dt_bias = torch.randn(heads, generator=gen) * 3
    for cuts in (CUTS, [[300, 1, 3], [2, 250, 100]]):
        slots = SLOTS[:len(cuts)]
        sequences = [torch.randn(sum(c), channels + 2 * heads, generator=gen) * 2 for c in cuts]
        state = torch.zeros(5, (taps - 1) * channels + 8, device=DEVICE)
        done, got = [0] * len(cuts), [[] for _ in cuts]
        for live, batch in batches_of(cuts, slots):
            rows = torch.cat([sequences[s][done[s]:done[s] + n] for s, n in zip(live, batch.q_lens)])
            proj = torch.nn.functional.pad(rows, (0, -rows.shape[1] % 4), value=9.0).to(DEVICE)
            qkv, beta, decay = (torch.full((batch.n, w), 5.0, device=DEVICE) for w in (channels, heads, heads))
            kernels.delta_prepare(proj, channels, channels + heads, conv.t().contiguous().to(DEVICE), rate.to(DEVICE),
                                  dt_bias.to(DEVICE), state, batch.tok_seq, batch.cu_q, batch.slots, qkv, beta, decay, kv, heads,
                                  dim, vdim, dim ** -0.5, 1e-6)
            if max(batch.q_lens) > 1:
                kernels.conv_state_update(proj, None, state, batch.cu_q, batch.slots, len(live), channels, taps)
            for i, s in enumerate(live):
                got[s].append(torch.cat([qkv, beta, decay], 1)[batch.rows(i)].double().cpu())
                done[s] += batch.q_lens[i]
        for s, sequence in enumerate(sequences):
            x, n = sequence.double(), len(sequence)
            y = plain.silu(plain.causal_conv(x[:, :channels], conv.double()))
            q = plain.over_length(y[:, :kv * dim].view(n, kv, dim)) * dim ** -0.5
            k = plain.over_length(y[:, kv * dim:2 * kv * dim].view(n, kv, dim))
            beta = torch.sigmoid(x[:, channels:channels + heads])
            g = torch.exp(rate.double() * plain.softplus(x[:, channels + heads:] + dt_bias.double()))
            want = torch.cat([q.reshape(n, -1), k.reshape(n, -1), y[:, 2 * kv * dim:], beta, g], 1)
            assert torch.allclose(torch.cat(got[s]), want, rtol=1e-4, atol=1e-5), s
            kept = torch.cat([torch.zeros(taps - 1, channels, dtype=F64), x[:, :channels]])[-(taps - 1):]
            assert torch.allclose(state[slots[s]].double().cpu()[:kept.numel()], kept.reshape(-1), atol=1e-6)


@pytest.mark.parametrize("heads, dim, rank, n", [(3, 20, 8, 21), (2, 128, 64, 5), (5, 4, 100, 40), (1, 256, 4, 1)])
def test_decays_per_channel(heads, dim, rank, n):
    gen = torch.Generator().manual_seed(rank)
    low, a2 = torch.randn(n, rank + 4, generator=gen) * 3, torch.randn(heads * dim, rank, generator=gen)
    bias, rate = torch.randn(heads * dim, generator=gen) * 2, -torch.rand(heads, generator=gen) * 2
    decay = torch.empty(n, heads, dim, device=DEVICE)
    kernels.delta_decay(low.to(DEVICE)[:, 4:], a2.to(DEVICE), bias.to(DEVICE), rate.to(DEVICE), decay)
    z = low.double()[:, 4:] @ a2.double().T + bias.double()
    want = torch.exp(rate.double()[:, None] * plain.softplus(z).view(n, heads, dim))
    assert torch.allclose(decay.double().cpu(), want, rtol=1e-4, atol=1e-6)


@pytest.mark.parametrize("heads, dim, vdim", [(3, 20, 28), (2, 64, 128), (5, 13, 7), (2, 128, 128), (1, 200, 40), (9, 8, 8)])
def test_lightning_recurrence_by_tokens_and_in_chunks(heads, dim, vdim):
    """q, k and v activated on their way in: the walk and, for heads that it takes, the chunked form without an ending."""
    gen = torch.Generator().manual_seed(dim)
    decay = torch.tensor([0.0, 1.0, 0.97, 0.5, 0.9, 0.999, 0.2, 0.8, 0.99])[:heads]
    cuts, slots = [[64, 1, 130], [63, 65, 64], [200, 128, 1], [0, 1, 7]], [3, 0, 2, 1]
    width = heads * (2 * dim + vdim)
    rows_of = [torch.randn(sum(c), width + 4, generator=gen) for c in cuts]
    size = kernels.retention_chunk_tokens()
    for chunked in (False, True) if max(dim, vdim) <= 128 else (False,):
        state = torch.zeros(4, heads, dim, vdim, device=DEVICE)
        done, got = [0] * len(cuts), [[] for _ in cuts]
        for live, batch in batches_of(cuts, slots):
            proj = torch.cat([rows_of[s][done[s]:done[s] + k] for s, k in zip(live, batch.q_lens)]).to(DEVICE)
            out = torch.empty(batch.n, heads * vdim, device=DEVICE)
            columns = (proj, 0, heads * dim, 2 * heads * dim)
            if chunked:
                chunks, first = kernels.scan_chunk_lists(batch.q_lens, size)
                kernels.retention_chunked(*columns, 0, decay.to(DEVICE), 1.0, 1e-5, state, batch.cu_q, batch.slots, len(live),
                                          ints(chunks), ints(first), len(chunks) // 2, out, heads, dim, vdim, silu=True, raw=True)
            else:
                kernels.retention_scan(*columns, decay.to(DEVICE), 1.0, state, batch.cu_q, batch.slots, len(live), out, heads, dim,
                                       vdim, silu=True)
            for i, s in enumerate(live):
                got[s].append(out[batch.rows(i)].double().cpu())
                done[s] += batch.q_lens[i]
        for s, rows in enumerate(rows_of):
            x, n = plain.silu(rows.double()), len(rows)
            q, k = (x[:, i * heads * dim:(i + 1) * heads * dim].view(n, heads, dim) for i in range(2))
            want = plain.decaying_sum(q, k, x[:, 2 * heads * dim:width].view(n, heads, vdim), decay.double()).reshape(n, -1)
            assert torch.allclose(torch.cat(got[s]), want, rtol=2e-4, atol=1e-4 * float(want.abs().max())), (chunked, s)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [60, 256, 1000, 2500])
@pytest.mark.parametrize("sigmoid", [False, True])
def test_one_norm_over_all_heads_with_a_gate(dtype, width, sigmoid):
    gen = torch.Generator().manual_seed(width)
    o, gate, w = torch.randn(9, width, generator=gen) * 5, torch.randn(9, width + 7, generator=gen), torch.randn(width, generator=gen)
    wide = torch.zeros(9, width + 16, dtype=dtype, device=DEVICE)
    kernels.norm_gate_rows(o.to(DEVICE), gate.to(DEVICE)[:, 3:3 + width], w.to(DEVICE), 1e-3, wide[:, 8:8 + width], sigmoid_gate=sigmoid)
    z = gate.double()[:, 3:3 + width]
    want = plain.over_rms(o.double(), 1e-3) * w.double() * (torch.sigmoid(z) if sigmoid else plain.silu(z))
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert torch.allclose(wide[:, 8:8 + width].double().cpu(), want, rtol=tol, atol=tol)
    assert float(wide[:, :8].abs().max()) == 0.0 and float(wide[:, 8 + width:].abs().max()) == 0.0


def test_heads_filled_up_with_zeros_keep_their_own_mean():
    gen = torch.Generator().manual_seed(1)
    o, gate = torch.randn(7, 3, 12, generator=gen), torch.randn(7, 3, 12, generator=gen)
    o[:, :, 9:] = 0.0
    weight = torch.cat([torch.rand(9, generator=gen), torch.zeros(3)])
    out = torch.empty(7, 36, device=DEVICE)
    kernels.gla_norm_gate(o.view(7, 36).to(DEVICE), gate.view(7, 36).to(DEVICE), weight.to(DEVICE), 1e-4, out, 3, 12,
                          sigmoid_gate=True, out_scale=-0.7, true_vdim=9)
    want = -0.7 * plain.over_rms(o.double()[:, :, :9], 1e-4) * weight.double()[:9] * torch.sigmoid(gate.double()[:, :, :9])
    got = out.double().cpu().view(7, 3, 12)
    assert torch.allclose(got[:, :, :9], want, atol=1e-5) and float(got[:, :, 9:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts, top, groups", [(6, 2, (3, 1)), (8, 3, (2, 2)), (16, 2, (4, 2)), (9, 2, (9, 3)), (40, 5, (8, 3)),
                                                  (5, 2, None), (1, 1, None), (128, 40, (2, 1)), (12, 6, (2, 1))])
def test_router_kernel_limited_to_the_best_groups(dtype, experts, top, groups):
    gen = torch.Generator().manual_seed(experts * 7 + top)
    n, width = 60, 72
    h, router = torch.randn(n, width, generator=gen).to(dtype), torch.randn(experts, width, generator=gen) * 0.3
    chosen, place = ints([0] * n * top), ints([0] * n * top)
    counts, weights = ints([0] * experts), torch.empty(n * top, dtype=torch.float32, device=DEVICE)
    count, keep = groups or (1, 1)
    kernels.moe_route_softmax(h.to(DEVICE), router.to(DEVICE), top, 0, None, chosen, weights, counts, place, n_groups=count, keep=keep)
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": count, "keep": keep}
    want, margin = plain.route(h.double(), router.double(), r)
    got_ids, got = chosen.view(n, top).cpu().long(), weights.view(n, top).cpu().double()
    clear = margin > 1e-3
    assert int(clear.sum()) > n // 2
    assert torch.equal(torch.sort(got_ids[clear], 1).values, torch.sort(want[clear], 1).values)
    scores = torch.gather(torch.softmax(h.double() @ router.double().T, -1), 1, got_ids)
    assert torch.allclose(got, scores / scores.sum(1, keepdim=True), atol=1e-5)
    assert int(counts.sum()) == n * top and torch.equal(torch.bincount(got_ids.flatten(), minlength=experts).to(torch.int32), counts.cpu())


def test_a_grouped_router_that_sees_no_numbers_stays_inside_its_arrays():
    h, router = torch.full((3, 40), float("nan"), device=DEVICE), torch.randn(6, 40, device=DEVICE)
    chosen, place, counts = ints([-1] * 6), ints([0] * 6), ints([0] * 6)
    weights = torch.empty(6, dtype=torch.float32, device=DEVICE)
    kernels.moe_route_softmax(h, router, 2, 0, None, chosen, weights, counts, place, n_groups=3, keep=1)
    assert int(chosen.min()) >= 0 and int(chosen.max()) < 6 and int(counts.sum()) == 6


@pytest.mark.parametrize("hidden", [40, 1002, 2048])
def test_a_step_vector_joins_what_is_still_to_be_added(hidden):
    """A vector for every row, alone or beside a product's float result: added by the next norm, or by whoever asks."""
    gen = torch.Generator().manual_seed(hidden)
    x, acc, vector, weight = (torch.randn(*shape, generator=gen).to(DEVICE) for shape in ((9, hidden), (9, hidden), (hidden,), (hidden,)))
    for there in (None, acc):
        want = x.double() + vector.double() + (there.double() if there is not None else 0.0)
        assert torch.allclose(PendingSum(there, vector, x.clone()).tensor().double(), want, atol=1e-5)
        stream, out = x.clone(), torch.empty(9, hidden, device=DEVICE)
        kernels.rmsnorm_pending(stream, there, vector, weight, 0.0, 1e-4, out)
        assert torch.allclose(stream.double(), want, atol=1e-5)
        assert torch.allclose(out.double(), plain.over_rms(want, 1e-4) * weight.double(), rtol=1e-5, atol=1e-5)


# ---------------------------------------------------------------------- single layers
BASE = lightning(2, 16, 16, [0.9, 0.99])
LAYERS_ALONE = {
    "lightning": lightning(3, 20, 28, [0.9, 0.99, 0.5]),
    "lightning_wide": lightning(2, 64, 128, [0.97, 0.999]),
    "lightning_wider_than_the_chunks": lightning(1, 144, 48, [0.995]),
    "lightning_without_or_with_all_memory": lightning(2, 16, 40, [0.0, 1.0]),
    "delta": delta(6, 2, 12, 20, 5),
    "delta_one_head": delta(1, 1, 96, 24, 3),
    "delta_64": delta(4, 4, 64, 64, 4),
    "delta_128_shared_keys": delta(4, 1, 128, 64, 2),
    "delta_odd_sizes_nine_taps": delta(5, 5, 5, 9, 9),
    "delta_one_tap_wide_keys": delta(2, 2, 200, 12, 1),
    "parallel": parallel((6, 3, 24, 40, 0.3, (12, 500.0)), (4, 2, 20, 28, 3), 0.7, 1.4),
    "parallel_tensor_core_heads": parallel((4, 2, 64, 64, 0.2, (64, 10000.0)), (2, 2, 64, 128, 4), 1.2, 0.9),
    "parallel_left_only_in_weight": parallel((2, 2, 16, 16, 0.4, (16, 300.0)), (2, 1, 8, 8, 2), 2.0, 0.01),
    "parallel_right_only_in_weight": parallel((2, 2, 16, 16, 0.4, (8, 300.0)), (4, 2, 32, 16, 4), 0.01, 2.0),
    "parallel_unrotated_odd": parallel((5, 5, 13, 21, 0.4, None), (3, 1, 13, 7, 1), 1.3, -0.9),
    "parallel_keys_wider": parallel((4, 1, 40, 24, 0.3, (40, 5000.0)), (2, 2, 128, 20, 3), -0.8, 1.0),
    "dense_feed_forward": dict(BASE, mlp=dense(72)),
    "experts_in_groups": dict(BASE, mlp=moe(40, 6, 2, (3, 1))),
    "experts_in_kept_groups": dict(BASE, mlp=moe(24, 8, 3, (4, 2), limit=0.4)),
    "experts_without_groups_or_limit": dict(BASE, mlp=moe(33, 5, 2, limit=None)),
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
@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 2), (1, 2, 4), (2, 3, 3)])
def test_repeated_runs_of_layers(loop, dtype):
    """Every pass has a cache and state of its own and its own step vector, wherever the run begins and ends."""
    raw = model(64, 120, [parallel((2, 1, 16, 16, 0.4, (16, 100.0)), (2, 1, 8, 12, 3), 0.6, 1.0, mlp=dense(40)),
                          delta(2, 1, 16, 8, 2), lightning(2, 8, 12, [0.9, 0.6], mlp=moe(24, 4, 2, (2, 1)))], loop=loop)
    run = Run(raw, draw(raw, seed=17, router_gain=3.0), dtype, max_tokens=4 * 128)
    assert len(run.replayer.model.cache_plan.state_of_entry) == len(plain.layer_runs(raw))
    tokens = ids(60, raw["vocab"], seed=6)
    for name, sizes in (("whole", [60]), ("cut", cycle), ("decoded", [20])):
        run.feed(name, tokens, sizes)
        run.check(name, tokens)


# ---------------------------------------------------------------------- planted tokens
def _align(raw, tensors):
    """The last query (token 89) points at the key of token 88 in every head (no rotation)."""
    m = raw["layers"][0]["mixer"]["left"]
    h88, h89 = (plain.over_rms(tensors["embed"][t], raw["norm"]["eps"]) * tensors["l0.norm1"] for t in (88, 89))
    k88 = (tensors["l0.mix.left.k"] @ h88).view(m["kv_heads"], m["dim"])
    group = m["heads"] // m["kv_heads"]
    target = torch.cat([k88[h // group] / k88[h // group].norm() for h in range(m["heads"])])
    tensors["l0.mix.left.q"] = (torch.outer(target, h89) / (h89 @ h89) * 3.0).contiguous()


PLANTED = {
    "simt": (parallel((2, 1, 32, 48, 1.2, None), (2, 1, 8, 8, 3), 1.5, 0.3), 430),
    "tensor_core": (parallel((4, 2, 64, 64, 0.9, None), (2, 1, 8, 8, 3), 1.5, 0.3), 430),
    "tensor_core_128": (parallel((4, 1, 128, 128, 0.7, None), (2, 1, 8, 8, 3), 1.5, 0.3), 200),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decode", [0, 50])
@pytest.mark.parametrize("name", list(PLANTED))
def test_one_key_decides_wherever_it_stands(name, decode, dtype):
    """The asked-for token among hundreds: the sequence's first ones, both sides of page borders, the place just before
    the last; in a whole prompt and with the tail decoded token by token."""
    layer, length = PLANTED[name]
    raw = single_layer(layer, vocab=90)
    tensors = draw(raw, seed=9)
    _align(raw, tensors)
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
            assert float(np.abs(row - base).max()) > 0.2, place


REMEMBERING = {"lightning": lightning(2, 16, 16, [1.0, 0.999]), "delta": delta(2, 1, 64, 16, 3),
               "channel_delta": parallel((2, 2, 16, 16, 0.1, None), (2, 2, 64, 16, 2), 0.02, 1.5)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(REMEMBERING))
def test_an_early_token_stays_in_the_state(kind, dtype):
    """One changed token at the start moves the last logits through the state alone (nothing else looks back), in every cut;
    a state that a portion drops, or a slot that keeps what it held, shows."""
    raw = single_layer(REMEMBERING[kind], vocab=90)
    tensors = draw(raw, seed=3)
    for name in tensors:
        if name.endswith("A_log"):
            tensors[name].fill_(-9.0)                                 # hardly any decay
        if name.endswith("mix.b") or name.endswith("right.b"):
            tensors[name].mul_(0.1)
    tokens = [t % 80 for t in ids(100, 90, seed=4)]
    other = list(tokens)
    other[2] = 85
    run = Run(raw, tensors, dtype, max_tokens=2 * 192, max_requests=2)
    weights = run.plain_weights
    expected = (plain.forward(raw, weights, tokens)[-1] - plain.forward(raw, weights, other)[-1]).abs().max()
    assert float(expected) > (2e-3 if dtype == "float32" else 5e-3)
    for turn, sizes in enumerate(([100], [], cycle, lambda turn: 2)):
        run.feed(f"a{turn}", tokens, sizes)
        run.check(f"a{turn}", tokens)
        run.feed(f"b{turn}", other, sizes)
        run.check(f"b{turn}", other)
        moved = np.abs(run.logits[(f"a{turn}", 99)] - run.logits[(f"b{turn}", 99)]).max()
        assert moved > float(expected) / 3, moved


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
    """A prompt long enough for the prompt-sized product kernels, many attention tiles, chunks and groups of the recurrences:
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
        model_ = model_from_tensors(config_of(raw, tensors), tensors, dtype="float32", device=DEVICE)
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
    assert "finish_reason:  length" in done.stdout and "Palelix" in done.stdout
