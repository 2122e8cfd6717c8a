"""A selective state-space recurrence (Mamba's): a state per channel whose decay and input depend on the token.

``SelectiveScanSpec``: ``[x | z] = W_in h``, ``u = silu(conv(x) + b)``, ``[low | B | C] = W_x u``,
``dt = softplus(W_dt low + b_dt)``, ``S <- exp(dt A) S + dt u B`` per channel from S = 0 and ``y = S C + D u``; the output is
``W_o (y * silu(z))``. Per request the state slot holds one float vector: the convolution's latest ``taps - 1`` inputs
[taps - 1, channels], then S [channels, states]; a step continues from it and leaves it for the next one, so a sequence
may be cut anywhere.

The large products run in the runtime dtype; their results, the steps and their softplus, the decays and exponentials, the
state and the gate are float. Steps in which no sequence brings more than one token fold the small product W_dt into the
recurrence's kernel.
"""

from __future__ import annotations

import math

import torch

from matricxon_b200.ops import kernels
from matricxon_b200.ops.linear import EPILOGUE_F32, linear
from matricxon_b200.parts.attention import one_token_each
from matricxon_b200.parts.base import BranchMixer, StateRequest, register_part
from matricxon_b200.weights.loader import WeightSpec


# tokens per chunk of a long portion, and the channels (over all sequences) per SM from which on the token-by-token walk
# has warps enough
CHUNK_TOKENS = 64
CHANNELS_THAT_FILL = 96


@register_part("mixer", "selective_scan")
class SelectiveScan(BranchMixer):
    capturable = True

    @classmethod
    def weight_specs(cls, spec, prefix):
        s, p, b = spec, prefix, spec.bias_suffix
        return [WeightSpec(p + s.input_name, (2 * s.channels, s.hidden_size), role="matrix", init="weight"),
                WeightSpec(p + s.conv_name, (s.channels, s.taps), role="vector", init="weight"),
                WeightSpec(p + s.conv_name + b, (s.channels,), role="vector", init="bias"),
                WeightSpec(p + s.low_name, (s.dt_rank + 2 * s.states, s.channels), role="matrix", init="weight"),
                WeightSpec(p + s.dt_name, (s.channels, s.dt_rank), role="matrix", init="weight"),
                WeightSpec(p + s.dt_name + b, (s.channels,), role="vector", init="bias"),
                WeightSpec(p + s.a_log_name, (s.channels, s.states), role="vector", init="bias"),
                WeightSpec(p + s.d_name, (s.channels,), role="vector", init="norm_weight"),
                WeightSpec(p + s.output_name, (s.hidden_size, s.channels), role="matrix", init="weight")]

    @classmethod
    def state_request(cls, spec):
        return StateRequest(shape=(spec.channels * (spec.taps - 1 + spec.states),), dtype=torch.float32)

    def load(self, fetch):
        p, s, b = self.prefix, self.spec, self.spec.bias_suffix
        self.input_weight = fetch(p + s.input_name)
        self.conv = fetch(p + s.conv_name).t().contiguous()          # [taps][channels]
        self.conv_bias = fetch(p + s.conv_name + b)
        self.low_weight = fetch(p + s.low_name)
        self.dt_weight = fetch(p + s.dt_name)
        self.dt_bias = fetch(p + s.dt_name + b)
        # A = -exp(A_log), times log2(e): a decay is then one base-2 exponential of dt times it
        self.a_log2 = (-torch.exp(fetch(p + s.a_log_name).double()) * math.log2(math.e)).float().contiguous()
        self.d = fetch(p + s.d_name)
        self.output_weight = fetch(p + s.output_name)

    def mix(self, proj, ctx, binding, out, scale=1.0):
        s, rt = self.spec, self.runtime
        if binding.state is None:
            raise RuntimeError("the recurrence needs a state tensor bound to it")
        n, c, state = proj.shape[0], s.channels, binding.state
        x, z = proj[:, :c], proj[:, c:2 * c]
        u = torch.empty((n, c), dtype=rt.dtype, device=proj.device)
        kernels.conv_silu(x, self.conv, self.conv_bias, state, ctx.tok_seq, ctx.cu_q, ctx.state_slots, u)
        low = linear(u, self.low_weight, None, EPILOGUE_F32, backend=rt.gemm_backend)
        recurrent = c * (s.taps - 1)                                  # where S starts in a slot's vector
        if one_token_each(ctx):
            kernels.selective_step(u, low, self.dt_weight, self.dt_bias, self.a_log2, self.d, z, state, recurrent, ctx.cu_q,
                                   ctx.state_slots, ctx.n_seqs, out, s.states, s.dt_rank, scale)
            return
        kernels.conv_state_update(x, None, state, ctx.cu_q, ctx.state_slots, ctx.n_seqs, c, s.taps)
        rank_rows = low[:, :s.dt_rank]
        if rt.dtype != torch.float32:
            rounded = torch.empty((n, s.dt_rank), dtype=rt.dtype, device=proj.device)
            kernels.cast_columns(rank_rows, rounded)
            rank_rows = rounded
        raw = linear(rank_rows, self.dt_weight, None, EPILOGUE_F32, backend=rt.gemm_backend)
        chunked = None
        if ctx.n_seqs * c < CHANNELS_THAT_FILL * ctx.sm_count and max(ctx.host.q_lens) > 2 * CHUNK_TOKENS:
            # a long portion of few sequences: token by token it would be left to a few warps per SM
            key = ("selective_chunks", CHUNK_TOKENS)
            if key not in ctx.memo:
                chunks, first = kernels.scan_chunk_lists(ctx.host.q_lens, CHUNK_TOKENS)
                both = torch.tensor(chunks + first, dtype=torch.int32).to(proj.device, non_blocking=True)
                ctx.memo[key] = (both[:len(chunks)], both[len(chunks):], len(chunks) // 2, CHUNK_TOKENS)
            chunked = ctx.memo[key]
        kernels.selective_scan(u, raw, low, self.dt_bias, self.a_log2, self.d, z, state, recurrent, ctx.cu_q,
                               ctx.state_slots, ctx.n_seqs, out, s.states, s.dt_rank, scale, chunked=chunked)
