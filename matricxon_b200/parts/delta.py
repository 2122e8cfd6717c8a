"""Linear attention by the gated delta rule (``DeltaRuleSpec``): a matrix state per value head that forgets, corrects what it
holds under the token's key, and is read with its query.

``S <- g S``, ``u = beta (v - S^T k)``, ``S <- S + k u^T``, ``o = S^T q`` with q, k and v behind short causal convolutions and
silu, q and k of unit length, and g one decay per head or one per head and key channel. Per request the state slot holds one
float vector: the convolutions' latest ``taps - 1`` inputs, then S of every head, transposed ([heads, values, keys]); a step
continues from it and leaves it for the next one, so a sequence may be cut anywhere.

One fused product gives float rows ``[q | k | v | gate | decay | beta]`` (the low-rank maps' first products in the places of
gate and decay); a kernel convolves, activates and normalises them and forms the steps, another the decays per channel from
float operands. Portions run through the recurrence in groups of eight tokens with the state in registers; steps of one token a sequence
have a kernel of their own that also ends the mixer (norm, weight, gate). Everything between the products is float in
both dtypes; of the low-rank maps the decay's second product is float too, the gate's runs in the runtime dtype.

Head sizes are filled up to multiples of four at load, with rows of zeros in the matrices: the kernels then read and write 16
bytes at a time whatever the sizes.
"""

from __future__ import annotations

import torch

from matricxon_b200.ops import kernels
from matricxon_b200.ops.linear import EPILOGUE_F32, linear
from matricxon_b200.parts.attention import one_token_each
from matricxon_b200.parts.base import BranchMixer, StateRequest, register_part
from matricxon_b200.weights.loader import WeightSpec

_KERNEL_TAPS = (2, 3, 4, 8, 16)      # shorter convolutions are filled up with zero taps on the oldest side


def _up(n: int, multiple: int) -> int:
    return -(-n // multiple) * multiple


def _pad_heads(rows: torch.Tensor, heads: int, size: int, padded: int) -> torch.Tensor:
    """[heads * size, ...] -> [heads * padded, ...] with zeros behind every head's entries."""
    if size == padded:
        return rows
    out = torch.zeros((heads, padded, *rows.shape[1:]), dtype=rows.dtype, device=rows.device)
    out[:, :size] = rows.view(heads, size, *rows.shape[1:])
    return out.view(heads * padded, *rows.shape[1:])


@register_part("mixer", "delta_rule")
class DeltaRule(BranchMixer):
    capturable = True

    def __init__(self, spec, runtime, prefix):
        super().__init__(spec, runtime, prefix)
        self.dim, self.vdim, self.taps, self.channels = self._sizes(spec)
        self.per_channel, self.low_gate = len(spec.decay_names) == 2, len(spec.gate_names) == 2

    @staticmethod
    def _sizes(spec):
        """(key entries of a head, value entries of a head, taps, convolved channels) as the kernels see them."""
        dim, vdim = _up(spec.head_dim, 4), _up(spec.value_dim, 4)
        taps = next(t for t in _KERNEL_TAPS if t >= spec.taps)
        return dim, vdim, taps, 2 * spec.num_kv_heads * dim + spec.num_heads * vdim

    @classmethod
    def _projections(cls, spec):
        """(name, heads, entries of a head) of the convolved projections, in the order of their columns."""
        return [(spec.query_name, spec.num_kv_heads, spec.head_dim), (spec.key_name, spec.num_kv_heads, spec.head_dim),
                (spec.value_name, spec.num_heads, spec.value_dim)]

    @classmethod
    def weight_specs(cls, spec, prefix):
        s, p = spec, prefix
        specs = []
        for name, heads, size in cls._projections(s):
            specs += [WeightSpec(p + name, (heads * size, s.hidden_size), role="matrix", init="weight"),
                      WeightSpec(p + name + s.conv_suffix, (heads * size, s.taps), role="vector", init="weight")]
        specs += [WeightSpec(p + s.beta_name, (s.num_heads, s.hidden_size), role="matrix", init="weight"),
                  WeightSpec(p + s.a_log_name, (s.num_heads,), role="vector", init="bias"),
                  WeightSpec(p + s.norm_name, (s.value_dim,), role="vector", init="norm_weight")]
        if len(s.decay_names) == 2:
            # the second decay product runs in float: its matrix is held like a vector
            specs += [WeightSpec(p + s.decay_names[0], (s.decay_rank, s.hidden_size), role="matrix", init="weight"),
                      WeightSpec(p + s.decay_names[1], (s.num_heads * s.head_dim, s.decay_rank), role="vector", init="weight"),
                      WeightSpec(p + s.dt_bias_name, (s.num_heads * s.head_dim,), role="vector", init="bias")]
        else:
            specs += [WeightSpec(p + s.decay_names[0], (s.num_heads, s.hidden_size), role="matrix", init="weight"),
                      WeightSpec(p + s.dt_bias_name, (s.num_heads,), role="vector", init="bias")]
        values = s.num_heads * s.value_dim
        if len(s.gate_names) == 2:
            specs += [WeightSpec(p + s.gate_names[0], (s.gate_rank, s.hidden_size), role="matrix", init="weight"),
                      WeightSpec(p + s.gate_names[1], (values, s.gate_rank), role="matrix", init="weight")]
        else:
            specs.append(WeightSpec(p + s.gate_names[0], (values, s.hidden_size), role="matrix", init="weight"))
        specs.append(WeightSpec(p + s.output_name, (s.hidden_size, values), role="matrix", init="weight"))
        return specs

    @classmethod
    def state_request(cls, spec):
        dim, vdim, taps, channels = cls._sizes(spec)
        return StateRequest(shape=((taps - 1) * channels + spec.num_heads * vdim * dim,), dtype=torch.float32)

    def load(self, fetch):
        p, s = self.prefix, self.spec
        matrices, convs = [], []
        for (name, heads, size), padded in zip(self._projections(s), (self.dim, self.dim, self.vdim)):
            matrices.append(_pad_heads(fetch(p + name), heads, size, padded))
            convs.append(_pad_heads(fetch(p + name + s.conv_suffix), heads, size, padded))
        conv = torch.cat(convs).t()                                                            # [taps][channels]
        self.conv = torch.nn.functional.pad(conv, (0, 0, self.taps - s.taps, 0)).contiguous()

        def rows_of_four(matrix):                       # the next matrix's columns start on a 16-byte boundary
            return torch.nn.functional.pad(matrix, (0, 0, 0, -matrix.shape[0] % 4))

        gate = fetch(p + s.gate_names[0])
        self.gate_rows = s.gate_rank if self.low_gate else s.num_heads * self.vdim
        matrices.append(rows_of_four(gate if self.low_gate else _pad_heads(gate, s.num_heads, s.value_dim, self.vdim)))
        self.gate_weight = (_pad_heads(fetch(p + s.gate_names[1]), s.num_heads, s.value_dim, self.vdim)
                            if self.low_gate else None)
        decay = rows_of_four(fetch(p + s.decay_names[0]))
        self.decay_rows = decay.shape[0]
        matrices += [decay, fetch(p + s.beta_name)]
        weight = torch.cat(matrices)
        self.input_weight = torch.nn.functional.pad(weight, (0, 0, 0, -weight.shape[0] % 8))
        self.rate = -torch.exp(fetch(p + s.a_log_name).double()).float().contiguous()
        self.dt_bias = fetch(p + s.dt_bias_name)
        self.decay_up = None
        if self.per_channel:
            up = _pad_heads(fetch(p + s.decay_names[1]), s.num_heads, s.head_dim, self.dim)
            self.decay_up = torch.nn.functional.pad(up, (0, self.decay_rows - s.decay_rank)).contiguous()
            self.dt_bias = _pad_heads(self.dt_bias, s.num_heads, s.head_dim, self.dim)
        self.norm_weight = torch.nn.functional.pad(fetch(p + s.norm_name), (0, self.vdim - s.value_dim)).contiguous()
        self.output_weight = _pad_heads(fetch(p + s.output_name).t(), s.num_heads, s.value_dim, self.vdim).t().contiguous()

    def mix(self, proj, ctx, binding, out, scale=1.0):
        s, rt, state = self.spec, self.runtime, binding.state
        if state is None:
            raise RuntimeError("the delta rule needs a state tensor bound to it")
        n, heads, dim, vdim, device = proj.shape[0], s.num_heads, self.dim, self.vdim, proj.device
        gate_col = self.channels
        decay_col = gate_col + _up(self.gate_rows, 4)
        beta_col = decay_col + self.decay_rows
        qkv = torch.empty((n, self.channels), dtype=torch.float32, device=device)
        beta = torch.empty((n, heads), dtype=torch.float32, device=device)
        decay = torch.empty((n, heads, dim) if self.per_channel else (n, heads), dtype=torch.float32, device=device)
        kernels.delta_prepare(proj, beta_col, decay_col, self.conv, None if self.per_channel else self.rate, self.dt_bias,
                              state, ctx.tok_seq, ctx.cu_q, ctx.state_slots, qkv, beta, None if self.per_channel else decay,
                              s.num_kv_heads, heads, dim, vdim, s.query_scale, s.unit_eps)
        if self.per_channel:
            kernels.delta_decay(proj[:, decay_col:beta_col], self.decay_up, self.dt_bias, self.rate, decay)
        gate = proj[:, gate_col:gate_col + self.gate_rows]
        if self.low_gate:
            low = torch.empty((n, s.gate_rank), dtype=rt.dtype, device=device)
            if rt.dtype == torch.float32:
                low.copy_(gate)
            else:
                kernels.cast_columns(gate, low)
            gate = linear(low, self.gate_weight, None, EPILOGUE_F32, backend=rt.gemm_backend)
        offset, sigmoid = self.channels * (self.taps - 1), s.gate == "sigmoid"
        if one_token_each(ctx):
            kernels.delta_step(qkv, beta, decay, state, offset, ctx.cu_q, ctx.state_slots, ctx.n_seqs, gate, sigmoid,
                               self.norm_weight, s.eps, out, s.num_kv_heads, heads, dim, vdim, out_scale=scale,
                               true_vdim=s.value_dim)
            return
        kernels.conv_state_update(proj, None, state, ctx.cu_q, ctx.state_slots, ctx.n_seqs, self.channels, self.taps)
        o = torch.empty((n, heads * vdim), dtype=torch.float32, device=device)
        kernels.delta_scan(qkv, beta, decay, state, offset, ctx.tok_seq, ctx.cu_q, ctx.state_slots, ctx.n_seqs, o,
                           s.num_kv_heads, heads, dim, vdim)
        kernels.gla_norm_gate(o, gate, self.norm_weight, s.eps, out, heads, vdim, sigmoid_gate=sigmoid, out_scale=scale,
                              true_vdim=s.value_dim)
