"""Linear attention: a matrix state per head that decays.

Gated linear attention decays per key channel, by the token.
Per token t and head (``GlaSpec``): ``q = Wq h * query_scale``, ``k = Wk h``, ``v = Wv h``, a decay per key channel
``a = sigmoid(A2 (A1 h) + b)^(1/tau)``; ``S_t = diag(a_t) S_(t-1) + k_t v_t^T`` from S = 0 and ``o_t = S_t^T q_t``.
Every head's o is RMS-normalised over its value width with one plain weight, multiplied by ``silu(Wg h)`` and
projected by Wo. Per request the state slot holds S for every head, float32; a step continues from it and leaves
it for the next one, so a sequence may be cut anywhere.

One fused product gives float rows ``[q | k | v | gate | A1 h]``; the second decay product (rank x channels, tiny)
stays on the FP32 cores with float weights, so the decays, their logarithms and exponentials, the state, the norm
and the gate are float in both dtypes; only the large projections run in the runtime dtype.

Retention (``RetentionSpec``) decays by one constant per head: ``S_t = decay_h S_(t-1) + k_t v_t^T``, ``o_t = S_t^T q_t`` with
q and k rotated over their first entries. It shares the recurrence's kernel (which takes no decay operand then), the
state's layout and the kernel behind it (no weight in its norm); short portions are rotated by a pass of their own, steps
of one token a sequence on the operands' way into the recurrence. In another form (lightning attention) q, k and v are the
silu of their projections, taken on the operands' way in, and one norm with a weight spans all heads. Long portions of heads of up to 128 x 128 run in chunks
of tokens whose products take the place of the updates, with rotation, norm and gate in the same kernels.
"""

from __future__ import annotations

import torch

from matricxon_b200.ops import kernels
from matricxon_b200.ops.linear import EPILOGUE_F32, EPILOGUE_RESIDUAL, linear
from matricxon_b200.parts.attention import one_token_each
from matricxon_b200.parts.base import BranchMixer, Mixer, StateRequest, build_part, register_part
from matricxon_b200.weights.loader import WeightSpec


@register_part("mixer", "gla")
class GatedLinearAttention(Mixer):
    capturable = True

    @classmethod
    def _matrices(cls, spec):
        keys, values = spec.num_heads * spec.head_dim, spec.num_heads * spec.value_dim
        return [(spec.query_name, keys), (spec.key_name, keys), (spec.value_name, values), (spec.gate_name, values),
                (spec.decay_down_name, spec.decay_rank)]

    @classmethod
    def weight_specs(cls, spec, prefix):
        s = spec
        specs = [WeightSpec(prefix + name, (rows, s.hidden_size), role="matrix", init="weight")
                 for name, rows in cls._matrices(s)]
        channels = s.num_heads * s.head_dim
        # the second decay product runs in float: its matrix is held like a vector
        specs.append(WeightSpec(prefix + s.decay_up_name, (channels, s.decay_rank), role="vector", init="weight"))
        specs.append(WeightSpec(prefix + s.decay_up_name + s.bias_suffix, (channels,), role="vector", init="bias"))
        specs.append(WeightSpec(prefix + s.norm_name, (s.value_dim,), role="vector", init="norm_weight"))
        specs.append(WeightSpec(prefix + s.output_name, (s.hidden_size, s.num_heads * s.value_dim), role="matrix",
                                init="weight"))
        return specs

    @classmethod
    def state_request(cls, spec):
        return StateRequest(shape=(spec.num_heads, spec.head_dim, spec.value_dim), dtype=torch.float32)

    def load(self, fetch):
        p, s = self.prefix, self.spec
        self.proj_weight = torch.cat([fetch(p + name) for name, _ in self._matrices(s)])
        self.decay_up = fetch(p + s.decay_up_name)
        self.decay_bias = fetch(p + s.decay_up_name + s.bias_suffix)
        self.norm_weight = fetch(p + s.norm_name)
        self.o_weight = fetch(p + s.output_name)

    def forward(self, h, residual, ctx, binding):
        s, rt = self.spec, self.runtime
        if binding.state is None:
            raise RuntimeError("gated linear attention needs a state tensor bound to it")
        n = h.shape[0]
        keys, values = s.num_heads * s.head_dim, s.num_heads * s.value_dim
        proj = linear(h, self.proj_weight, None, EPILOGUE_F32, backend=rt.gemm_backend)
        k_col, v_col, g_col, low_col = keys, 2 * keys, 2 * keys + values, 2 * keys + 2 * values
        decay = torch.empty((n, keys), dtype=torch.float32, device=h.device)
        kernels.gla_decay(proj[:, low_col:low_col + s.decay_rank], self.decay_up, self.decay_bias, s.tau, decay)
        o = torch.empty((n, values), dtype=torch.float32, device=h.device)
        kernels.gla_scan(proj, 0, k_col, v_col, decay, s.query_scale, binding.state, ctx.cu_q, ctx.state_slots,
                         ctx.n_seqs, o, s.num_heads, s.head_dim, s.value_dim)
        out = torch.empty((n, values), dtype=rt.dtype, device=h.device)
        kernels.gla_norm_gate(o, proj[:, g_col:g_col + values], self.norm_weight, s.eps, out, s.num_heads, s.value_dim)
        if residual is None:
            return linear(out, self.o_weight, None, EPILOGUE_F32, backend=rt.gemm_backend)
        return linear(out, self.o_weight, None, EPILOGUE_RESIDUAL, residual=residual, out=residual,
                      backend=rt.gemm_backend, defer_sum=getattr(ctx, "sums_may_pend", False))


@register_part("mixer", "retention")
class Retention(BranchMixer):
    capturable = True

    def __init__(self, spec, runtime, prefix):
        super().__init__(spec, runtime, prefix)
        self.position = (build_part("position", spec.position, runtime, prefix)
                         if spec.position is not None and spec.position.rotary_dim > 0 else None)
        if self.position is not None and (not hasattr(self.position, "frequencies")
                                          or getattr(self.position, "interleaved", False)
                                          or getattr(self.position, "amplitude", 1.0) != 1.0):
            raise ValueError(f"retention rotates by a plain table with halves paired, not by {spec.position!r}")
        if self.position is not None and spec.activation is not None:
            raise ValueError("activated heads are not rotated by any kernel")
        self.silu, self.sigmoid_gate, self.joint = spec.activation == "silu", spec.gate == "sigmoid", spec.norm == "all"

    @classmethod
    def _matrices(cls, spec):
        keys, values = spec.num_heads * spec.head_dim, spec.num_heads * spec.value_dim
        return [(spec.query_name, keys), (spec.key_name, keys), (spec.value_name, values), (spec.gate_name, values)]

    @classmethod
    def weight_specs(cls, spec, prefix):
        specs = [WeightSpec(prefix + name, (rows, spec.hidden_size), role="matrix", init="weight")
                 for name, rows in cls._matrices(spec)]
        if spec.norm_name is not None:
            specs.append(WeightSpec(prefix + spec.norm_name, (spec.num_heads * spec.value_dim,), role="vector",
                                    init="norm_weight"))
        specs.append(WeightSpec(prefix + spec.output_name, (spec.hidden_size, spec.num_heads * spec.value_dim),
                                role="matrix", init="weight"))
        return specs

    @classmethod
    def state_request(cls, spec):
        return StateRequest(shape=(spec.num_heads, spec.head_dim, spec.value_dim), dtype=torch.float32)

    def load(self, fetch):
        p, s = self.prefix, self.spec
        self.input_weight = torch.cat([fetch(p + name) for name, _ in self._matrices(s)])
        self.output_weight = fetch(p + s.output_name)
        self.norm_weight = fetch(p + s.norm_name) if s.norm_name is not None else None
        self.decay = torch.tensor(s.decay, dtype=torch.float32, device=self.runtime.device)

    def mix(self, proj, ctx, binding, out, scale=1.0):
        s = self.spec
        if binding.state is None:
            raise RuntimeError("retention needs a state tensor bound to it")
        if scale != 1.0:
            raise RuntimeError("retention's output is normalised per head: it takes no scale")
        n, keys, values = proj.shape[0], s.num_heads * s.head_dim, s.num_heads * s.value_dim
        rotation = {}
        if self.position is not None:
            freq, rot = self.position.frequencies, s.position.rotary_dim
        if not one_token_each(ctx) and max(s.head_dim, s.value_dim) <= 128 and \
                max(ctx.host.q_lens) > kernels.retention_chunk_tokens() // 2:
            # long portions in chunks of tokens, products in place of updates
            size = kernels.retention_chunk_tokens()
            key = ("retention_chunks", size)
            if key not in ctx.memo:
                chunks, first = kernels.scan_chunk_lists(ctx.host.q_lens, size)
                both = torch.tensor(chunks + first, dtype=torch.int32).to(proj.device, non_blocking=True)
                ctx.memo[key] = (both[:len(chunks)], both[len(chunks):], len(chunks) // 2)
            if self.position is not None:
                rotation = {"positions": ctx.positions, "freq": freq, "rot": rot}
            # the kernel ends in a silu-gated norm of every head; another ending follows it as a kernel of its own
            raw = self.joint or self.sigmoid_gate
            o = torch.empty((n, values), dtype=torch.float32, device=proj.device) if raw else out
            kernels.retention_chunked(proj, 0, keys, 2 * keys, 2 * keys + values, self.decay, s.key_scale, s.eps,
                                      binding.state, ctx.cu_q, ctx.state_slots, ctx.n_seqs, *ctx.memo[key], o,
                                      s.num_heads, s.head_dim, s.value_dim, silu=self.silu, raw=raw, **rotation)
            if raw:
                self._norm_gate(o, proj, out)
            return
        if self.position is not None:
            if one_token_each(ctx):
                rotation = {"positions": ctx.positions, "freq": freq, "rot": rot}
            else:                                                     # q and k heads lie side by side
                kernels.rotate_heads(proj, 0, 2 * s.num_heads, s.head_dim, rot, ctx.positions, freq)
        o = torch.empty((n, values), dtype=torch.float32, device=proj.device)
        # the scale of k goes on q: the output is linear in both, and the state then holds the plain k v^T
        kernels.retention_scan(proj, 0, keys, 2 * keys, self.decay, s.key_scale, binding.state, ctx.cu_q, ctx.state_slots,
                               ctx.n_seqs, o, s.num_heads, s.head_dim, s.value_dim, silu=self.silu, **rotation)
        self._norm_gate(o, proj, out)

    def _norm_gate(self, o, proj, out):
        s = self.spec
        keys, values = s.num_heads * s.head_dim, s.num_heads * s.value_dim
        gate = proj[:, 2 * keys + values:2 * keys + 2 * values]
        if self.joint:
            kernels.norm_gate_rows(o, gate, self.norm_weight, s.eps, out, sigmoid_gate=self.sigmoid_gate)
        else:
            kernels.gla_norm_gate(o, gate, None, s.eps, out, s.num_heads, s.value_dim, sigmoid_gate=self.sigmoid_gate)
