"""A state-space mixer with one decay per head and token (Mamba-2; Dao and Gu, "Transformers are SSMs"): a recurrent
mixer that keeps, per sequence and head, a state S of ``state`` x ``value_dim`` 32-bit floats, and the last inputs of its
short convolutions, in the cache's state area.

With h the mixer's input, H heads of P = value_dim lanes, G groups of B and C (head a uses group a // (H / G)), N =
state, and conv_T a causal convolution over time per channel (T taps, the last one the current token's, zeros before the
sequence's start) with a bias:

    z, x, B, C, dt = W_in h                                             [H, P], [H, P], [G, N], [G, N], [H]
    x, B, C = silu(conv_T(x, B, C) + b)
    dt = softplus(dt + dt_bias),   la = -exp(A_log) dt                  one of each per head
    S <- exp(la) S + dt B x^T,     y = S^T C + D x
    out = W_o (norm(y * silu(z)) * w)                                   norm: equal parts, each over its own root mean square

W_in is one product with 32-bit results (its rows padded with zeros to a multiple of 8).  Step sizes, decays, the
recurrence, the state and the gated norm are 32-bit in both run types; what leaves the convolutions is rounded to the run's
element type in a prompt step and stays 32-bit in a decode step.  A decode step is one launch from the projections to y;
prompts of a bfloat16 run go through the chunked form on the tensor cores, other steps through the scan that walks the
tokens in order.
"""
from __future__ import annotations

import torch

from ..cache import StateRequest
from ..errors import UnsupportedModel
from ..kernels import ops
from ..weights.params import ParamSpec
from .base import Mixer, register_mixer

MAX_STATE = 512        # the scan kernel spreads a column's rows over the 32 lanes of a warp, 16 rows a lane
MAX_TAPS = 32
CHUNKS_FROM_TOKENS = 16    # new tokens per sequence from which a prompt step of a bfloat16 run goes in chunks


@register_mixer("state_space")
class StateSpace(Mixer):
    accepts_deferred_norm = True    # x goes to Runtime.linear alone

    def __init__(self, spec, reads_other_cache: bool = False):
        if reads_other_cache:
            raise UnsupportedModel(f"{spec.name}: a recurrent mixer keeps no keys and values that another layer could read")
        if spec.state > MAX_STATE:
            raise UnsupportedModel(f"{spec.name}: states of {spec.state} rows (at most {MAX_STATE})")
        if not 1 <= spec.conv <= MAX_TAPS:
            raise UnsupportedModel(f"{spec.name}: convolutions of {spec.conv} taps (1 to {MAX_TAPS})")
        if spec.n_heads % spec.n_groups:
            raise UnsupportedModel(f"{spec.name}: {spec.n_heads} heads over {spec.n_groups} groups")
        s = self.spec = spec
        self.inner = s.n_heads * s.value_dim
        if self.inner % s.norm_groups:
            raise UnsupportedModel(f"{spec.name}: a norm of {self.inner} lanes in {s.norm_groups} parts")
        self.channels = self.inner + 2 * s.n_groups * s.state           # what the convolutions run over
        self.proj_size = self.inner + self.channels + s.n_heads
        self.padded_size = (self.proj_size + 7) // 8 * 8
        self.sizes = (s.n_heads, s.value_dim, s.n_groups, s.state, s.conv)
        self.state_floats = s.n_heads * s.state * s.value_dim

    def state_request(self):
        return StateRequest((ops.ssm_state_floats(*self.sizes),), torch.float32)

    def params(self):
        s = self.spec
        return [ParamSpec(f"{s.name}.in", (self.proj_size, s.hidden_size)),
                ParamSpec(f"{s.name}.conv", (self.channels, s.conv), init=("normal", 0.5)),
                ParamSpec(f"{s.name}.conv.b", (self.channels,), init=("normal", 0.1)),
                ParamSpec(f"{s.name}.dt_bias", (s.n_heads,), init=("normal", 0.5)),
                ParamSpec(f"{s.name}.A_log", (s.n_heads,), init=("normal", 0.5)),
                ParamSpec(f"{s.name}.D", (s.n_heads,), init=("one_plus_normal", 0.1)),
                ParamSpec(f"{s.name}.norm", (self.inner,), init=("one_plus_normal", 0.1)),
                ParamSpec(f"{s.name}.o", (s.hidden_size, self.inner))]

    def bind(self, tensors, rt):
        s, self.rt = self.spec, rt
        w = tensors.pop(f"{s.name}.in")
        pad = self.padded_size - self.proj_size
        self.w_in = torch.cat([w, w.new_zeros(pad, w.shape[1])], dim=0).contiguous() if pad else w
        self.w_conv, self.b_conv = tensors[f"{s.name}.conv"].contiguous(), tensors[f"{s.name}.conv.b"]
        # the per-head numbers enter 32-bit arithmetic
        self.dt_bias, self.a_log, self.d_skip = (tensors[f"{s.name}.{n}"].to(torch.float32).contiguous()
                                                 for n in ("dt_bias", "A_log", "D"))
        self.w_norm, self.w_o = tensors[f"{s.name}.norm"], tensors[f"{s.name}.o"]

    def weight_bytes(self):
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_conv, self.w_o))

    def forward(self, ctx, x, residual, cache):
        s, rt = self.spec, self.rt
        n, H = x.shape[0], s.n_heads
        proj = rt.empty(n, self.padded_size, dtype=torch.float32)
        with rt.phase("ssm_in", self.w_in, n):
            rt.linear(x, self.w_in, None, proj)
        y = rt.empty(n, self.inner, dtype=torch.float32)
        state_bytes = 8.0 * ctx.n_seqs * self.state_floats              # read and written once a step
        flops = 5.0 * n * self.state_floats
        if ctx.is_decode:
            with rt.phase("ssm_scan", nbytes=state_bytes + 4.0 * (proj.numel() - n * self.inner + y.numel()), flops=flops):
                ops.ssm_step(proj, self.w_conv, self.b_conv, cache.state, ctx.tok_pos, ctx.seq_slots, self.dt_bias,
                             self.a_log, self.d_skip, y, self.sizes)
        else:
            xc = rt.empty(n, ops.ssm_row(*self.sizes[:4]))
            gd = rt.empty(n, 2 * H, dtype=torch.float32)
            with rt.phase("ssm_conv", nbytes=4.0 * n * (self.channels + H) + xc.numel() * xc.element_size()):
                ops.ssm_conv(proj, self.w_conv, self.b_conv, cache.state, ctx.tok_seq, ctx.tok_pos, ctx.seq_slots,
                             ctx.cu_seqlens, self.dt_bias, self.a_log, xc, gd, self.sizes)
            with rt.phase("ssm_scan", nbytes=state_bytes + xc.numel() * xc.element_size() + 4.0 * y.numel(), flops=flops):
                # prompts of a bfloat16 run in chunks on the tensor cores; a few tokens per sequence, and a float32 run, in order
                chunks = (xc.dtype == torch.bfloat16 and s.state <= ops.SSM_CHUNK_MAX_STATE
                          and n >= CHUNKS_FROM_TOKENS * ctx.n_seqs)
                scan = ops.ssm_chunk_scan if chunks else ops.ssm_scan
                scan(proj, xc, gd, cache.state, ctx.seq_slots, ctx.cu_seqlens, ctx.tok_pos, self.d_skip, y, ctx.n_seqs,
                     self.sizes)
        gated = rt.empty(n, self.inner)
        with rt.phase("ssm_gate", nbytes=8.0 * y.numel() + gated.numel() * gated.element_size()):
            ops.ssm_gated_norm(y, proj, self.w_norm, s.eps, gated, s.norm_groups)
        with rt.phase("ssm_out", self.w_o, n):
            rt.linear(gated, self.w_o, None, residual, accumulate=not getattr(ctx, "branch_is_fresh", False),
                      then_norm=getattr(ctx, "next_norm", None))
