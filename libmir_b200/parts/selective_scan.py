"""A selective state-space mixer (Mamba): a diagonal recurrence whose step size, input vector and read-out vector are
functions of the token.

With h the mixer's input [T, hidden], I channels and N state numbers per channel:
    [x' | z] = W_in h                                    I numbers each
    x   = silu(conv(x') + b_conv)                        causal per-channel convolution over the request's own tokens,
                                                         zeros before its start
    [r | B | C] = W_x x                                  dt_rank, N and N numbers
    dt  = softplus(W_dt r + b_dt)                        one step size per channel
    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n  A = -exp(A_log)
    y_c = sum_n S[c, n] C_n + D_c x_c
    out = W_o (y * silu(z))
Per request the mixer keeps two fixed-size states in the request's slot: S (32-bit, [I, N]) and the last taps - 1 inputs
of the convolution.  The product with W_dt leaves 32-bit numbers; the softplus, the exponentials, the state and its sums
are 32-bit (csrc/selective_scan.cu), and the read-out, the term with D and the gate leave that kernel as the input of
the last product.  Channels, dt_rank and N are padded to multiples of eight with zero weights so that every view starts
on a 16-byte boundary.
"""

from __future__ import annotations

import math

import torch

from .. import kernels
from ..config.spec import CacheBundle, FixedState, ParamSpec
from .base import Mixer


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class SelectiveScan(Mixer):
    graph_safe = True          # the batch is read from device tensors only; padding rows (position < 0) are skipped
    takes_normed_residual = True   # x is used by one product only, which can take a folded norm over

    def __init__(self, spec, env):
        super().__init__(spec, env)
        s = spec
        if min(s.inner, s.state, s.dt_rank, s.conv_taps) <= 0:
            raise ValueError("a selective scan needs inner, state, dt_rank and conv_taps above zero")
        if s.state > kernels.SELECTIVE_SCAN_MAX_STATE or s.conv_taps > 16:
            raise ValueError(f"the kernels take up to {kernels.SELECTIVE_SCAN_MAX_STATE} state numbers a channel and 16 taps")
        self.channels = _pad8(s.inner)
        self.rank = _pad8(s.dt_rank)
        self.columns = _pad8(s.state)            # of B and of C in a packed row of the second product
        self.w_in = self.w_x = self.w_dt = self.w_o = self.w_conv = None
        self.conv_bias = self.dt_bias = self.rates = self.skip = None

    def cache_requirement(self):
        s = self.spec
        return CacheBundle(None, (FixedState((self.channels, s.state), "float32"),
                                  FixedState((s.conv_taps - 1, self.channels), "float32")))

    def parameters(self):
        s = self.spec
        matrix = lambda rows, columns: ParamSpec((rows, columns), accept_transposed=False)
        return {
            "in": matrix(2 * s.inner, s.hidden_size),
            "conv": matrix(s.inner, s.conv_taps), "conv.b": ParamSpec((s.inner,), init="zeros", store="float32"),
            "x": matrix(s.dt_rank + 2 * s.state, s.inner),
            "dt": matrix(s.inner, s.dt_rank), "dt.b": ParamSpec((s.inner,), init="zeros", store="float32"),
            "A_log": ParamSpec((s.inner, s.state), init="zeros", store="float32", accept_transposed=False),
            "D": ParamSpec((s.inner,), init="ones", store="float32"),
            "o": matrix(s.hidden_size, s.inner),
        }

    def bind(self, tensors):
        s = self.spec

        def placed(shape, pieces):
            """A zero tensor with (rows, columns, source) pieces written into its corner at (rows, columns)."""
            out = torch.zeros(shape, dtype=pieces[0][2].dtype, device=pieces[0][2].device)
            for row, column, source in pieces:
                view = out[row:row + source.shape[0]]
                if source.dim() == 2:
                    view = view[:, column:column + source.shape[1]]
                view.copy_(source)
            return out
        inner, channels, n, rank = s.inner, self.channels, s.state, s.dt_rank
        w_in, w_x = tensors["in"], tensors["x"]
        self.w_in = placed((2 * channels, s.hidden_size), [(0, 0, w_in[:inner]), (channels, 0, w_in[inner:])])
        self.w_conv = placed((channels, s.conv_taps), [(0, 0, tensors["conv"])])
        self.conv_bias = placed((channels,), [(0, 0, tensors["conv.b"])])
        self.w_x = placed((self.rank + 2 * self.columns, channels),
                          [(0, 0, w_x[:rank]), (self.rank, 0, w_x[rank:rank + n]),
                           (self.rank + self.columns, 0, w_x[rank + n:])])
        self.w_dt = placed((channels, self.rank), [(0, 0, tensors["dt"])])
        self.dt_bias = placed((channels,), [(0, 0, tensors["dt.b"])])
        # what the kernel raises two to, per unit of the step size: A log2(e)
        self.rates = placed((channels, n), [(0, 0, (-torch.exp(tensors["A_log"].double()) / math.log(2.0)).float())])
        self.skip = placed((channels,), [(0, 0, tensors["D"])])
        self.w_o = placed((s.hidden_size, channels), [(0, 0, tensors["o"])])

    def weight_bytes(self):
        tensors = (self.w_in, self.w_conv, self.conv_bias, self.w_x, self.w_dt, self.dt_bias, self.rates, self.skip, self.w_o)
        return sum(t.numel() * t.element_size() for t in tensors)

    def forward(self, ctx, cache, x, residual, overwrite=False):
        """residual += W_o (...) (or residual = with `overwrite`, for an arrangement that norms the branch's result)."""
        tokens, dtype = residual.shape[0], self.env.dtype
        state, tail = cache.states[0], cache.states[1]
        packed = ctx.alloc((tokens, 2 * self.channels), dtype)
        kernels.linear(x, self.w_in, packed, alloc=ctx.alloc)
        convolved = ctx.alloc((tokens, self.channels), dtype)
        kernels.short_conv_silu(packed[:, :self.channels], self.w_conv, tail, ctx.row_of_token, ctx.query_starts,
                                ctx.state_slots, ctx.positions, convolved, bias=self.conv_bias,
                                single_tokens_only=ctx.decode_only)
        low = ctx.alloc((tokens, self.w_x.shape[0]), dtype)
        kernels.linear(convolved, self.w_x, low, alloc=ctx.alloc)
        step = ctx.alloc((tokens, self.channels), torch.float32)          # 32-bit: it enters the recurrence
        kernels.linear(low[:, :self.rank], self.w_dt, step, alloc=ctx.alloc)
        mixed = ctx.alloc((tokens, self.channels), dtype)
        kernels.selective_scan(convolved, step, self.dt_bias, low[:, self.rank:self.rank + self.columns],
                               low[:, self.rank + self.columns:], packed[:, self.channels:], self.rates, self.skip, state,
                               ctx.query_starts, ctx.state_slots, ctx.positions, mixed)
        if overwrite:
            kernels.linear(mixed, self.w_o, residual, alloc=ctx.alloc)
        else:
            ctx.accumulate(mixed, self.w_o, residual)
