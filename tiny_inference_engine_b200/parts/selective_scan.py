"""A selective scan: a recurrent mixer with a diagonal state per channel whose decay and input depend on the token.

    [x | z]     = h Win^T                                    x, z: `inner_size` each
    x           = silu(conv(x) + b_conv)                     a short causal convolution per channel over time
    [dt | B | C] = x Wx^T                                    dt: `dt_rank`; B, C: `state_size`
    dt          = softplus(dt Wdt^T + b_dt)                  one per channel
    S[c, n]    <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n   A = -exp(A_log), inner x state
    y_c         = sum_n S[c, n] C_n + D_c x_c
    out         = (y * silu(z)) Wo^T

S is float32 and starts at zero. A request's state is one float32 row in a state slot: S, then the convolution's last
`conv_taps - 1` inputs. The step sizes' second projection writes float32, and what enters the recurrence behind the
projections and the convolution (step sizes, decays, S, the read-out and its gate) is float32 in either compute dtype.
Sections of the products start at multiples of 8 columns.
"""
from __future__ import annotations

import math

import torch

from .. import ops
from ..errors import InvalidArgument
from ..weights.loader import TensorNeed
from .base import Mixer, StateNeed, register_part, to_compute


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


class SelectiveScan(Mixer):
    launches_only = False
    graph_safe = True       # the kernels read the step from device tensors only and skip sequences without a slot

    def __init__(self, spec, dtype, prefix: str = ""):
        p = spec.params
        self.prefix = prefix + p.get("prefix", "")
        self.hidden, self.inner = int(p["hidden_size"]), int(p["inner_size"])
        self.rank, self.states = int(p["dt_rank"]), int(p["state_size"])
        self.taps = int(p.get("conv_taps", 1))
        if min(self.inner, self.rank) <= 0 or not 1 <= self.taps <= 16 or not 0 < self.states <= 256:
            raise InvalidArgument(f"selective scan: bad sizes inner={self.inner} dt rank={self.rank} states={self.states} (1 to 256) "
                                  f"taps={self.taps} (1 to 16)")
        self.dtype = dtype
        self.z_off = _up8(self.inner)                   # columns of the input product
        self.width = 2 * self.z_off
        self.rank8 = _up8(self.rank)                    # columns of the second product: dt, B, C
        self.b_off = self.rank8
        self.c_off = self.b_off + _up8(self.states)
        self.low_width = self.c_off + _up8(self.states)
        self.state_floats = self.inner * self.states    # S; the convolution's inputs follow

    def _name(self, leaf):
        return self.prefix + leaf

    def needs(self):
        D, n, I, N = self.hidden, self._name, self.inner, self.states
        return {n("in"): TensorNeed((2 * I, D)), n("conv"): TensorNeed((I, self.taps)), n("conv.b"): TensorNeed((I,), "norm"),
                n("x"): TensorNeed((self.rank + 2 * N, I)), n("dt"): TensorNeed((I, self.rank)), n("dt.b"): TensorNeed((I,), "norm"),
                n("A_log"): TensorNeed((I, N), "norm"), n("D"): TensorNeed((I,), "norm"), n("o"): TensorNeed((D, I))}

    def bind(self, get):
        n, I, N = self._name, self.inner, self.states
        w_in = to_compute(get(n("in")), self.dtype)
        stacked = torch.zeros((self.width, self.hidden), dtype=self.dtype, device=w_in.device)
        stacked[:I], stacked[self.z_off:self.z_off + I] = w_in[:I], w_in[I:]
        self.gemm_in = ops.bound_gemm(stacked, split_many=False)
        self.w_in = self.gemm_in.w
        w_x = to_compute(get(n("x")), self.dtype)
        low = torch.zeros((self.low_width, I), dtype=self.dtype, device=w_x.device)
        low[:self.rank] = w_x[:self.rank]
        low[self.b_off:self.b_off + N] = w_x[self.rank:self.rank + N]
        low[self.c_off:self.c_off + N] = w_x[self.rank + N:]
        self.gemm_x = ops.bound_gemm(low, split_many=True)
        self.w_x = self.gemm_x.w
        w_dt = to_compute(get(n("dt")), self.dtype)
        padded = torch.zeros((I, self.rank8), dtype=self.dtype, device=w_dt.device)      # k padded to the section's width
        padded[:, :self.rank] = w_dt
        self.gemm_dt = ops.bound_gemm(padded, split_many=False)
        self.w_dt = self.gemm_dt.w
        self.gemm_o = ops.bound_gemm(to_compute(get(n("o")), self.dtype).contiguous(), split_many=True)
        self.w_o = self.gemm_o.w
        f32 = lambda leaf: get(n(leaf)).to(torch.float32).contiguous()
        self.conv_w = f32("conv").t().contiguous()        # [taps, inner]: a tap of every channel side by side
        self.conv_b, self.dt_b, self.skip = f32("conv.b"), f32("dt.b"), f32("D")
        # exp(dt A) = exp2(dt A log2 e): the factor is formed once, in float64
        self.a2 = (-torch.exp(get(n("A_log")).to(torch.float64)) * math.log2(math.e)).to(torch.float32).contiguous()
        self._capacity = None

    def state_need(self):
        return StateNeed((self.state_floats + (self.taps - 1) * self.inner,), torch.float32)

    def forward(self, h, ctx, cache, state):
        T, I = h.shape[0], self.inner
        if state is None:
            raise InvalidArgument("the selective scan needs state slots (make the cache with `make_cache`)")
        proj = ctx.ws.rows("scan.proj", T, self.width, self.dtype)
        self.gemm_in(h, proj)
        x = ctx.ws.rows("scan.x", T, I, self.dtype)
        ops.short_conv_act(proj, 0, self.conv_w, self.conv_b, state, self.state_floats, ctx, x)
        low = ctx.ws.rows("scan.low", T, self.low_width, self.dtype)
        self.gemm_x(x, low)
        raw = ctx.ws.rows("scan.dt", T, I, torch.float32)
        self.gemm_dt(low[:, :self.rank8], raw)
        y = ctx.ws.rows("scan.y", T, I, self.dtype)
        ops.selective_scan(x, proj[:, self.z_off:self.z_off + I], low, self.b_off, self.c_off, raw, self.dt_b, self.a2, self.skip, state, ctx, y)
        out = ctx.ws.rows("mixer.out", T, self.hidden, self.dtype)
        if self._capacity is None:
            self._capacity = ops.partial_capacity(ctx.ws.max_rows, self.gemm_o.N, self.gemm_o.K)
        return self.gemm_o(y, out, lambda m: ctx.ws.flat("mixer.out.partial", m, torch.float32, self._capacity))


register_part("mixer", "selective_scan", SelectiveScan, replace=True)
