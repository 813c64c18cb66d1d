"""The selective scan of Mamba: a diagonal state-space recurrence whose step size and projections depend on the token.

With ``h`` the mixer's input: ``W_in h`` is ``[u' | z]`` (``inner`` channels each); u' passes a causal convolution over time per
channel (``conv`` [inner, taps], the last column the current token's, bias ``conv.b``, zeros before the sequence's start) and
silu, giving u; ``W_x u`` is ``[d | B | C]`` (``dt_rank``, ``state`` and ``state`` values); the step size per channel is
``dt = softplus(W_dt d + dt.b)``; ``A = -exp(A_log)`` [inner, state].  Per channel c and state n, with S starting at zero,

    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n          y_c = sum_n S[c, n] C_n + D_c u_c

and the mixer returns ``W_o (y * silu(z))``.

Per request two state rows, both 32-bit: S as ``[inner, padded state]`` (a power-of-two number of slices per channel, see the scan
kernel) and the convolution's last ``taps - 1`` inputs (none with one tap), so a sequence may be cut into steps anywhere.  Step
sizes leave their product in 32-bit; softplus, decays, state and read-out are 32-bit in every run.  The rows of ``W_x`` are
padded at load so that d fills a multiple of eight columns and B starts on one (``W_dt`` gets as many zero columns).
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import Mixer, ParamSpec, FixedStateNeed, StepContext
from ..registry import register_part

MAX_STATES = 128                # states per channel the scan kernel takes (csrc/selective_scan.cu)


def padded_states(states: int) -> int:
    """States of a channel's row as the scan kernel lays it out: a power-of-two number of slices of 4."""
    pad = 4
    while pad < states:
        pad *= 2
    return pad


def _up8(n: int) -> int:
    return -(-n // 8) * 8


@register_part("mixer", "selective_scan")
class SelectiveScan(Mixer):
    def __init__(self, prefix: str, d_model: int, inner: int, state: int, dt_rank: int, taps: int, names: Optional[Dict[str, str]] = None):
        super().__init__(prefix)
        self.d_model, self.inner, self.state, self.dt_rank, self.taps = int(d_model), int(inner), int(state), int(dt_rank), int(taps)
        if not 1 <= self.state <= MAX_STATES:
            raise ValueError(f"selective scan: {state} states per channel (1 to {MAX_STATES})")
        if self.taps < 1:
            raise ValueError(f"selective scan: the convolution needs at least one tap, got {taps}")
        self.names = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "x": "x", "dt": "dt", "dt_bias": "dt.b", "A_log": "A_log",
                      "D": "D", "o": "o"}
        if names:
            self.names.update(names)

    def param_specs(self):
        n, d, I, N, R = self.names, self.d_model, self.inner, self.state, self.dt_rank
        return {n["in"]: ParamSpec((2 * I, d)),
                n["conv"]: ParamSpec((I, self.taps), storage="vector", init="normal", std=0.3),
                n["conv_bias"]: ParamSpec((I,), storage="vector", init="normal", std=0.1),
                n["x"]: ParamSpec((R + 2 * N, I)), n["dt"]: ParamSpec((I, R)),
                n["dt_bias"]: ParamSpec((I,), storage="vector", init="normal", std=1.0),
                n["A_log"]: ParamSpec((I, N), storage="vector", init="normal", std=0.5),
                n["D"]: ParamSpec((I,), storage="vector", init="ones"), n["o"]: ParamSpec((d, I))}

    def load(self, params):
        n, I, N, R = self.names, self.inner, self.state, self.dt_rank
        self.w_in = params[n["in"]].contiguous()                                               # [u' | z]
        self.conv_w = params[n["conv"]].float().t().contiguous()                               # tap-major [taps, inner]: a tap's weights lie side by side
        self.conv_b = params[n["conv_bias"]].float().contiguous()
        Rp, wx, wdt = _up8(R), params[n["x"]], params[n["dt"]]
        self.col_b, self.col_c = Rp, Rp + N
        w = torch.zeros((_up8(Rp + 2 * N), I), dtype=wx.dtype, device=wx.device)               # [d | zeros | B | C | zeros]
        w[:R] = wx[:R]
        w[Rp:Rp + 2 * N] = wx[R:]
        self.w_x = w
        self.w_dt = torch.zeros((I, Rp), dtype=wdt.dtype, device=wdt.device)
        self.w_dt[:, :R] = wdt
        self.dt_b = params[n["dt_bias"]].float().contiguous()
        self.A = torch.zeros((I, padded_states(N)), dtype=torch.float32, device=wx.device)     # padded states: decay 1, no input, never read out
        self.A[:, :N] = -torch.exp(params[n["A_log"]].float())
        self.D = params[n["D"]].float().contiguous()
        self.w_out = params[n["o"]].contiguous()

    def product_weights(self):
        return [self.w_in, self.w_x, self.w_out]

    def cache_needs(self):
        needs = [FixedStateNeed((self.inner, padded_states(self.state)), "float32")]
        if self.taps > 1:
            needs.append(FixedStateNeed((self.taps - 1, self.inner), "float32"))
        return needs

    def forward(self, x: torch.Tensor, ctx: StepContext, cache) -> torch.Tensor:
        ops, I = self.ops, self.inner
        S, tail = cache[0].state, (cache[1].state if self.taps > 1 else None)
        proj = ops.linear(x, self.w_in, None)                                                  # [T, u' | z]
        lowp = x.dtype != torch.float32
        u32, u_c = ops.causal_conv(proj, 0, I, self.taps, self.conv_w, self.conv_b, tail, ctx.token_seq, ctx.query_start_loc, ctx.slot_ids,
                                   lowp, first_row=0, act="silu", want_f32=not lowp)
        u = u_c if lowp else u32
        low = ops.linear_narrow(u, self.w_x)                                                  # [T, d | B | C]
        dt = ops.linear(low[:, :self.w_dt.shape[1]], self.w_dt, None, out_dtype=torch.float32)  # [T, inner] float32
        y = ops.selective_scan(u, dt, self.dt_b, self.A, self.D, low, self.col_b, self.col_c, proj[:, I:], S, proj, tail, self.taps,
                               ctx.query_start_loc, ctx.slot_ids, ctx.num_seqs, self.state)
        return ops.linear(y, self.w_out, None, partial_ok=True)
