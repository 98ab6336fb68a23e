"""A selective state space as a mixer: per channel a vector of ``state`` numbers whose decay, drive and read-out follow the token.

    [x | z] = W_in h (``inner`` channels each);   x = silu(conv(x) + b)          a causal convolution over time per channel (``taps``)
    [low | b | b'] = W_x x (``dt_rank``, ``state``, ``state``);   dt = softplus(W_dt low + b_dt), a step size per channel
    per channel, with its row a = -e^(A_log) and its number d:   s <- e^(dt a) * s + (dt x) b  (elementwise);   y = b'.s + d x
    out = W_o (y * silu(z))

The state S (float32 [inner, state]) and the convolution's last taps - 1 inputs live in slots of the cache manager, zero at
admission, are read at the start of a request's portion and left at its end, so a prompt may be cut anywhere.  Step sizes, decays,
state and sums are float32 in both precisions (csrc/selective_scan.cu).  The reference has no recurrent mixer
(src/layers/attention.cpp is its only one).
"""
from __future__ import annotations

import math
from typing import Dict

import torch

from ..csrc import ops
from .base import CompositeSpec, Mixer, ParamSpec, StateSpec, register_mixer, workspace_piece


@register_mixer("selective_state")
class SelectiveStateSpace(Mixer):
    def __init__(self, hidden_size: int, inner: int, state: int, dt_rank: int, taps: int, dtype, device):
        if min(hidden_size, inner, state, dt_rank) <= 0:
            raise ValueError("selective_state: sizes must be positive")
        if state > ops.SELECTIVE_MAX_STATE:
            raise ValueError(f"selective_state: up to {ops.SELECTIVE_MAX_STATE} state numbers a channel, got {state}")
        if not 1 <= taps <= ops.CONV_MAX_TAPS:
            raise ValueError(f"selective_state: a convolution of 1 to {ops.CONV_MAX_TAPS} taps, got {taps}")
        self.hidden, self.inner, self.N, self.rank, self.taps = hidden_size, inner, state, dt_rank, taps
        self.dtype, self.device = dtype, device
        self.w_in = self.w_x = self.w_dt = self.w_o = self.conv = self.conv_b = self.dt_b = self.a_log2 = self.skip = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        I, N, R = self.inner, self.N, self.rank
        return {"in": ParamSpec((2 * I, self.hidden)), "conv": ParamSpec((I, self.taps), "bias"), "conv.b": ParamSpec((I,), "bias"),
                "x": ParamSpec((R + 2 * N, I)), "dt": ParamSpec((I, R)), "dt.b": ParamSpec((I,), "bias"),
                "A_log": ParamSpec((I, N), "bias"), "D": ParamSpec((I,), "gain"), "o": ParamSpec((self.hidden, I))}

    def load_params(self, t):
        self.w_in, self.w_x, self.w_dt, self.w_o = (t[n].contiguous() for n in ("in", "x", "dt", "o"))
        self.conv, self.conv_b, self.dt_b, self.skip = (t[n].contiguous() for n in ("conv", "conv.b", "dt.b", "D"))
        # the kernel's exponentials are powers of two
        self.a_log2 = (-torch.exp(t["A_log"].double()) * math.log2(math.e)).float().contiguous()

    def product_weights(self):
        return [(w, 0) for w in (self.w_in, self.w_x, self.w_dt, self.w_o) if w is not None]

    def cache_spec(self):
        return CompositeSpec((StateSpec((self.inner, self.N), torch.float32), StateSpec((max(1, self.taps - 1), self.inner), torch.float32)))

    def workspace_bytes(self, n_tokens, n_reqs):
        return (workspace_piece((n_tokens, 2 * self.inner), self.dtype) + 3 * workspace_piece((n_tokens, self.inner), self.dtype)
                + workspace_piece((n_tokens, self.rank + 2 * self.N), self.dtype))

    def in_width(self) -> int:
        return 2 * self.inner

    def forward(self, x, out, step, cache, writes_cache, ws):
        mark = ws.mark()
        proj = ws.take((x.shape[0], 2 * self.inner), self.dtype)
        ops.linear(x, self.w_in, proj)
        self.forward_projected(proj, out, step, cache, writes_cache, ws)
        ws.release(mark)

    def forward_projected(self, proj, out, step, cache, writes_cache, ws):
        """``forward`` from the rows [x | z] of the input product on (a mixer that shares its input product calls this)."""
        n, I, R, N = proj.shape[0], self.inner, self.rank, self.N
        states, window = cache.views
        mark = ws.mark()
        x = ws.take((n, I), self.dtype)
        ops.causal_conv(proj[:, :I], self.conv, window.slots, x, step.q_start, step.state_slots, step.n_reqs, step.max_q_len,
                        bias=self.conv_b, act="silu")
        low = ws.take((n, R + 2 * N), self.dtype)
        ops.linear(x, self.w_x, low)
        dt = ws.take((n, I), self.dtype)
        ops.linear(low[:, :R], self.w_dt, dt)
        y = ws.take((n, I), self.dtype)
        ops.selective_scan(x, dt, low[:, R: R + N], low[:, R + N:], proj[:, I:], self.dt_b, self.a_log2, self.skip, states.slots, y,
                           step.q_start, step.state_slots, step.n_reqs, step.max_q_len)
        ops.linear(y, self.w_o, out)
        ws.release(mark)
