"""A state space as a mixer whose memory is a matrix per head that decays by one number per token, in the form that is also a masked
attention (state-space duality):

    [z | x | B | C | dt] = W_in h              ``inner`` = heads * v_head_dim channels each of z and x, groups * state each of B and C,
                                               a number per head of dt
    [x | B | C] = silu(conv(.) + b)            a causal convolution over time per channel (``taps``)
    dt = softplus(dt + dt_bias)                a step size per head
    per head h (group h // (heads / groups)):  S <- exp(-e^(A_log_h) dt_h) S + B (dt_h x_h)^T,   y_h = S^T C + D_h x_h
    out = W_o (rms(y * silu(z)) * w)           the gate first, then the norm, in ``norm_groups`` equal parts of the channels

The state S (float32 [heads, state, v_head_dim]) and the convolution's last taps - 1 inputs live in slots of the cache manager, zero
at admission, are read at the start of a request's portion and left at its end, so a prompt may be cut anywhere.  Step sizes, decays,
state and sums are float32 in both precisions (csrc/state_dual.cu: single tokens are walked, bfloat16 portions run on tensor cores in
chunks).  The reference has no recurrent mixer (src/layers/attention.cpp is its only one).
"""
from __future__ import annotations

import math
from typing import Dict

import torch

from ..csrc import ops
from .base import CompositeSpec, Mixer, ParamSpec, StateSpec, register_mixer, workspace_piece


@register_mixer("state_dual")
class StateSpaceDual(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, v_head_dim: int, state: int, groups: int, taps: int, norm_groups: int, eps: float,
                 dtype, device):
        if min(hidden_size, num_heads, v_head_dim, state, groups, norm_groups) <= 0 or not eps > 0:
            raise ValueError("state_dual: sizes and eps must be positive")
        if num_heads % groups:
            raise ValueError(f"state_dual: {num_heads} heads cannot share {groups} groups")
        if (num_heads * v_head_dim) % norm_groups:
            raise ValueError(f"state_dual: {num_heads * v_head_dim} channels cannot be normed in {norm_groups} equal parts")
        if state > ops.STATE_DUAL_MAX_STATE:
            raise ValueError(f"state_dual: up to {ops.STATE_DUAL_MAX_STATE} state numbers, got {state}")
        if not 1 <= taps <= ops.CONV_MAX_TAPS:
            raise ValueError(f"state_dual: a convolution of 1 to {ops.CONV_MAX_TAPS} taps, got {taps}")
        self.hidden, self.H, self.P, self.N, self.G, self.taps = hidden_size, num_heads, v_head_dim, state, groups, taps
        self.inner, self.norm_groups, self.eps = num_heads * v_head_dim, norm_groups, float(eps)
        self.channels = self.inner + 2 * groups * state                 # what the convolution runs over
        self.dtype, self.device = dtype, device
        self.w_in = self.w_o = self.conv = self.conv_b = self.dt_b = self.a_log2 = self.skip = self.w_norm = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        H = (self.H,)
        return {"in": ParamSpec((self.in_width(), self.hidden)), "conv": ParamSpec((self.channels, self.taps), "bias"),
                "conv.b": ParamSpec((self.channels,), "bias"), "dt_bias": ParamSpec(H, "bias"), "A_log": ParamSpec(H, "bias"),
                "D": ParamSpec(H, "gain"), "norm": ParamSpec((self.inner,), "gain"), "o": ParamSpec((self.hidden, self.inner))}

    def load_params(self, t):
        self.w_in, self.w_o = t["in"].contiguous(), t["o"].contiguous()
        self.conv, self.conv_b, self.dt_b, self.skip, self.w_norm = (t[n].contiguous() for n in ("conv", "conv.b", "dt_bias", "D", "norm"))
        # the kernel's decays are powers of two
        self.a_log2 = (-torch.exp(t["A_log"].double()) * math.log2(math.e)).float().contiguous()

    def product_weights(self):
        return [(w, 0) for w in (self.w_in, self.w_o) if w is not None]

    def cache_spec(self):
        return CompositeSpec((StateSpec((self.H, self.N, self.P), torch.float32), StateSpec((max(1, self.taps - 1), self.channels), torch.float32)))

    def in_width(self) -> int:
        return self.inner + self.channels + self.H

    def workspace_bytes(self, n_tokens, n_reqs):
        return (workspace_piece((n_tokens, self.in_width()), self.dtype) + workspace_piece((n_tokens, self.channels), self.dtype)
                + workspace_piece((n_tokens, self.inner), torch.float32) + workspace_piece((n_tokens, self.inner), self.dtype))

    def forward(self, x, out, step, cache, writes_cache, ws):
        mark = ws.mark()
        proj = ws.take((x.shape[0], self.in_width()), self.dtype)
        ops.linear(x, self.w_in, proj)
        self.forward_projected(proj, out, step, cache, writes_cache, ws)
        ws.release(mark)

    def forward_projected(self, proj, out, step, cache, writes_cache, ws):
        """``forward`` from the rows [z | x | B | C | dt] of the input product on (a mixer that shares its input product calls this)."""
        n, I, C, GN = proj.shape[0], self.inner, self.channels, self.G * self.N
        states, window = cache.views
        mark = ws.mark()
        u = ws.take((n, C), self.dtype)
        ops.causal_conv(proj[:, I: I + C], self.conv, window.slots, u, step.q_start, step.state_slots, step.n_reqs, step.max_q_len,
                        bias=self.conv_b, act="silu")
        y = ws.take((n, I), torch.float32)
        ops.state_dual(u[:, :I], u[:, I: I + GN], u[:, I + GN:], proj[:, I + C: I + C + self.H], self.dt_b, self.a_log2, self.skip, states.slots, y,
                       step.q_start, step.state_slots, step.n_reqs, step.max_q_len, num_groups=self.G)
        gated = ws.take((n, I), self.dtype)
        ops.gated_group_norm(y, proj[:, :I], self.w_norm, gated, group=I // self.norm_groups, eps=self.eps, gate_act="silu", gate_first=True)
        ops.linear(gated, self.w_o, out)
        ws.release(mark)
