"""A generalised delta rule as a mixer: per head a matrix S of key channels by value channels that every token decays per
key channel, from which it removes, at a rate per key channel, what S holds under the token's unit key, and to which it adds
the outer product of its plain key and value:

    [r; k; v] = [W_r; W_k; W_v] h;   w = exp(-decay_rate * sigmoid(W_w2 tanh(W_w1 h) + w0));   a = sigmoid(W_a h + b_a)
    u = k / sqrt(sum k^2 + 1e-6) per head;   S <- diag(w) S - (a * u) (u^T S) + k v^T  (both terms of the old S);   o = S^T r
    out = W_o (rms_head(o) * norm * sigmoid(W_g h))            a gain per channel of all heads

The state lives in a slot of the cache manager (StateSpec, zero at admission), is read at the start of a request's portion and
left at its end.  Everything between the projections and o is float32 in both precisions (csrc/general_delta.cu).  The inner
width of the decay's products comes from the checkpoint's tensors.  The reference has no recurrent mixer
(src/layers/attention.cpp is its only one).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..csrc import ops
from .base import Mixer, ParamSpec, StateSpec, register_mixer, workspace_piece

DEFAULT_DECAY_RANK = 32      # inner width of the decay's two products where no checkpoint gives it (random weights)
UNIT_KEY_EPS = 1e-6


@register_mixer("general_delta")
class GeneralDeltaRule(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int, decay_rate: float, eps: float, dtype, device):
        if min(hidden_size, num_heads, head_dim, v_head_dim) <= 0:
            raise ValueError("general_delta: sizes must be positive")
        if head_dim > 1024:
            raise ValueError("general_delta: key heads of up to 1024 channels")
        if not eps > 0 or not decay_rate > 0:
            raise ValueError("general_delta: eps and decay_rate must be positive")
        self.hidden, self.H, self.dk, self.dv = hidden_size, num_heads, head_dim, v_head_dim
        self.decay_rate, self.eps = float(decay_rate), float(eps)
        self.dtype, self.device = dtype, device
        self.rank = None             # the checkpoint's tensors give it
        self.w_in = self.w_w2 = self.w_o = self.b_a = self.b_w = self.w_norm = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        kk, vv, D, R = self.H * self.dk, self.H * self.dv, self.hidden, DEFAULT_DECAY_RANK
        return {"r": ParamSpec((kk, D)), "k": ParamSpec((kk, D)), "v": ParamSpec((vv, D)), "g": ParamSpec((vv, D)),
                "a": ParamSpec((kk, D)), "a.b": ParamSpec((kk,), "bias"),
                "w1": ParamSpec((-1, D), default_shape=(R, D)), "w2": ParamSpec((kk, -1), default_shape=(kk, R)), "w0": ParamSpec((kk,), "bias"),
                "norm": ParamSpec((vv,), "gain"), "o": ParamSpec((D, vv))}

    def load_params(self, t):
        if t["w1"].shape[0] != t["w2"].shape[1]:
            raise ValueError(f"general_delta: the decay's products do not fit: w1 {tuple(t['w1'].shape)}, w2 {tuple(t['w2'].shape)}")
        self.rank = int(t["w1"].shape[0])
        self.w_in = torch.cat([t[n] for n in ("r", "k", "v", "g", "a", "w1")], dim=0).contiguous()
        self.w_w2, self.w_o = t["w2"].contiguous(), t["o"].contiguous()
        self.b_a, self.b_w, self.w_norm = t["a.b"].contiguous(), t["w0"].contiguous(), t["norm"].contiguous()

    def product_weights(self):
        return [(self.w_in, 0), (self.w_w2, 0), (self.w_o, 0)]

    def cache_spec(self):
        return StateSpec((self.H, self.dk, self.dv), torch.float32)

    def in_width(self) -> int:
        return self.H * (3 * self.dk + 2 * self.dv) + (self.rank if self.rank is not None else DEFAULT_DECAY_RANK)

    def workspace_bytes(self, n_tokens, n_reqs):
        kk, vv = self.H * self.dk, self.H * self.dv
        rank = self.rank if self.rank is not None else DEFAULT_DECAY_RANK
        return (workspace_piece((n_tokens, self.in_width()), self.dtype) + workspace_piece((n_tokens, rank), self.dtype)
                + workspace_piece((n_tokens, kk), self.dtype) + workspace_piece((n_tokens, vv), torch.float32)
                + workspace_piece((n_tokens, vv), self.dtype) + workspace_piece((ops.general_delta_work(n_tokens, self.H, self.dk, self.dv),), torch.float32))

    def forward(self, x, out, step, cache, writes_cache, ws):
        n, H, kk, vv = x.shape[0], self.H, self.H * self.dk, self.H * self.dv
        mark = ws.mark()
        proj = ws.take((n, self.in_width()), self.dtype)
        ops.linear(x, self.w_in, proj)
        r, k, v, g, a, low = torch.split(proj, (kk, kk, vv, vv, kk, self.rank), dim=1)
        act = ws.take((n, self.rank), self.dtype)
        ops.tanh_rows(low, act)
        z = ws.take((n, kk), self.dtype)
        ops.linear(act, self.w_w2, z)
        o = ws.take((n, vv), torch.float32)
        portions = step.max_q_len >= ops.DELTA_PORTIONS_FROM
        work = ws.take((ops.general_delta_work(n, H, self.dk, self.dv),), torch.float32) if portions else None
        ops.general_delta(r, k, v, a, z, self.b_a, self.b_w, cache.slots, o, step.q_start, step.state_slots, step.n_reqs, step.max_q_len,
                          num_heads=H, rate=self.decay_rate, unit_eps=UNIT_KEY_EPS, work=work)
        y = ws.take((n, vv), self.dtype)
        ops.gated_group_norm(o, g, self.w_norm, y, group=self.dv, eps=self.eps, gate_act="sigmoid")
        ops.linear(y, self.w_o, out)
        ws.release(mark)
