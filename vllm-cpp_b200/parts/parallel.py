"""Two mixers side by side: both read the same input, and the layer's result is
``left_scale * left(x) + right_scale * right(x)``, with ``result_eps`` each of the two first RMS-normed over the model's
width with a gain of its own (tensors ``left.out`` and ``right.out``).  The members are any registered mixers (PartSpecs);
their tensors sit under ``left.`` and ``right.``, and each keeps the cache it would keep alone: the pair declares a
CompositeSpec and hands each member its own view.  Members that both offer ``forward_projected`` share one input product.
An arrangement that norms and adds a sublayer's result itself may take the two results as they are (``pair_result``,
``forward_pair``) and join them in its own kernel.  The reference has no such part.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..config.model_spec import PartSpec
from ..csrc import ops
from .base import MIXERS, CompositeSpec, Mixer, ParamSpec, build_part, register_mixer, workspace_piece


@register_mixer("parallel")
class ParallelMixers(Mixer):
    def __init__(self, hidden_size: int, left: PartSpec, right: PartSpec, left_scale: float, right_scale: float, dtype, device,
                 result_eps: Optional[float] = None):
        if result_eps is not None and not result_eps > 0:
            raise ValueError("parallel: result_eps must be positive")
        self.hidden, self.dtype, self.result_eps = hidden_size, dtype, result_eps
        self.w_left = self.w_right = None         # gains of the norms on the results
        self.w_in = None                          # the members' shared input product, left rows first
        self.left = build_part(MIXERS, "mixer", left, dtype=dtype, device=device)
        self.right = build_part(MIXERS, "mixer", right, dtype=dtype, device=device)
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)

    def members(self):
        return (("left.", self.left), ("right.", self.right))

    def param_specs(self) -> Dict[str, ParamSpec]:
        out = {prefix + name: ps for prefix, m in self.members() for name, ps in m.param_specs().items()}
        if self.result_eps is not None:
            out.update({prefix + "out": ParamSpec((self.hidden,), "gain") for prefix, _ in self.members()})
        return out

    def load_params(self, tensors):
        for prefix, m in self.members():
            m.load_params({name: tensors[prefix + name] for name in m.param_specs()})
        if self.result_eps is not None:
            self.w_left, self.w_right = tensors["left.out"].contiguous(), tensors["right.out"].contiguous()
        if all(hasattr(m, "forward_projected") for _, m in self.members()):
            self.w_in = torch.cat([self.left.w_in, self.right.w_in], dim=0).contiguous()
            self.left.w_in = self.right.w_in = None

    def product_weights(self):
        return ([(self.w_in, 0)] if self.w_in is not None else []) + [pw for _, m in self.members() for pw in m.product_weights()]

    def step_arrays(self):
        out = {}
        for _, m in self.members():
            out.update(m.step_arrays())
        return out

    def reserve(self, n_tokens, n_reqs, device):
        for _, m in self.members():
            m.reserve(n_tokens, n_reqs, device)

    def cache_spec(self):
        return CompositeSpec((self.left.cache_spec(), self.right.cache_spec()))

    def workspace_bytes(self, n_tokens, n_reqs):
        shared = sum(m.in_width() for _, m in self.members()) if all(hasattr(m, "forward_projected") for _, m in self.members()) else 0
        return (2 * workspace_piece((n_tokens, self.hidden), self.dtype) + workspace_piece((n_tokens, shared), self.dtype)
                + max(m.workspace_bytes(n_tokens, n_reqs) for _, m in self.members()))

    def pair_result(self):
        """(left gain, right gain, left scale, right scale, eps) of the norms with which the two results are joined, for an
        arrangement that joins them itself; None if they are added as they are."""
        if self.result_eps is None:
            return None
        return self.w_left, self.w_right, self.left_scale, self.right_scale, self.result_eps

    def plain_scales(self):
        """(left scale, right scale) if the two results are added as they are, for an arrangement whose norm kernel joins them
        itself; None if they are normed first."""
        return (self.left_scale, self.right_scale) if self.result_eps is None else None

    def forward_pair(self, x, a, b, step, cache, writes_cache, ws):
        """The two members' results as they are."""
        if self.w_in is None:
            self.left.forward(x, a, step, cache.views[0], writes_cache, ws)
            self.right.forward(x, b, step, cache.views[1], writes_cache, ws)
            return
        mark = ws.mark()
        proj = ws.take((x.shape[0], self.w_in.shape[0]), self.dtype)
        ops.linear(x, self.w_in, proj)
        split = self.left.in_width()
        self.left.forward_projected(proj[:, :split], a, step, cache.views[0], writes_cache, ws)
        self.right.forward_projected(proj[:, split:], b, step, cache.views[1], writes_cache, ws)
        ws.release(mark)

    def forward(self, x, out, step, cache, writes_cache, ws):
        mark = ws.mark()
        n = x.shape[0]
        a = ws.take((n, self.hidden), self.dtype)
        b = ws.take((n, self.hidden), self.dtype)
        self.forward_pair(x, a, b, step, cache, writes_cache, ws)
        if self.result_eps is None:
            ops.scaled_sum(a, b, out, self.left_scale, self.right_scale)
        else:
            ops.pair_norm(a, b, self.w_left, self.w_right, self.left_scale, self.right_scale, self.result_eps, out)
        ws.release(mark)
