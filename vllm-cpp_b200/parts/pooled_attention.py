"""Grouped-query attention over a sliding window of tokens plus, for what lies before the window, one mean key and one mean
value per block of ``pool`` tokens:

    (q, k, v) = conv([W_q; W_k; W_v] h + b)                                  a causal convolution over time per channel (``taps``)
    q, k rotated by position on the first ``rotary_dim`` coordinates of a head (interleaved pairs; "none": no rotation)
    score = (q . k) * scale * temp[head]
    position i sees the tokens j with 0 <= i - j < window, and the block b of the positions b P .. b P + P - 1 if
    b P + P - 1 <= i - window; a block's key and value are the means of its tokens' cached keys and values.  Between the two
    lies a gap of fewer than P tokens that nothing shows.  One softmax over tokens and blocks.
    out = W_o concat_heads(.)

``window`` 0: every token is seen; ``pool`` 0: nothing before the window is.  The mixer keeps three things per request: the
window's pages (of which those of a block that is not complete yet are not given back, PagedKVSpec.keep_block), pages with a row
per complete block (PagedKVSpec.stride), and the convolutions' last inputs in a state slot.  Convolution, rotation, the
heads' factor and the cache write are one kernel, the means of the blocks a step completes a second (csrc/attention_pooled.cu),
attention the third: in bfloat16, with heads of 64 or 128 and keys as wide as values, the tensor-core kernels of
csrc/attention_mma.cu, which walk the tiles of block rows before the tiles of tokens and take the softmax weights as two
bfloat16 terms; else the plain kernel.  The reference's attention (src/layers/attention.cpp) has a rotation and none of the rest.
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config.model_spec import PartSpec
from ..csrc import ops
from .attention import PagedAttentionKernels
from .base import POSITION_ENCODINGS, CompositeSpec, PagedKVSpec, ParamSpec, StateSpec, build_part, register_mixer, workspace_piece


@register_mixer("pooled_window_attention")
class PooledWindowAttention(PagedAttentionKernels):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int, taps: int, scale: float,
                 window: int, pool: int, position: PartSpec, dtype, device, qkv_bias: bool = True, temperature: bool = True):
        if min(hidden_size, num_heads, num_kv_heads, head_dim, v_head_dim) <= 0 or num_heads % num_kv_heads:
            raise ValueError(f"pooled_window_attention: {num_heads} heads cannot share {num_kv_heads} kv heads")
        if v_head_dim > 512 or head_dim > 1024:
            raise ValueError("pooled_window_attention: head sizes up to 1024 (keys) and 512 (values)")
        if window < 0 or pool < 0 or (pool and not window):
            raise ValueError("pooled_window_attention: window and pool must not be negative, and blocks need a window")
        if not 1 <= taps <= ops.CONV_MAX_TAPS:
            raise ValueError(f"pooled_window_attention: convolutions of 1 to {ops.CONV_MAX_TAPS} taps, got {taps}")
        self.hidden, self.nh, self.nkv, self.dk, self.dv, self.taps = hidden_size, num_heads, num_kv_heads, head_dim, v_head_dim, taps
        self.row = max(head_dim, v_head_dim)
        self.d = self.row
        self.scale, self.window, self.pool = float(scale), int(window), int(pool)
        self.qkv_bias, self.temperature = bool(qkv_bias), bool(temperature)
        self.dtype, self.device = dtype, device
        self.position = build_part(POSITION_ENCODINGS, "position encoding", position, dtype=dtype, device=device)
        fused = self.position.fused()
        if fused is None or (fused["rotary_dim"] and (fused["pairing"] != 1 or not hasattr(self.position, "inv_freq"))):
            raise ValueError("pooled_window_attention: positions enter by a rotation of interleaved pairs with given frequencies, or not at all")
        if getattr(self.position, "magnitude", 1.0) != 1.0:
            raise ValueError("pooled_window_attention: a rotation whose cosine and sine carry a factor is not built")
        self.rot = int(fused["rotary_dim"])
        if self.rot > head_dim:
            raise ValueError(f"pooled_window_attention: {self.rot} rotated coordinates in heads of {head_dim}")
        self.inv_freq = self.position.inv_freq if self.rot else None
        self.w_in = self.w_o = self.bias = self.conv = self.temp = None

    @property
    def channels(self) -> int:
        return self.nh * self.dk + self.nkv * (self.dk + self.dv)

    def param_specs(self) -> Dict[str, ParamSpec]:
        sizes = {"q": self.nh * self.dk, "k": self.nkv * self.dk, "v": self.nkv * self.dv}
        specs = {}
        for name, c in sizes.items():
            specs[name] = ParamSpec((c, self.hidden))
            if self.qkv_bias:
                specs[name + ".b"] = ParamSpec((c,), "bias")
            specs[name + ".conv"] = ParamSpec((c, self.taps), "bias")
        if self.temperature:
            specs["temp"] = ParamSpec((self.nh,), "gain")
        specs["o"] = ParamSpec((self.hidden, self.nh * self.dv))
        return specs

    def load_params(self, t):
        self.w_in = torch.cat([t[n] for n in ("q", "k", "v")], dim=0).contiguous()
        self.conv = torch.cat([t[n + ".conv"] for n in ("q", "k", "v")], dim=0).contiguous()
        if self.qkv_bias:
            self.bias = torch.cat([t[n + ".b"] for n in ("q", "k", "v")]).contiguous()
        if self.temperature:
            self.temp = t["temp"].contiguous()
        self.w_o = t["o"].contiguous()
        if self.dk == self.dv:
            self.warn_if_plain()

    def tensors(self):
        return super().tensors() + self.position.tensors()

    def product_weights(self):
        return [(w, 0) for w in (self.w_in, self.w_o) if w is not None]

    def cache_spec(self):
        parts = [PagedKVSpec(self.nkv, self.row, self.window, keep_block=self.pool or 1)]
        if self.pool:
            parts.append(PagedKVSpec(self.nkv, self.row, stride=self.pool))
        parts.append(StateSpec((max(1, self.taps - 1), self.channels), torch.float32))
        return CompositeSpec(tuple(parts))

    def _tensor_core_path(self) -> bool:
        # bfloat16 heads of 64 and 128 with keys as wide as values: the tcgen05 kernel for portions, split-KV for single tokens
        return self.dk == self.dv and super()._tensor_core_path()

    def score_shaping(self):
        # the design wants its attention weights in 32-bit: the tensor-core kernels take them as two bfloat16 terms
        return {"precise_weights": True}

    def workspace_bytes(self, n_tokens, n_reqs):
        return (workspace_piece((n_tokens, self.channels), self.dtype) + workspace_piece((n_tokens, self.nh * self.dk), self.dtype)
                + workspace_piece((n_tokens, self.nh * self.dv), self.dtype))

    def in_width(self) -> int:
        return self.channels

    def forward(self, x, out, step, cache, writes_cache, ws):
        mark = ws.mark()
        proj = ws.take((x.shape[0], self.channels), self.dtype)
        ops.linear(x, self.w_in, proj)
        self.forward_projected(proj, out, step, cache, writes_cache, ws)
        ws.release(mark)

    def forward_projected(self, proj, out, step, cache, writes_cache, ws):
        """``forward`` from the rows of the input product on (a mixer that shares its input product calls this)."""
        if not writes_cache:
            raise ValueError("pooled_window_attention: a call that reads another call's cache is not built")
        n = proj.shape[0]
        mark = ws.mark()
        tokens, conv = cache.views[0], cache.views[-1]
        blocks = cache.views[1] if self.pool else None
        table = step.block_tables[tokens.group]
        pool_table = step.block_tables[blocks.group] if blocks is not None else None
        pages = tokens.pages.view(tokens.pages.shape[0], -1)
        pooled = blocks.pages.view(blocks.pages.shape[0], -1) if blocks is not None else None
        sizes = dict(num_kv_heads=self.nkv, head_dim=self.dk, v_head_dim=self.dv, row=self.row, page_size=tokens.page_size)
        q = ws.take((n, self.nh * self.dk), self.dtype)
        ops.conv_rope_cache_write(proj, self.bias, self.conv, conv.slots, self.inv_freq, self.temp, q, pages, step.q_start, step.positions,
                                  step.state_slots, table, step.n_reqs, step.max_q_len, num_heads=self.nh, **sizes)
        if blocks is not None:
            ops.pool_blocks(pages, pooled, step.q_start, step.ctx_lens, table, pool_table, step.n_reqs, step.max_q_len, pool=self.pool, **sizes)
        attn = ws.take((n, self.nh * self.dv), self.dtype)
        if self._tensor_core_path() and tokens.page_size % 8 == 0:
            self.attend(q, attn, step, tokens, table, blocks=None if blocks is None else (blocks.pages, pool_table))
        else:
            ops.attention_pooled(q, pages, pooled, attn, step.positions, step.req_of_token, table, pool_table, num_heads=self.nh,
                                 window=self.window, pool=self.pool, scale=self.scale, **sizes)
        ops.linear(attn, self.w_o, out)
        ws.release(mark)
