"""Mixture-of-experts feed-forward: a router chooses ``top`` of ``experts`` gated feed-forward layers per token.

Router (fp32 logits ``z = W_r h``, plus a bias with ``router_bias``): ``router="sigmoid"`` — ``s = sigmoid(z)``, the ``top``
largest scores, weights ``s_k / (Σ_chosen s + 1e-20) · scale``; ``router="sigmoid_raw"`` — the same choice, weights ``s_k · scale``
(not normalised); ``router="softmax"`` — the ``top`` largest logits, weights = the softmax over the chosen logits only, times
``scale``; ``router="softmax_all"`` — ``s = softmax(z)`` over all choices, the ``top`` largest ``s + correction`` (``correction``: a learned
number per choice that takes part in the choice only), weights ``s_k · scale``.  With ``identity`` > 0 the router has that many
further choices after the experts; such an identity expert has no tensors, its output is the token itself.  Expert: ``W_down (act(W_gate h) · W_up h)`` without biases (``act="swish_clamp"`` with ``limit``: ``g = min(W_gate h, limit)``,
``u = clamp(W_up h, ±limit)``, ``W_down (g · sigmoid(1.702 g) · (u + 1))``), or — ``gated=False`` — ``W_down act(W_up h)``; the layer's output is the weighted sum over the chosen
experts, or — ``weight_input`` — the plain sum of the experts run on ``weight · h``.  The expert
matrices are stacked — ``gate_up`` ``[E, 2·ff, width]`` (gate rows, then up rows; ``up`` ``[E, ff, width]`` without a gate) and ``down`` ``[E, width, ff]`` — so that an
expert's two input matrices are one product.

Two execution forms (:mod:`libai_b200.ops.kv_functional`): prompt steps sort the (token, expert) pairs by expert and run every
expert as dense products on its rows; single-token steps (and anything as small) let every pair read its expert's matrices in
two kernels without any host-side decision, so that the step can be captured in a CUDA graph.
"""
from __future__ import annotations

from typing import NamedTuple, Optional

import torch
from torch import nn

from libai_b200.ops import kv_functional as KF

from ._param import create_parameter, xavier_normal_, zeros_


class MoEOutput(NamedTuple):
    """The routed experts' part of a layer: ``y`` per token (``pos`` and ``wts`` are ``None``), or sorted rows with the row and the weight of
    every pair; ``keep`` ``[tokens]``: the weight of the token's own input (``None`` without identity experts)."""

    y: torch.Tensor
    pos: Optional[torch.Tensor]
    wts: Optional[torch.Tensor]
    keep: Optional[torch.Tensor]


class MoEFeedForward(nn.Module):
    PAIR_FORM_MAX_TOKENS = 16          # at most this many tokens run pair by pair even when the step is not single-token

    def __init__(self, width, ff, experts, top, *, router_scale=1.0, act="silu", router="sigmoid", router_bias=False, limit=0.0,
                 weight_input=False, identity=0, correction=False, gated=True, init_method=xavier_normal_, layer_idx=0):
        super().__init__()
        self.identity, self.gated = int(identity), bool(gated)
        choices = experts + self.identity
        assert 1 <= top <= choices and router in ("sigmoid", "softmax", "sigmoid_raw", "softmax_all")
        assert not correction or router == "softmax_all", "a correction of the choice is built into the softmax_all router"
        self.width, self.ff, self.experts, self.top, self.router_scale, self.act = width, ff, experts, top, float(router_scale), act
        self.limit, self.weight_input = float(limit), bool(weight_input)
        self.route_mode = {"sigmoid": KF.ROUTE_SIGMOID, "softmax": KF.ROUTE_SOFTMAX, "sigmoid_raw": KF.ROUTE_SIGMOID_RAW,
                           "softmax_all": KF.ROUTE_SOFTMAX_ALL}[router]
        mk = lambda shape: create_parameter(shape, init_method, layer_idx=layer_idx)
        self.router = mk((choices, width))
        self.router_b = create_parameter((choices,), zeros_, layer_idx=layer_idx) if router_bias else None
        self.correction = create_parameter((choices,), zeros_, layer_idx=layer_idx) if correction else None
        self._f32 = {}
        if self.gated:
            self.gate_up = mk((experts, 2 * ff, width))
        else:
            self.up = mk((experts, ff, width))
        self.down = mk((experts, width, ff))

    def _fp32(self, name):
        """The router's arithmetic is fp32: a float copy of a small parameter, kept until the parameter changes."""
        p = getattr(self, name)
        if p is None:
            return None
        key = (p.device, p._version)
        if name not in self._f32 or self._f32[name][0] != key:
            self._f32[name] = (key, p.detach().float().contiguous())
        return self._f32[name][1]

    def forward(self, h, graph_safe: bool = False):
        """``h`` ``[tokens, width]`` → ``(y, pos, wts)``: either ``y`` fp32 ``[tokens, width]`` with ``pos = wts = None``, or the
        sorted expert outputs ``y`` ``[tokens·top, width]`` with the row ``pos[t, k]`` and weight ``wts[t, k]`` of every pair —
        the caller's residual operator gathers the weighted sum (``wts`` is ``None`` with ``weight_input``: a plain sum)."""
        if self.identity:
            raise ValueError("a layer with identity experts is run through MoEFeedForward.run, whose result carries their weight")
        return self.run(h, graph_safe)[:3]

    def run(self, h, graph_safe: bool = False, z=None) -> MoEOutput:
        """:meth:`forward` with the weight of the identity experts.  ``z``: fp32 router logits when the caller has them (leading columns
        of a wider product)."""
        act, ups = KF.ACTS[self.act], self.gate_up if self.gated else self.up
        keep = torch.empty(h.shape[0], dtype=torch.float32, device=h.device) if self.identity else None
        how = dict(bias=self._fp32("router_b"), mode=self.route_mode, z=z, choices=self.experts + self.identity, experts=self.experts,
                   correction=self._fp32("correction"), keep=keep)
        if graph_safe or h.shape[0] <= self.PAIR_FORM_MAX_TOKENS:
            idx, wts = KF.moe_route(h, self.router, self.top, self.router_scale, **how)
            return MoEOutput(KF.moe_pairs(h, ups, self.down, idx, wts, act, self.limit, self.weight_input, self.gated), None, None, keep)
        counts = torch.zeros(self.experts, dtype=torch.int32, device=h.device)
        idx, wts = KF.moe_route(h, self.router, self.top, self.router_scale, counts, **how)
        ys, pos = KF.moe_sorted(h, ups, self.down, idx, counts, act, self.limit, wts if self.weight_input else None, self.gated)
        return MoEOutput(ys, pos, None if self.weight_input else wts, keep)


class FeedForward(nn.Module):
    """``W_down act(W_up h)`` without biases.  ``token_gate``: the layer owns a row ``sg`` ``[1, width]``; its caller multiplies the output
    of a token by ``sigmoid(sg · h)`` (the logit rides in a product the caller makes anyway)."""

    def __init__(self, width, ff, act="gelu", *, token_gate=False, init_method=xavier_normal_, layer_idx=0):
        super().__init__()
        self.act, self.ff = act, ff
        self.up = create_parameter((ff, width), init_method, layer_idx=layer_idx)
        self.down = create_parameter((width, ff), init_method, layer_idx=layer_idx)
        self.sg = create_parameter((1, width), init_method, layer_idx=layer_idx) if token_gate else None

    def forward(self, h):
        """``h`` ``[rows, width]`` → fp32 ``[rows, width]`` (not gated)."""
        u = KF.linear(h, self.up)
        KF.act_rows(u, u, KF.ACTS[self.act])
        return KF.linear_f32(u, self.down)


class GatedFeedForward(nn.Module):
    """``W_down (act(W_gate h) · W_up h)`` without biases; ``gate_up`` stacks the two input matrices (gate rows, then up rows).
    ``act`` names an activation of :data:`libai_b200.ops.kv_functional.ACTS` (``"swish_clamp"`` takes ``limit``)."""

    def __init__(self, width, ff, act="gelu_tanh", *, limit=0.0, init_method=xavier_normal_, layer_idx=0):
        super().__init__()
        self.act, self.ff, self.limit = act, ff, float(limit)
        self.gate_up = create_parameter((2 * ff, width), init_method, layer_idx=layer_idx)
        self.down = create_parameter((width, ff), init_method, layer_idx=layer_idx)

    def forward(self, h):
        """``h`` ``[rows, width]`` → fp32 ``[rows, width]``."""
        gu = KF.linear(h, self.gate_up)
        a = torch.empty(h.shape[0], self.ff, dtype=h.dtype, device=h.device)
        KF.act_rows(gu, a, KF.ACTS[self.act], gated=True, limit=self.limit)
        return KF.linear_f32(a, self.down)
