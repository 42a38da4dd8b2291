"""Matrix memory with exponential gates: a sequence mixer whose state is one fp32 matrix per head (the mLSTM cell of Beck et al.,
"xLSTM: Extended Long Short-Term Memory", 2024).

Per head, ``q = W_q h · dim^(−1/2)``, ``k = W_k h`` ``[dim]``, ``v = W_v h`` ``[vdim]``; the log input gate is ``i = cap · tanh((W_i h + b_i) / cap)``, the
log forget gate ``f = log sigmoid(cap · tanh((W_f h + b_f) / cap))`` (one number each per head and token).  With a running maximum ``m``
that starts at 0::

    m' = max(f + m, i);   S ← e^(f+m−m') S + e^(i−m') k vᵀ;   z ← e^(f+m−m') z + e^(i−m') k
    o  = Sᵀ q / (max(|z·q|, e^(−m')) + 1e-6)

Every head's ``o`` is divided by its root mean square, the heads are concatenated, multiplied by a weight ``[heads·vdim]`` and by
``sigmoid(W_g h)``, and ``W_o`` projects the result.

The gates (their logits leave the product in fp32), the recurrence, the norm and the output gate's activation are fp32 in every compute
dtype.  State per sequence (:class:`libai_b200.inference.state_cache.SequenceStateCache`, kind ``recurrent`` with ``peaks``): ``S``, the sums
``z`` and ``m``.  Prompt steps turn the logits into what the recurrence needs per token (a scan of pairs), then run it: chunk by
chunk on the tensor cores in bf16, through the norm and the gate, or token by token; single-token steps are one kernel from the
projections to the input of ``W_o``.
"""
from __future__ import annotations

import torch
from torch import nn

from libai_b200.ops import kv_functional as KF
from libai_b200.ops import lin_functional as LF
from libai_b200.ops import seq_functional as SF

from ._param import create_parameter, ones_, xavier_normal_, zeros_


class MatrixMemory(nn.Module):
    def __init__(self, width, heads, dim, vdim, *, gate_cap, eps=1e-6, init_method=xavier_normal_, layer_idx=0):
        super().__init__()
        assert gate_cap > 0
        self.width, self.heads, self.dim, self.vdim = width, heads, dim, vdim
        self.gate_cap, self.eps, self.q_scale, self.layer_idx = float(gate_cap), eps, float(dim) ** -0.5, layer_idx
        mk = lambda shape, init=init_method: create_parameter(shape, init, layer_idx=layer_idx)
        self.q, self.k, self.v = mk((heads * dim, width)), mk((heads * dim, width)), mk((heads * vdim, width))
        self.g, self.o = mk((heads * vdim, width)), mk((width, heads * vdim))
        self.i, self.f = mk((heads, width)), mk((heads, width))
        self.i_b, self.f_b = mk((heads,), zeros_), mk((heads,), zeros_)
        self.norm = mk((heads * vdim,), ones_)
        self._gates = None

    # ------------------------------------------------------------------ protocol of the blocks
    @property
    def mix_features(self) -> int:
        return self.heads * self.vdim

    def state_spec(self):
        return "recurrent", dict(heads=self.heads, dim=self.dim, vdim=self.vdim, taps=1, conv_channels=0, peaks=True)

    def input_weights(self):
        return [("q", self.q), ("k", self.k), ("v", self.v), ("g", self.g)]

    def output_weight(self):
        return self.o

    def gate_weights(self):
        """``(W [rows, width], bias fp32 [rows], first row of the forget gates)``: both gates' logits as one product (kept until a
        parameter changes)."""
        key = tuple((p.device, p.dtype, p._version) for p in (self.i, self.f, self.i_b, self.f_b))
        if self._gates is None or self._gates[0] != key:
            w, where = SF.fuse_rows([("i", self.i.detach()), ("f", self.f.detach())])
            b = SF.fuse_biases({"i": self.i_b.detach().float(), "f": self.f_b.detach().float()}, where)
            self._gates = (key, w, b, where["f"][0])
        return self._gates[1:]

    def mix(self, parts, rb, bufs, y, shared=None, out_scale: float = 1.0, h=None):
        """From the projections of the layer input ``h`` (``parts``: name → column view) to the normed, gated read-out written into
        ``y`` ``[tokens, heads·vdim]`` (the input of ``W_o``), times ``out_scale``."""
        w, b, foff = self.gate_weights()
        z = KF.router_logits(h, w)                             # gate logits leave the product in fp32
        q, k, v, g = parts["q"], parts["k"], parts["v"], parts["g"]
        if rb.single:
            return LF.memory_step(q, k, v, z, b, foff, self.gate_cap, self.q_scale, bufs, rb, self.norm, g, self.eps, y, out_scale)
        return LF.memory_prompt(q, k, v, z, b, foff, self.gate_cap, self.q_scale, bufs, rb, self.norm, g, self.eps, y, out_scale)

    def forward(self, h, rb, bufs):
        """Unfused form: ``h`` ``[tokens, width]`` packed rows → ``[tokens, width]``."""
        parts = {name: KF.linear(h, w) for name, w in self.input_weights()}
        y = torch.empty(h.shape[0], self.mix_features, dtype=h.dtype, device=h.device)
        return KF.linear(self.mix(parts, rb, bufs, y, h=h), self.o)
