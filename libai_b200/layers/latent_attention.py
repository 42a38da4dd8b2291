"""Attention whose keys and values are up-projections of one cached low-rank latent per token: over a sliding window
(:class:`LatentAttention`) or over the whole past with a shared rotated key part (:class:`PagedLatentAttention`).

:class:`LatentAttention`.

``c_q = rmsnorm(W_dq h)``, ``q = W_uq c_q``; ``c = rmsnorm(W_dkv h)`` is the only thing cached; per head ``k = W_uk c``,
``v = W_uv c``; ``score = (q·k)·scale``; position ``i`` sees ``j`` with ``0 ≤ i − j < window``; plain softmax; head ``h`` of
the result is multiplied by ``sigmoid(W_g h)_h``; ``W_o`` mixes the heads.  No positional signal enters the scores.

Prompts expand keys and values for the rows a step needs (one GEMM on ``[cached window | new latents]``) and run the
windowed softmax kernel; single-token steps use the absorbed form — ``q`` is pulled through ``W_uk`` so the scores and the
weighted sum run on the cached latents themselves and ``W_uv`` is applied to the result — which reads ``window·C`` numbers
per sequence instead of expanding ``window`` keys and values.  State per sequence: a ring of the last ``window`` latents
(:class:`libai_b200.inference.state_cache.SequenceStateCache`, kind ``latent``).
"""
from __future__ import annotations

import torch
from torch import nn

from libai_b200.ops import kv_functional as KF
from libai_b200.ops import latent_functional as LF
from libai_b200.ops import seq_functional as SF

from ._param import create_parameter, ones_, xavier_normal_, zeros_


class LatentAttention(nn.Module):
    def __init__(self, width, heads, dim, vdim, q_rank, kv_rank, window, scale=None, eps=1e-6, out_gate=True,
                 init_method=xavier_normal_, absorbed_decode=True, *, layer_idx=0):
        super().__init__()
        self.width, self.heads, self.dim, self.vdim, self.q_rank, self.kv_rank = width, heads, dim, vdim, q_rank, kv_rank
        self.window, self.scale, self.eps = int(window), float(scale if scale is not None else dim ** -0.5), eps
        self.absorbed_decode = absorbed_decode
        mk = lambda shape, init=init_method: create_parameter(shape, init, layer_idx=layer_idx)
        self.dq, self.dq_norm, self.uq = mk((q_rank, width)), mk((q_rank,), ones_), mk((heads * dim, q_rank))
        self.dkv, self.dkv_norm = mk((kv_rank, width)), mk((kv_rank,), ones_)
        self.uk, self.uv = mk((heads * dim, kv_rank)), mk((heads * vdim, kv_rank))
        self.g = mk((heads, width)) if out_gate else None
        self.o = mk((width, heads * vdim))
        self._ukv = self._uk3 = self._uv3 = None

    @property
    def mix_features(self) -> int:
        return self.heads * self.vdim

    def state_spec(self):
        return "latent", dict(ring_len=self.window, channels=self.kv_rank)

    def input_weights(self):
        out = [("dq", self.dq), ("dkv", self.dkv)]
        if self.g is not None:
            out.append(("g", self.g))
        return out

    def output_weight(self):
        return self.o

    def _derived(self):
        if self._ukv is None or self._ukv.dtype != self.uk.dtype or self._ukv.device != self.uk.device:
            self._ukv = torch.cat([self.uk, self.uv], 0).detach().contiguous()
            self._uk3 = self.uk.detach().view(self.heads, self.dim, self.kv_rank)
            self._uv3 = self.uv.detach().view(self.heads, self.vdim, self.kv_rank)

    def mix(self, parts, rb, bufs, y):
        self._derived()
        T, dt, dev = parts["dq"].shape[0], parts["dq"].dtype, parts["dq"].device
        cq = torch.empty(T, self.q_rank, dtype=dt, device=dev)
        SF.rms_norm_rows(parts["dq"], self.dq_norm, offset=0.0, eps=self.eps, out=cq)
        c = torch.empty(T, self.kv_rank, dtype=dt, device=dev)
        SF.rms_norm_rows(parts["dkv"], self.dkv_norm, offset=0.0, eps=self.eps, out=c)
        q = SF.linear(cq, self.uq)
        gate = parts.get("g")
        ring = bufs["ring"]
        H, D, V = self.heads, self.dim, self.vdim
        if rb.single and self.absorbed_decode:
            qa = torch.einsum("bhd,hdc->bhc", q.view(T, H, D).float(), self._uk3.float())
            lat = SF.latent_decode(qa.contiguous(), ring, c, rb, self.window, self.scale)
            SF.head_gate(torch.einsum("bhc,hvc->bhv", lat, self._uv3.float()).contiguous(), gate, y, H, V)
        else:
            kv = SF.linear(SF.latent_gather(ring, c, rb, self.window), self._ukv)
            SF.window_attention(q, kv, gate, rb, y, H, D, V, self.window, self.scale)
        SF.latent_write(ring, c, rb)
        return y

    def forward(self, h, rb, bufs):
        parts = {name: SF.linear(h, w) for name, w in self.input_weights()}
        y = torch.empty(h.shape[0], self.mix_features, dtype=h.dtype, device=h.device)
        return SF.linear(self.mix(parts, rb, bufs, y), self.o)


class PagedLatentAttention(nn.Module):
    """Causal latent attention over the whole past of a sequence, on a paged cache of ``[latent | shared rotated key part]`` rows.

    ``[c | r] = W_dkv h`` with ``c`` RMS-normed and ``r`` rotated; per head ``k = W_uk c`` (unrotated, ``dim``), ``v = W_uv c`` (``vdim``); a
    head's query is ``[dim unrotated | rot_dim rotated]``, from ``W_q h`` or — ``q_rank`` — from ``W_uq rmsnorm(W_dq h)``;
    ``score = (q_unrotated · k + q_rotated · r) · scale``.  Rotary positions turn the first ``rot_dims`` of the ``rot_dim`` channels in
    interleaved pairs ``(2i, 2i + 1)``; frequencies and the factor on cos / sin from :func:`libai_b200.ops.kv_functional.rotary_frequencies`.
    ``sink``: a learned number per head whose exponential joins the softmax denominator without a key or a value.

    A step prepares its rows in one kernel (norms, rotation of the key part, page write); queries are rotated by the attention
    kernels while they load them.  Prompts expand keys and values (one product on the latents of the step, or of every cached
    position when a sequence continues); single-token steps — and steps of at most ``absorb_max_tokens`` rows that continue a
    sequence — use the absorbed form on the cached rows.  State: kind ``paged`` of
    :class:`libai_b200.inference.state_cache.SequenceStateCache`, no convolution tails."""

    def __init__(self, width, heads, dim, rot_dim, vdim, kv_rank, *, q_rank=None, scale=None, rot_dims=None, rot_base=10000.0, rot_scaling=None,
                 sink=False, eps=1e-6, absorb_max_tokens=16, init_method=xavier_normal_, layer_idx=0):
        super().__init__()
        self.rot_dims = int(rot_dim if rot_dims is None else rot_dims)
        assert rot_dim % 2 == 0 and self.rot_dims % 2 == 0 and self.rot_dims <= rot_dim
        self.width, self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = width, heads, dim, rot_dim, vdim, kv_rank
        self.q_rank, self.scale, self.eps = q_rank, float(scale if scale is not None else (dim + rot_dim) ** -0.5), eps
        self.absorb_max_tokens = int(absorb_max_tokens)
        mk = lambda shape, init=init_method: create_parameter(shape, init, layer_idx=layer_idx)
        if q_rank is None:
            self.q = mk((heads * (dim + rot_dim), width))
        else:
            self.dq, self.dq_norm, self.uq = mk((q_rank, width)), mk((q_rank,), ones_), mk((heads * (dim + rot_dim), q_rank))
        self.dkv, self.dkv_norm = mk((kv_rank + rot_dim, width)), mk((kv_rank,), ones_)
        self.uk, self.uv = mk((heads * dim, kv_rank)), mk((heads * vdim, kv_rank))
        self.sink = mk((heads,), zeros_) if sink else None
        self.o = mk((width, heads * vdim))
        freq, self.rot_mscale = KF.rotary_frequencies(self.rot_dims, rot_base, rot_scaling) if self.rot_dims else (torch.zeros(0), 1.0)
        self.register_buffer("rot_freq", freq.float(), persistent=False)
        self._ukv = self._sink32 = None

    @property
    def mix_features(self) -> int:
        return self.heads * self.vdim

    def state_spec(self):
        return "paged", dict(channels=LF.row_channels(self.kv_rank, self.rot_dim), taps=1, conv_channels=0)

    def input_weights(self):
        return [("q", self.q) if self.q_rank is None else ("dq", self.dq), ("dkv", self.dkv)]

    def output_weight(self):
        return self.o

    def _derived(self, dev):
        if self._ukv is None or self._ukv.dtype != self.uk.dtype or self._ukv.device != self.uk.device:
            self._ukv = torch.cat([self.uk, self.uv], 0).detach().contiguous()
            self._sink32 = self.sink.detach().float().contiguous() if self.sink is not None else None
        if self.rot_freq.device != dev:
            self.rot_freq = self.rot_freq.to(dev)

    def mix(self, parts, rb, bufs, y):
        """``parts``: the down- (or query) projections of the step's rows, column slices of one product; ``bufs``: this layer's cache
        entry; ``y`` ``[tokens, H·vdim]`` receives the heads' outputs."""
        self._derived(y.device)
        H, D, R, V, C = self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank
        absorbed = rb.single or (rb.tokens <= self.absorb_max_tokens and any(rb.past_list))
        pool, table = bufs["pool"], bufs["table"]
        cs, cq, lat = LF.latent_prepare(parts["dkv"], self.dkv_norm, self.rot_freq, self.rot_mscale, self.eps, pool, table, rb, C, R,
                                        dq=parts.get("dq"), wq=self.dq_norm if self.q_rank is not None else None,
                                        packed=not absorbed and not any(rb.past_list))
        q = parts["q"] if self.q_rank is None else KF.linear(cq, self.uq)
        if absorbed:
            return LF.latent_absorbed(q, self.uk, self.uv, cs, pool, table, rb, y, H, D, R, V, C, self.scale, sink=self._sink32)
        lat, ext_off = LF.latent_rows(pool, table, rb, lat)
        kv = KF.linear(lat[:, :C], self._ukv)
        return LF.latent_prompt(q, kv, lat, ext_off, cs, rb, y, H, D, R, V, C, self.scale, sink=self._sink32)

    def forward(self, h, rb, bufs):
        """Unfused form: ``h`` ``[tokens, width]`` packed rows → ``[tokens, width]``."""
        parts = {name: KF.linear(h, w) for name, w in self.input_weights()}
        y = torch.empty(h.shape[0], self.mix_features, dtype=h.dtype, device=h.device)
        return KF.linear(self.mix(parts, rb, bufs, y), self.o)
