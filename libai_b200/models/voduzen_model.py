"""Voduzen: a decoder-only language model whose blocks norm the sublayers' outputs only, with latent attention over the whole past
and mixture-of-experts feed-forwards that may pass a token on unchanged.

Structure (every size and constant comes from the configuration):

* embedding: ``embed[token] · embedding.scale``;
* a block: ``x ← x + norm1(mixer(x))``, then ``x ← x + norm2(ff(x))`` — the sublayers read the residual itself; the norms are RMS norms
  whose stored weight is the deviation from one (:func:`libai_b200.ops.paged_functional.outnorm_residual`); a block may have no
  feed-forward;
* mixers (:class:`libai_b200.layers.PagedLatentAttention`): ``latent_attention`` — queries straight from the residual, YaRN-blended
  rotary frequencies where the configuration has them, a learned sink per head in the softmax denominator; ``latent_attention_2`` —
  queries through a normed latent of their own, no sink;
* feed-forward ``moe`` (:class:`libai_b200.layers.MoEFeedForward`): softmax scores over all choices, a learned correction that takes part
  in the choice only, the chosen scores as weights (not renormalised); the last ``router.identity`` choices are identity experts;
  experts are ``W_down relu(W_up h)²``; a shared expert of the same form (:class:`libai_b200.layers.FeedForward`) runs for every token,
  times ``sigmoid(w · h)``;
* logits: the final norm, the output projection, times ``logit_scale``.

The residual, the norms, angles, attention scores and softmax, the router and the token gates are fp32 whatever the compute dtype.
Execution is the framework's generation path for stateful models: packed rows (:class:`~libai_b200.inference.ragged.RaggedBatch`)
against a :class:`~libai_b200.inference.state_cache.SequenceStateCache`.  A block is one product for all down-projections of the
residual, the mixer's kernels, the output product, one product for router and token-gate logits, the experts, and one residual
kernel per sublayer — which also gathers the routed experts' rows, gates the shared expert and adds the identity experts' share.
"""
from __future__ import annotations

from typing import List

import torch
from torch import nn

from libai_b200.config import configurable
from libai_b200.inference.ragged import RaggedBatch
from libai_b200.inference.state_cache import SequenceStateCache
from libai_b200.layers import FeedForward, MoEFeedForward, PagedLatentAttention, RMSLayerNorm
from libai_b200.layers._param import create_parameter, normal_init
from libai_b200.ops import kv_functional as KF
from libai_b200.ops import paged_functional as PF
from libai_b200.ops import seq_functional as SF

from .stateful_lm import StatefulCausalLM, _plain


def build_latent_mixer(kind: str, width: int, m: dict, eps: float, layer_idx: int) -> PagedLatentAttention:
    """Mixer of one block from its ``type`` and ``mixer`` record."""
    rot = m.get("rot") or {}
    common = dict(scale=m.get("scale"), rot_dims=rot.get("dims"), rot_base=rot.get("base", 10000.0), rot_scaling=rot.get("scaling"), eps=eps,
                  layer_idx=layer_idx)
    sizes = (width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"])
    if kind == "latent_attention":
        return PagedLatentAttention(*sizes, sink=True, **common)
    if kind == "latent_attention_2":
        return PagedLatentAttention(*sizes, q_rank=m["q_rank"], **common)
    raise ValueError(f"unknown mixer type {kind!r}")


class OutputNormBlock(nn.Module):
    """``x ← x + norm1(mixer(x))``, ``x ← x + norm2(ff(x))`` on the fp32 residual ``x`` ``[rows, width]`` (updated in place); ``h`` is its
    copy in the compute dtype (``x`` itself in fp32), which the products read."""

    def __init__(self, width, kind, mixer_cfg, mlp_cfg, eps, *, layer_idx=0):
        super().__init__()
        self.kind, self.width, self.eps = kind, width, eps
        self.norm1 = RMSLayerNorm(width, eps=eps, layer_idx=layer_idx, zero_centered=True)
        self.mix = build_latent_mixer(kind, width, mixer_cfg, eps, layer_idx)
        self.mlp = self.shared = self.norm2 = None
        if mlp_cfg:
            if mlp_cfg.get("kind", "moe") != "moe":
                raise ValueError(f"unknown feed-forward kind {mlp_cfg.get('kind')!r}")
            self.norm2 = RMSLayerNorm(width, eps=eps, layer_idx=layer_idx, zero_centered=True)
            r = mlp_cfg["router"]
            self.mlp = MoEFeedForward(width, mlp_cfg["expert"]["ff"], r["experts"], r["top"], router="softmax_all", act="relu2",
                                      identity=int(r.get("identity") or 0), correction=True, gated=False, layer_idx=layer_idx)
            if mlp_cfg.get("shared"):
                self.shared = FeedForward(width, mlp_cfg["shared"]["ff"], "relu2", token_gate=True, layer_idx=layer_idx)
        self._fused = None

    def _fuse(self):
        w = self.norm1.weight
        if self._fused is None or self._fused[0].dtype != w.dtype or self._fused[0].device != w.device:
            ins = SF.fuse_rows([(n, t.detach()) for n, t in self.mix.input_weights()])
            logits = (None, {})
            if self.mlp is not None:                           # router logits, then the shared expert's gate: one fp32 product
                rows = torch.cat([self.mlp.router] + ([self.shared.sg] if self.shared is not None else []), 0).detach()
                logits = SF.fuse_rows([("z", rows)])
            self._fused = ins + logits
        return self._fused

    def _copy(self, x):
        """Where the next products read the residual from: a compute-dtype buffer, or ``None`` when that is ``x`` itself."""
        dt = self.norm1.weight.dtype
        return None if dt == torch.float32 else torch.empty(x.shape, dtype=dt, device=x.device)

    def forward(self, x, h, rb, bufs):
        """Returns the copy of the new ``x`` for the products."""
        w_in, cols, w_z, _ = self._fuse()
        proj = KF.linear(h, w_in)
        parts = {n: proj[:, lo:lo + size] for n, (lo, size) in cols.items()}
        y = torch.empty(x.shape[0], self.mix.mix_features, dtype=w_in.dtype, device=x.device)
        self.mix.mix(parts, rb, bufs, y)
        hb = self._copy(x)
        PF.outnorm_residual(x, self.norm1.weight, self.eps, y=KF.linear_f32(y, self.mix.o), h=hb)
        h = x if hb is None else hb
        if self.mlp is None:
            return h
        z = KF.router_logits(h, w_z)
        routed = self.mlp.run(h, graph_safe=rb.single, z=z)
        shared = self.shared(h) if self.shared is not None else None
        gate = z[:, self.mlp.router.shape[0]] if shared is not None else None
        hb = self._copy(x)
        PF.outnorm_residual(x, self.norm2.weight, self.eps, y=shared, gate=gate, y2=routed.y, pos=routed.pos, cw=routed.wts, keep=routed.keep, h=hb)
        return x if hb is None else hb


class VoduzenModel(nn.Module):
    def __init__(self, vocab, width, layers, embedding=None, eps=1e-6, initializer_range=0.02):
        super().__init__()
        self.vocab, self.width, self.eps = vocab, width, eps
        self.embedding_scale = float((embedding or {}).get("scale", 1.0))
        self.embed = create_parameter((vocab, width), normal_init(initializer_range), layer_idx=0)
        self.layers = nn.ModuleList(
            [OutputNormBlock(width, lc["type"], lc["mixer"], lc.get("mlp"), eps, layer_idx=i) for i, lc in enumerate(layers)])
        self.final_norm = RMSLayerNorm(width, eps=eps, layer_idx=-1, zero_centered=True)

    def register_state(self, cache: SequenceStateCache) -> List[int]:
        out = []
        for blk in self.layers:
            kind, shape = blk.mix.state_spec()
            out.append(cache.register(kind, **shape))
        return out

    def forward(self, tokens, rb: RaggedBatch, cache: SequenceStateCache, handles, tap=None):
        """``tokens`` ``[rows]`` int64 packed → the fp32 residual after the last block ``[rows, width]``.  ``tap(run, x)`` is called
        with the residual after every block (diagnostics)."""
        dt = self.embed.dtype
        x = torch.empty(tokens.shape[0], self.width, dtype=torch.float32, device=tokens.device)
        KF.embed_scale(self.embed, tokens, self.embedding_scale, x)
        h = x if dt == torch.float32 else x.to(dt)
        for i, blk in enumerate(self.layers):
            h = blk(x, h, rb, cache.buffers(handles[i]))
            if tap is not None:
                tap(i, x)
        return x


class VoduzenForCausalLM(StatefulCausalLM):
    @configurable
    def __init__(self, vocab, width, layers, embedding=None, logit_scale=1.0, norm_eps=1e-6, initializer_range=0.02, kv_page_size=64, cfg=None):
        super().__init__()
        self.cfg = cfg
        self.kv_page_size = int(kv_page_size)                  # positions per page of the attention layers' pools
        self.logit_scale = float(logit_scale)
        self.model = VoduzenModel(vocab, width, layers, embedding=embedding, eps=norm_eps, initializer_range=initializer_range)
        self.head = create_parameter((vocab, width), normal_init(initializer_range), layer_idx=-1)

    @classmethod
    def from_config(cls, cfg):
        get = cfg.get if hasattr(cfg, "get") else (lambda k, d=None: getattr(cfg, k, d))
        norm, scale = get("norm") or {}, get("logit_scale")
        return dict(vocab=get("vocab"), width=get("width"), layers=_plain(get("layers")), embedding=_plain(get("embedding")),
                    logit_scale=1.0 if scale is None else scale, norm_eps=norm.get("eps", 1e-6) if hasattr(norm, "get") else 1e-6,
                    initializer_range=get("initializer_range") or 0.02, kv_page_size=get("kv_page_size") or 64, cfg=cfg)

    @torch.no_grad()
    def step_device(self, tokens, rb: RaggedBatch, logits_rows=None, tap=None):
        """The device work of :meth:`step` alone (kernel launches only, no host-side bookkeeping): this is what a CUDA graph of a
        single-token step captures."""
        cache = self.state_cache()
        x = self.model(tokens, rb, cache, self._handles, tap=tap)
        if logits_rows is not None:
            x = x.index_select(0, logits_rows)
        h = torch.empty(x.shape, dtype=self.head.dtype, device=x.device)
        # the constant on the logits rides in the final norm
        PF.postnorm_residual(x, self.model.final_norm.weight, self.model.eps, h=h, inplace=False, out_scale=self.logit_scale)
        return KF.linear_f32(h, self.head)
