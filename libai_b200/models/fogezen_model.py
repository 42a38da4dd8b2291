"""Fogezen: a decoder-only language model of sequential blocks with an RMS norm before and after every sublayer, whose mixers are softmax
attention over the whole past, or chunked attention side by side with a matrix memory; a span of blocks may run several times.

Structure (every size and constant comes from the configuration):

* embedding: ``embed[token] · embedding.scale``;
* blocks ``x ← x + m · norm1b(mixer(norm1(x)))``, then ``x ← x + m · norm2b(ff(norm2(x)))`` with ``m`` = ``residual_mult``; the norms are RMS norms
  whose stored weight is the deviation from one; a block may have no feed-forward;
* mixer ``attention`` (:class:`libai_b200.layers.PagedAttention` in its plain form): grouped-query attention over the whole past, biased
  projections, no rotation, queries multiplied by a temperature that grows with the position;
* mixer ``parallel`` (:class:`SideBySideMixer`): grouped-query attention inside chunks of the sequence — per-head query/key norm, rotation of
  interleaved pairs, a channel-wise sigmoid output gate (:class:`libai_b200.layers.RingAttention`) — beside a matrix memory with
  exponential gates (:class:`libai_b200.layers.MatrixMemory`); each output is RMS-normed over the model width with a plain weight of its
  own and the mixer's result is half their sum;
* feed-forward (:class:`libai_b200.layers.GatedFeedForward`): ``W_down (gelu_tanh(W_gate h) · W_up h)``;
* loop: the blocks ``start … stop − 1`` run ``times`` times in a row with the same weights, each pass with its own state, and the row ``t`` of
  ``loop.step`` is added to ``x`` before pass ``t``;
* logits: the final norm times the embedding table (without its scale).

The residual, the norms, angles, attention scores, the gates and the state of the recurrence are fp32 whatever the compute dtype.
Execution is the framework's generation path for stateful models: packed rows (:class:`~libai_b200.inference.ragged.RaggedBatch`)
against a :class:`~libai_b200.inference.state_cache.SequenceStateCache`.  One kernel closes a sublayer (both norms of a ``parallel`` mixer's
outputs, the block's closing norm, the residual sum), adds the row that enters a pass and opens the next sublayer.
"""
from __future__ import annotations

from typing import List, NamedTuple, Optional

import torch
from torch import nn

from libai_b200.config import configurable
from libai_b200.inference.ragged import RaggedBatch
from libai_b200.inference.state_cache import SequenceStateCache
from libai_b200.layers import GatedFeedForward, MatrixMemory, PagedAttention, RingAttention, RMSLayerNorm
from libai_b200.layers._param import create_parameter, normal_init, zeros_
from libai_b200.ops import kv_functional as KF
from libai_b200.ops import paged_functional as PF
from libai_b200.ops import seq_functional as SF

from .stateful_lm import StatefulCausalLM, _plain


class SideBySideMixer(nn.Module):
    """Chunked attention and a matrix memory on the same input; ``left_out`` / ``right_out`` are the weights of the norms over the model
    width that their outputs pass through before half their sum is taken (the block's residual kernel does all of it)."""

    def __init__(self, width, m, eps, layer_idx=0):
        super().__init__()
        a, b = m["left"], m["right"]
        rot = a.get("rot") or {}
        self.left = RingAttention(width, a["heads"], a["kv_heads"], a["dim"], a["vdim"], chunk=a["mask"]["size"], scale=a.get("scale"),
                                  rot_dims=rot.get("dims", 0), rot_base=rot.get("base", 10000.0), rot_pairs="interleaved", qk_norm="head",
                                  out_gate="channel", eps=eps, layer_idx=layer_idx)
        self.right = MatrixMemory(width, b["heads"], b["dim"], b["vdim"], gate_cap=b["gate_cap"], eps=eps, layer_idx=layer_idx)
        self.left_out = RMSLayerNorm(width, eps=eps, layer_idx=layer_idx)
        self.right_out = RMSLayerNorm(width, eps=eps, layer_idx=layer_idx)

    def parts(self):
        return [("left.", self.left), ("right.", self.right)]


def build_mixer(kind: str, width: int, m: dict, eps: float, layer_idx: int):
    """Mixer of one block from its ``type`` and ``mixer`` record."""
    if kind == "parallel":
        return SideBySideMixer(width, m, eps, layer_idx)
    if kind == "attention":
        qt = m.get("q_temp")
        return PagedAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], scale=m.get("scale"), qk_norm=False, bias=True,
                              q_temp=(qt["coef"], qt["every"]) if qt else None, eps=eps, layer_idx=layer_idx)
    raise ValueError(f"unknown mixer type {kind!r}")


class Boundary(NamedTuple):
    """What follows a block on the residual: the row that enters a pass (or ``None``), then the norm that opens the next sublayer."""

    add: Optional[torch.Tensor]
    norm: Optional[RMSLayerNorm]


class ScaledSandwichBlock(nn.Module):
    """``x ← x + m · norm1b(mixer(norm1(x)))``, ``x ← x + m · norm2b(ff(norm2(x)))`` on the fp32 residual ``x`` (updated in place).  The
    opening norm of a sublayer is applied by the kernel that closes the sublayer before it, so a block receives ``h = norm1(x)`` and
    returns what the boundary after it opens."""

    def __init__(self, width, kind, mixer_cfg, mlp_cfg, mult, eps, *, layer_idx=0):
        super().__init__()
        self.kind, self.width, self.mult, self.eps = kind, width, float(mult), eps
        mk = lambda: RMSLayerNorm(width, eps=eps, layer_idx=layer_idx, zero_centered=True)
        self.norm1, self.norm1b = mk(), mk()
        self.mix = build_mixer(kind, width, mixer_cfg, eps, layer_idx)
        self.mlp = None
        if mlp_cfg:
            if mlp_cfg.get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {mlp_cfg.get('kind')!r}")
            self.norm2, self.norm2b = mk(), mk()
            self.mlp = GatedFeedForward(width, mlp_cfg["ff"], "gelu_tanh", layer_idx=layer_idx)
        self._fused = None

    def parts(self):
        return self.mix.parts() if isinstance(self.mix, SideBySideMixer) else [("", self.mix)]

    def state_specs(self):
        return [m.state_spec() for _, m in self.parts()]

    def _fuse(self):
        """Every projection that reads the mixer's input as one matrix (and one bias)."""
        w = self.norm1.weight
        if self._fused is None or self._fused[0].dtype != w.dtype or self._fused[0].device != w.device:
            w_in, cols = SF.fuse_rows([(p + n, t.detach()) for p, m in self.parts() for n, t in m.input_weights()])
            biases = {p + n: t.detach() for p, m in self.parts() if hasattr(m, "input_biases") for n, t in m.input_biases().items()}
            self._fused = w_in, cols, SF.fuse_biases(biases, cols) if biases else None
        return self._fused

    def _close(self, x, norm: RMSLayerNorm, after: Boundary, y, y2=None, branch=None):
        """Residual update with the sublayer's output(s), then the boundary; returns the next sublayer's input (``None`` without one)."""
        h = torch.empty(x.shape, dtype=norm.weight.dtype, device=x.device) if after.norm is not None else None
        PF.sandwich_residual(x, self.eps, y=y, post=norm.weight, mult=self.mult, y2=y2, branch=branch, add=after.add,
                             nxt=after.norm.weight if after.norm is not None else None, h=h)
        return h

    def forward(self, x, h, rb, bufs, after: Boundary):
        """``bufs``: the state entries of the mixer's parts, in their order."""
        w_in, cols, b_in = self._fuse()
        proj = KF.linear(h, w_in, b_in)
        outs = []
        for (p, m), buf in zip(self.parts(), bufs):
            parts = {n[len(p):]: proj[:, lo:lo + size] for n, (lo, size) in cols.items() if n.startswith(p)}
            y = torch.empty(x.shape[0], m.mix_features, dtype=w_in.dtype, device=x.device)
            m.mix(parts, rb, buf, y, {}, h=h)
            outs.append(KF.linear_f32(y, m.output_weight()))
        middle = Boundary(None, self.norm2) if self.mlp is not None else after
        if len(outs) == 2:
            h = self._close(x, self.norm1b, middle, outs[0], outs[1], (self.mix.left_out.weight, self.mix.right_out.weight))
        else:
            h = self._close(x, self.norm1b, middle, outs[0])
        return h if self.mlp is None else self._close(x, self.norm2b, after, self.mlp(h))


class FogezenModel(nn.Module):
    def __init__(self, vocab, width, layers, residual_mult=1.0, embedding=None, loop=None, eps=1e-6, initializer_range=0.02):
        super().__init__()
        self.vocab, self.width, self.eps = vocab, width, eps
        self.embedding_scale = float((embedding or {}).get("scale", 1.0))
        self.embed = create_parameter((vocab, width), normal_init(initializer_range), layer_idx=0)
        self.layers = nn.ModuleList(
            [ScaledSandwichBlock(width, lc["type"], lc["mixer"], lc.get("mlp"), residual_mult, eps, layer_idx=i) for i, lc in enumerate(layers)])
        self.final_norm = RMSLayerNorm(width, eps=eps, layer_idx=-1, zero_centered=True)
        # (block index, pass that it enters or None) for every block run, in execution order
        n, self.loop = len(layers), dict(loop) if loop else None
        self.runs = [(i, None) for i in range(n)]
        self.loop_step = None
        if self.loop:
            a, b, times = int(self.loop["start"]), int(self.loop["stop"]), int(self.loop["times"])
            if not (0 <= a < b <= n and times >= 1):
                raise ValueError(f"a loop over the blocks {a} … {b - 1}, {times} times, does not fit {n} blocks")
            passes = [(i, t if i == a else None) for t in range(times) for i in range(a, b)]
            self.runs = self.runs[:a] + passes + self.runs[b:]
            self.loop_step = create_parameter((times, width), zeros_, layer_idx=a)

    def register_state(self, cache: SequenceStateCache) -> List[List[int]]:
        """Per block run the state entries of its mixer's parts (a block that runs several times keeps a state per pass)."""
        return [[cache.register(kind, **shape) for kind, shape in self.layers[i].state_specs()] for i, _ in self.runs]

    def _boundary(self, run: int) -> Boundary:
        """What comes on the residual right before block run ``run`` (after the last one: nothing)."""
        if run >= len(self.runs):
            return Boundary(None, None)
        i, entered = self.runs[run]
        return Boundary(None if entered is None else self.loop_step[entered], self.layers[i].norm1)

    def _open(self, x, at: Boundary):
        if at.norm is None:
            return None
        h = torch.empty(x.shape, dtype=self.embed.dtype, device=x.device)
        PF.sandwich_residual(x, self.eps, add=at.add, nxt=at.norm.weight, h=h)
        return h

    def forward(self, tokens, rb: RaggedBatch, cache: SequenceStateCache, handles, tap=None):
        """``tokens`` ``[rows]`` int64 packed → the fp32 residual after the last block ``[rows, width]`` (before the final norm).
        ``tap(run, x)`` is called with the residual after every block run, before what enters the next pass (diagnostics)."""
        x = torch.empty(tokens.shape[0], self.width, dtype=torch.float32, device=tokens.device)
        KF.embed_scale(self.embed, tokens, self.embedding_scale, x)
        h = self._open(x, self._boundary(0))
        for run, (i, _) in enumerate(self.runs):
            bufs = [cache.buffers(q) for q in handles[run]]
            after = self._boundary(run + 1)
            if tap is None:
                h = self.layers[i](x, h, rb, bufs, after)
                continue
            self.layers[i](x, h, rb, bufs, Boundary(None, None))
            tap(run, x)
            h = self._open(x, after)
        return x


class FogezenForCausalLM(StatefulCausalLM):
    @configurable
    def __init__(self, vocab, width, layers, residual_mult=1.0, embedding=None, loop=None, norm_eps=1e-6, initializer_range=0.02,
                 kv_page_size=64, cfg=None):
        super().__init__()
        self.cfg = cfg
        self.kv_page_size = int(kv_page_size)                  # positions per page of the attention layers' pools
        self.model = FogezenModel(vocab, width, layers, residual_mult=residual_mult, embedding=embedding, loop=loop, eps=norm_eps,
                                  initializer_range=initializer_range)

    @property
    def head(self):
        """The output projection is the embedding table."""
        return self.model.embed

    @classmethod
    def from_config(cls, cfg):
        get = cfg.get if hasattr(cfg, "get") else (lambda k, d=None: getattr(cfg, k, d))
        norm, mult = get("norm") or {}, get("residual_mult")
        return dict(vocab=get("vocab"), width=get("width"), layers=_plain(get("layers")), residual_mult=1.0 if mult is None else mult,
                    embedding=_plain(get("embedding")), loop=_plain(get("loop")),
                    norm_eps=norm.get("eps", 1e-6) if hasattr(norm, "get") else 1e-6,
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
        PF.sandwich_residual(x, self.model.eps, nxt=self.model.final_norm.weight, h=h)
        return KF.linear_f32(h, self.head)
