"""Operators of attention on paged low-rank latents with a shared rotated key part (``csrc/latent_mixers.cu``): the latent norms,
rotation and page write, attention of prompts on expanded keys and values, and the absorbed form for single-token steps and short
portions, which runs on the cached rows themselves.

A cache row is ``[C latent | R rotated key part | zeros up to the pool's row size]``.  Every operator takes the step's
:class:`~libai_b200.inference.ragged.RaggedBatch`.  On a CUDA device the native kernels run (a missing extension is an error,
there is no fallback); on the CPU the same operators are plain PyTorch, sequence by sequence, which is what the CPU tests use.
Norms, angles, scores and the softmax are fp32 in both.
"""
from __future__ import annotations

from typing import Optional

import torch

from . import count_launch, impl, load_ext, load_kv_ext


def _native(t: torch.Tensor) -> bool:
    return t.is_cuda and impl() == "native"


def row_channels(C: int, R: int, align: int = 8) -> int:
    """Numbers per cache row: latent and rotated part, padded so that rows start on 16-byte boundaries."""
    return -(-(C + R) // align) * align


def _positions(rb):
    return torch.cat([torch.arange(p, p + n) for p, n in zip(rb.past_list, rb.lens)])


def _page_rows(table, slot: int, hi: int, page_size: int):
    p = torch.arange(hi, device=table.device)
    return table[slot, p // page_size].long(), p % page_size


def rotate_pairs(t, cs):
    """``t`` ``[rows, …, R]``: channel ``2i`` turns with channel ``2i + 1`` by the row's ``cs`` ``[rows, R/2, 2]`` = (cos, sin)."""
    cs = cs.view(cs.shape[0], *([1] * (t.dim() - 2)), *cs.shape[1:])
    c, s = cs[..., 0], cs[..., 1]
    u, v = t[..., 0::2], t[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def latent_prepare(dkv, wkv, freq, mscale: float, eps: float, pool, table, rb, C: int, R: int, *, dq=None, wq=None, packed: bool = False):
    """From the down-projections of a step's rows — ``dkv`` ``[tokens, C + R]`` and, for queries with a latent of their own, ``dq``
    ``[tokens, q_rank]`` (column slices) — RMS norm of the latents with the weights ``wkv`` / ``wq``, rotation of the shared key part
    by ``position · freq[i]`` (times ``mscale``; pairs beyond ``len(freq)`` pass), and the write of ``[latent | rotated part]`` into
    the sequence's pages.  Returns ``(cs, cq, lat)``: the step's cos / sin table ``[tokens, R/2, 2]`` fp32, the normed query latent
    (``None`` without ``dq``) and — ``packed`` — a copy of the cache rows ``[tokens, row size]``."""
    T, CS, dev = dkv.shape[0], pool.shape[2], dkv.device
    cs = torch.empty(T, R // 2, 2, dtype=torch.float32, device=dev)
    cq = torch.empty(T, dq.shape[1], dtype=dkv.dtype, device=dev) if dq is not None else None
    lat = torch.empty(T, CS, dtype=dkv.dtype, device=dev) if packed else None
    if _native(dkv):
        count_launch()
        load_kv_ext().latent_prepare(dkv, dq, wkv, wq, freq, float(mscale), float(eps), pool, table, lat, cq, cs, rb.tok_seq, rb.seq_off, rb.slots,
                                     rb.past, C, R)
        return cs, cq, lat
    unit = lambda t: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps)
    if dq is not None:
        cq.copy_(unit(dq.float()) * wq.float())
    ang = _positions(rb).float()[:, None] * freq.float()[None, :]
    cs[..., 0], cs[..., 1] = 1.0, 0.0
    cs[:, : freq.numel(), 0], cs[:, : freq.numel(), 1] = ang.cos() * mscale, ang.sin() * mscale
    rows = torch.cat([unit(dkv[:, :C].float()) * wkv.float(), rotate_pairs(dkv[:, C:].float(), cs),
                      torch.zeros(T, CS - C - R)], 1).to(pool.dtype)
    for b in range(rb.B):
        lo, n, past = rb.offsets[b], rb.lens[b], rb.past_list[b]
        page, row = _page_rows(table, rb.slot_list[b], past + n, pool.shape[1])
        pool[page[past:], row[past:]] = rows[lo:lo + n]
    if packed:
        lat.copy_(rows)
    return cs, cq, lat


def latent_rows(pool, table, rb, lat):
    """The cache rows that a prompt step reads, packed sequence by sequence, and their layout ``(rows, ext_off)``: the step's own
    rows ``lat`` when no sequence has a past, otherwise a gather of every sequence's pages."""
    if not any(rb.past_list):
        return lat, rb.seq_off
    ext = rb.page_ext()
    if _native(pool):
        out = torch.empty(ext.rows, pool.shape[2], dtype=pool.dtype, device=pool.device)
        count_launch()
        load_kv_ext().latent_pages_gather(pool, table, ext.ext_seq, ext.ext_off, rb.slots, out)
        return out, ext.ext_off
    parts = []
    for b in range(rb.B):
        page, row = _page_rows(table, rb.slot_list[b], rb.past_list[b] + rb.lens[b], pool.shape[1])
        parts.append(pool[page, row])
    return torch.cat(parts), ext.ext_off


MMA_QUERY_TILE = 64            # queries per block of the mma.sync prompt kernel
TC_QUERY_TILE = 128            # queries per block of the tcgen05 prompt kernel
TC_MIN_TOKENS = 64             # a step whose longest sequence brings fewer tokens would leave most of its tile empty


def prompt_tc_eligible(q, kv, lat, y, D: int, R: int, V: int, C: int, scale: float) -> bool:
    """bf16 prompt steps whose sizes the tcgen05 prompt kernel is built for."""
    return (q.dtype == torch.bfloat16 and D in (64, 128) and V in (64, 128) and R % 8 == 0 and 8 <= R <= 64 and C % 8 == 0 and scale > 0
            and all(t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0 for t in (q, kv, lat, y)))


def prompt_mma_eligible(q, kv, lat, y, D: int, R: int, V: int, C: int) -> bool:
    """bf16 prompt steps whose sizes the tensor-core prompt kernel is built for."""
    return (q.dtype == torch.bfloat16 and D % 8 == 0 and R % 8 == 0 and V % 8 == 0 and C % 8 == 0 and D + R <= 256 and V <= 256
            and q.stride(0) % 2 == 0 and q.data_ptr() % 4 == 0 and kv.stride(0) % 8 == 0 and kv.data_ptr() % 16 == 0
            and lat.stride(0) % 8 == 0 and lat.data_ptr() % 16 == 0 and y.stride(0) % 2 == 0 and y.data_ptr() % 4 == 0)


def _softmax_rows(s, sink):
    """Softmax over the last dimension of ``s`` ``[H, …, keys]`` whose denominator also holds ``exp(sink_h)``."""
    if sink is None:
        return torch.softmax(s, -1)
    extra = sink.float().view(-1, *([1] * (s.dim() - 1))).expand(*s.shape[:-1], 1)
    return torch.softmax(torch.cat([s, extra], -1), -1)[..., :-1]


def latent_prompt(q, kv, lat, ext_off, cs, rb, y, H: int, D: int, R: int, V: int, C: int, scale: float, *, sink=None, mma: bool = True,
                  tc: Optional[bool] = None):
    """Causal softmax attention of every packed query over the rows ``0 … its own position`` of its sequence.  ``q``
    ``[tokens, H·(D+R)]`` (per head ``[D | R]``, the ``R`` part still unrotated: it is turned by ``cs``), ``kv`` ``[rows, H·D keys | H·V
    values]`` and the shared rotated key part in columns ``C … C+R`` of ``lat`` ``[rows, row size]``, both laid out by ``ext_off``.
    ``sink`` (fp32 ``[H]``): the denominator also holds ``exp(sink_h)``.  The result goes to ``y`` ``[tokens, H·V]``.  bf16 inputs take the
    tcgen05 kernel where it is built for their sizes and the step is long enough (``tc`` decides otherwise), then the mma.sync kernel
    where that one is; ``mma=False`` keeps them on the generic kernel (fp32 inputs always are)."""
    if _native(q):
        if tc is None:
            tc = mma and max(rb.lens) >= TC_MIN_TOKENS
        if tc and prompt_tc_eligible(q, kv, lat, y, D, R, V, C, scale):
            seq, start = rb.query_tiles(TC_QUERY_TILE, longest_first=True)
            if seq.numel() <= 65535:
                count_launch()
                load_ext(required=True).latent_prompt_tc(q, kv, lat[:, C:C + R], cs, sink, ext_off, rb.seq_off, rb.past, seq, start, y, H, D, R, V, float(scale))
                return y
        tiles = rb.query_tiles(MMA_QUERY_TILE) if mma and prompt_mma_eligible(q, kv, lat, y, D, R, V, C) else (None, None)
        count_launch()
        load_kv_ext().latent_prompt(q, kv, lat, cs, sink, ext_off, rb.tok_seq, rb.seq_off, rb.past, tiles[0], tiles[1], y, H, D, R, V, C, float(scale))
        return y
    qf = q.float().view(-1, H, D + R)
    qf = torch.cat([qf[..., :D], rotate_pairs(qf[..., D:], cs)], -1).to(q.dtype).float()
    off = ext_off.tolist()
    for b in range(rb.B):
        lo, n, past, eo = rb.offsets[b], rb.lens[b], rb.past_list[b], off[b]
        rows = kv[eo:eo + past + n].float()
        kr = lat[eo:eo + past + n, C:C + R].float()
        s = torch.einsum("ihd,jhd->hij", qf[lo:lo + n, :, :D], rows[:, :H * D].view(-1, H, D)) + torch.einsum("ihr,jr->hij", qf[lo:lo + n, :, D:], kr)
        i, j = torch.arange(past, past + n)[:, None], torch.arange(past + n)[None, :]
        p = _softmax_rows((s * scale).masked_fill((j > i)[None], float("-inf")), sink)
        y[lo:lo + n] = torch.einsum("hij,jhv->ihv", p, rows[:, H * D:].view(-1, H, V)).reshape(n, H * V).to(y.dtype)
    return y


def latent_absorbed(q, wuk, wuv, cs, pool, table, rb, y, H: int, D: int, R: int, V: int, C: int, scale: float, *, sink=None,
                    parts: Optional[int] = None, mma: bool = True):
    """The same attention in the absorbed form: a row's query is pulled through the key up-projection (``wuk`` ``[H·D, C]``), so that
    scores and the weighted sum run on the cached rows in the pages, and the value up-projection (``wuv`` ``[H·V, C]``) is applied to
    the result.  Nothing is expanded and nothing is decided on the host, so single-token steps can be captured in a CUDA graph.
    ``parts``: into how many parts the keys of a row are cut (``None``: enough blocks for the device)."""
    if _native(q):
        ext = load_kv_ext()
        mma = mma and q.dtype == torch.bfloat16 and pool.data_ptr() % 16 == 0 and ext.latent_absorbed_mma_ok(C, R, pool.shape[2])
        if parts is None:
            groups = q.shape[0] * -(-H // (16 if mma else 8))
            parts = max(1, min(64, 148 // groups if mma else -(-592 // groups)))     # mma: one wave of one block per SM
        count_launch(3)
        ext.latent_absorbed(q, wuk, wuv, cs, sink, pool, table, rb.tok_seq, rb.seq_off, rb.slots, rb.past, y, H, D, R, V, C, float(scale), parts, mma)
        return y
    qf = q.float().view(-1, H, D + R)
    qa = torch.cat([torch.einsum("thd,hdc->thc", qf[..., :D], wuk.float().view(H, D, C)), rotate_pairs(qf[..., D:], cs)], -1)
    lat = torch.empty(q.shape[0], H, C)
    for b in range(rb.B):
        for t in range(rb.lens[b]):
            r = rb.offsets[b] + t
            page, row = _page_rows(table, rb.slot_list[b], rb.past_list[b] + t + 1, pool.shape[1])
            rows = pool[page, row].float()
            p = _softmax_rows(qa[r] @ rows[:, :C + R].T * scale, sink)
            lat[r] = p @ rows[:, :C]
    y.copy_(torch.einsum("thc,hvc->thv", lat, wuv.float().view(H, V, C)).reshape(-1, H * V))
    return y
