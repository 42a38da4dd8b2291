"""Voduzen against a plain float64 oracle (``voduzen_oracle.py``): every mechanism alone, whole prompts, decoding through the paged
latent cache, prompt portions, ragged batches, pages and slots that are freed and used again, keys far away and at page borders
made decisive by their content or by their position alone, the first tokens of a sequence, long decoding, other sizes, generation.

The CPU parametrisation exercises the framework's PyTorch operators; the ``cuda`` one (marked ``gpu``) the sm_100a kernels.
"""
import importlib.util
import json
import math
import os

import pytest
import torch

from libai_b200.inference.ragged import RaggedBatch
from libai_b200.inference.scheduler import RequestScheduler
from libai_b200.inference.state_cache import SequenceStateCache
from libai_b200.layers import FeedForward, MoEFeedForward, PagedLatentAttention
from libai_b200.layers._param import param_defaults
from libai_b200.models.utils.model_loader.auto import load_pretrained
from libai_b200.ops import kv_functional as KF
from libai_b200.ops import latent_functional as LF
from libai_b200.ops import paged_functional as PF

from . import voduzen_oracle as O

DEVICES = [pytest.param("cpu", id="cpu"), pytest.param("cuda", id="cuda", marks=pytest.mark.gpu)]
REPO = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
F64 = torch.float64
YARN = {"factor": 4.0, "original": 64, "fast": 4.0, "slow": 1.0}


def rel_err(got, want):
    """Error of logits the way a user sees it: mean removed, RMS over the vocabulary, relative to the RMS of the target."""
    got, want = got.detach().cpu().double(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float(d.pow(2).mean(-1).sqrt().max() / scale)


def save_model(tmp_path, cfg, weights, name="m"):
    from safetensors.torch import save_file

    d = os.path.join(str(tmp_path), name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights.items()}, os.path.join(d, "model.safetensors"))
    return d


def make(tmp_path, cfg, device, dtype=torch.float32, seed=0, weights=None, page_size=4):
    """The loaded model (pages of ``page_size`` positions: small, so that short prompts cross many page borders) and its weights."""
    weights = weights if weights is not None else O.random_weights(cfg, seed)
    model = load_pretrained(save_model(tmp_path, cfg, weights), dtype=dtype, device=device)
    model.kv_page_size = page_size
    return model, weights


def run_schedule(model, prompts, cuts, **kw):
    """Feed ``prompts`` together: step s brings ``cuts[i][s]`` tokens of prompt i (requests that have nothing left drop out).
    Returns per prompt the logits of all its positions."""
    sched = RequestScheduler(model, **kw)
    at = [0] * len(prompts)
    got = [[] for _ in prompts]
    for s in range(max(len(c) for c in cuts)):
        entries, who = [], []
        for i, p in enumerate(prompts):
            if s < len(cuts[i]):
                n = cuts[i][s]
                entries.append((("r", i), p[at[i]:at[i] + n], list(range(n))))
                who.append((i, n))
                at[i] += n
        logits = sched.step(entries)
        o = 0
        for i, n in who:
            got[i].append(logits[o:o + n].clone())
            o += n
        sched.finish([("r", i) for i, p in enumerate(prompts) if at[i] == len(p)])
    assert sched.cache.live() == 0
    return [torch.cat(g) for g in got]


def tokens(n, vocab=50, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def mixed_cfg(**kw):
    """Every branch once: both mixers, YaRN and plain frequencies, experts with and without identity experts and a shared expert, a
    block without a feed-forward, value heads wider and narrower than key heads, latents of unequal sizes."""
    layers = [O.layer(O.mixer_cfg(scaling=YARN), mlp=O.moe_cfg()),
              O.layer(O.mixer_cfg(heads=2, dim=8, rot_dim=2, vdim=5, kv_rank=9, q_rank=7, scale=0.5, base=1000.0), mlp=None),
              O.layer(O.mixer_cfg(heads=4, dim=4, rot_dim=8, vdim=4, kv_rank=6, scale=0.4), mlp=O.moe_cfg(ff=4, experts=3, top=1, identity=1, shared_ff=12)),
              O.layer(O.mixer_cfg(heads=1, dim=10, rot_dim=6, vdim=12, kv_rank=16, q_rank=20, base=30.0), mlp=O.moe_cfg(ff=6, experts=4, top=3, identity=0, shared_ff=0)),
              O.layer(O.mixer_cfg(rot_dim=6, scaling=dict(YARN, factor=2.0, original=30)), mlp=O.moe_cfg(experts=2, top=3, identity=4))]
    return O.model_cfg(layers, **kw)


def build_mixer(m, width, eps, W, p, device, dtype=torch.float32):
    rot = m["rot"]
    with param_defaults(dtype=dtype, device=device):
        mod = PagedLatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], q_rank=m.get("q_rank"), scale=m["scale"],
                                   rot_dims=rot["dims"], rot_base=rot["base"], rot_scaling=rot.get("scaling"), sink="q_rank" not in m, eps=eps)
    with torch.no_grad():
        for name, t in mod.named_parameters():
            t.copy_(W[p + name.replace("_norm", ".norm")])
    return mod


def run_mixer(mod, h, device, lens, page_size=4, dtype=torch.float32):
    """A mixer module alone on one sequence ``h`` ``[n, width]`` fed in the portions ``lens``; returns ``[n, width]``."""
    cache = SequenceStateCache(device, dtype, page_size=page_size)
    kind, shape = mod.state_spec()
    handle = cache.register(kind, **shape)
    slot = cache.allocate(3)[1:2]                                   # not slot 0
    out, at = [], 0
    for n in lens:
        cache.prepare(slot, [n])
        rb = RaggedBatch([n], slot, [at], device)
        with torch.no_grad():
            out.append(mod(h[at:at + n].to(dtype).to(device), rb, cache.buffers(handle)).cpu().double())
        cache.advance(slot, [n])
        at += n
    return torch.cat(out)


# ------------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dims,base,scaling", [(16, 3e5, None), (2, 7.0, None), (16, 2e4, {"factor": 5.0, "original": 512, "fast": 30.0, "slow": 1.5}),
                                               (8, 30.0, {"factor": 3.0, "original": 8, "fast": 9.0, "slow": 0.01}), (6, 1e4, YARN),
                                               (4, 50.0, {"factor": 1.0, "original": 100, "fast": 2.0, "slow": 2.0})])
def test_rotary_frequencies(dims, base, scaling):
    want, mag = O.pair_frequencies(dims, base, scaling)
    got, got_mag = KF.rotary_frequencies(dims, base, scaling)
    assert torch.allclose(got.double(), torch.tensor(want, dtype=F64), rtol=1e-6) and got_mag == pytest.approx(mag, rel=1e-12)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("C,R,QR,rot", [(12, 4, 10, 4), (7, 6, None, 6), (32, 8, 24, 4), (16, 2, 16, 2)])
def test_preparation_writes_the_cache_rows(device, C, R, QR, rot):
    """Latent norms, rotation and page write alone, for two sequences of which one goes on."""
    g = torch.Generator().manual_seed(1)
    ps, eps, lens, past = 3, 1e-3, [5, 4], [0, 7]
    T = sum(lens)
    proj = torch.randn(T, C + R + (QR or 0), generator=g)
    wkv, wq = torch.rand(C, generator=g) + 0.5, torch.rand(QR or 1, generator=g) + 0.5
    cfg = {"dims": rot, "base": 20.0, "scaling": YARN}
    freq, mag = KF.rotary_frequencies(rot, 20.0, YARN)
    cache = SequenceStateCache(device, torch.float32, page_size=ps)
    handle = cache.register("paged", channels=LF.row_channels(C, R), taps=1, conv_channels=0)
    slots = cache.allocate(2)
    cache.prepare(slots, [a + b for a, b in zip(lens, past)])
    bufs = cache.buffers(handle)
    bufs["pool"].fill_(float("nan"))
    rb = RaggedBatch(lens, slots, past, device)
    d = proj.to(device)
    cs, cq, lat = LF.latent_prepare(d[:, :C + R], wkv.to(device), freq.to(device), mag, eps, bufs["pool"], bufs["table"], rb, C, R,
                                    dq=d[:, C + R:] if QR else None, wq=wq.to(device) if QR else None, packed=True)
    p64 = proj.double()
    pool, table = bufs["pool"].cpu().double(), bufs["table"].cpu()
    for b in range(2):
        start = torch.zeros(past[b] + lens[b], 1, R, dtype=F64)
        start[past[b]:, 0] = p64[rb.offsets[b]:rb.offsets[b + 1], C:C + R]
        turned = O.rotate_pairs(start, cfg)[past[b]:, 0]
        want = torch.cat([O.unit_rms(p64[rb.offsets[b]:rb.offsets[b + 1], :C], eps) * wkv.double(), turned], 1)
        for i in range(lens[b]):
            pos = past[b] + i
            row = pool[int(table[slots[b], pos // ps]), pos % ps]
            assert torch.allclose(row[:C + R], want[i], atol=1e-5) and bool((row[C + R:] == 0).all())
            assert torch.equal(lat[rb.offsets[b] + i].cpu().double(), row)
    if QR:
        assert torch.allclose(cq.cpu().double(), O.unit_rms(p64[:, C + R:], eps) * wq.double(), atol=1e-5)
    assert torch.allclose(cs[:, 0, 0].cpu().double(), mag * torch.cos(torch.tensor([0., 1, 2, 3, 4, 7, 8, 9, 10], dtype=F64) * float(freq[0])), atol=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("lens", [[21], [1] * 21, [5, 1, 9, 2, 4], [3, 18]])
@pytest.mark.parametrize("m", [O.mixer_cfg(), O.mixer_cfg(scaling=YARN), O.mixer_cfg(heads=1, dim=8, rot_dim=2, vdim=3, kv_rank=5, q_rank=6),
                               O.mixer_cfg(heads=17, dim=4, rot_dim=6, vdim=8, kv_rank=20, q_rank=9, base=9.0), O.mixer_cfg(rot_dim=8, rot_dims=4)],
                         ids=["direct", "yarn", "latent_query", "many_heads", "partial_rotation"])
def test_mixer_alone(device, lens, m):
    width, eps, p = 16, 1e-5, "l0.mix."
    W = O.random_weights(O.model_cfg([O.layer(m)], width=width), seed=3)
    sink = "q_rank" not in m
    mod = build_mixer(m, width, eps, W, p, device)
    h = torch.randn(21, width, generator=torch.Generator().manual_seed(1), dtype=F64)
    want = O.mixer(h, W, p, m, eps, sink)
    for absorb in (0, 16):                                          # short portions in the expanded and in the absorbed form
        mod.absorb_max_tokens = absorb
        assert torch.allclose(run_mixer(mod, h, device, lens), want, atol=3e-5)
    # each ingredient is visible in the result
    far = lambda Wx, mx=m: not torch.allclose(O.mixer(h, Wx, p, mx, eps, sink), want, atol=1e-2)
    if sink:
        assert far({**W, p + "sink": W[p + "sink"] - 30.0})
    assert far(W, dict(m, rot={"dims": 0})) and far(W, dict(m, scale=2 * m["scale"]))
    if m["rot"].get("scaling"):
        assert far(W, dict(m, rot={"dims": m["rot"]["dims"], "base": m["rot"]["base"]}))
    assert not far({**W, p + "dkv": torch.cat([3.0 * W[p + "dkv"][: m["kv_rank"]], W[p + "dkv"][m["kv_rank"]:]])})   # the latent is normed …
    assert far({**W, p + "dkv": torch.cat([W[p + "dkv"][: m["kv_rank"]], 3.0 * W[p + "dkv"][m["kv_rank"]:]])})       # … the rotated part is not


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("n", [24, 19, 1100])
def test_outer_norm_residual(device, n):
    g = torch.Generator().manual_seed(5)
    rows, top = 9, 3
    x, y, ys = torch.randn(rows, n, generator=g), torch.randn(rows, n, generator=g), torch.randn(rows * top, n, generator=g)
    w = (0.3 * torch.randn(n, generator=g)).to(torch.bfloat16).float()
    pos = torch.randperm(rows * top, generator=g).view(rows, top).int()
    pos[2, 1] = pos[5, 0] = pos[5, 1] = pos[5, 2] = -1
    cw, keep, z = torch.rand(rows, top, generator=g), torch.rand(rows, generator=g), torch.randn(rows, 4, generator=g)
    gathered = (ys.double()[pos.clamp(min=0).long()] * (cw * (pos >= 0)).double()[:, :, None]).sum(1)
    v = torch.sigmoid(z[:, 2:3].double()) * y.double() + gathered + keep.double()[:, None] * x.double()
    want = x.double() + O.centred_norm(v, w.double(), 1e-2)
    xd, h = x.clone().to(device), torch.empty(rows, n, device=device)
    PF.outnorm_residual(xd, w.to(device), 1e-2, y=y.to(device), y2=ys.to(device), pos=pos.to(device), cw=cw.to(device), gate=z.to(device)[:, 2],
                        keep=keep.to(device), h=h)
    assert torch.allclose(xd.cpu().double(), want, atol=1e-5) and torch.equal(xd, h)
    xd = x.clone().to(device)                                      # one sublayer output and nothing else
    PF.outnorm_residual(xd, w.to(device), 1e-2, y=y.to(device))
    assert torch.allclose(xd.cpu().double(), x.double() + O.centred_norm(y.double(), w.double(), 1e-2), atol=1e-5)
    h = torch.empty(rows, n, device=device)                        # a constant on the normed row
    PF.postnorm_residual(xd, w.to(device), 1e-2, h=h, inplace=False, out_scale=0.37)
    assert torch.allclose(h.cpu().double(), 0.37 * O.centred_norm(xd.cpu().double(), w.double(), 1e-2), atol=1e-5)


def build_moe(mc, width, W, p, device, dtype=torch.float32):
    r = mc["router"]
    with param_defaults(dtype=dtype, device=device):
        mod = MoEFeedForward(width, mc["expert"]["ff"], r["experts"], r["top"], router="softmax_all", act="relu2", identity=r["identity"], correction=True,
                             gated=False)
        shared = FeedForward(width, mc["shared"]["ff"], "relu2", token_gate=True) if mc.get("shared") else None
    with torch.no_grad():
        mod.router.copy_(W[p + "router"])
        mod.correction.copy_(W[p + "correction"])
        mod.up.copy_(torch.stack([W[f"{p}e{e}.up"] for e in range(r["experts"])]))
        mod.down.copy_(torch.stack([W[f"{p}e{e}.down"] for e in range(r["experts"])]))
        if shared is not None:
            for name in ("up", "down", "sg"):
                getattr(shared, name).copy_(W[p + "shared." + name])
    return mod, shared


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("experts,identity,top,rows", [(5, 2, 2, 40), (4, 0, 1, 7), (2, 3, 5, 21), (40, 8, 6, 3), (1, 1, 1, 30), (33, 5, 34, 4)])
def test_experts_alone(device, experts, identity, top, rows):
    width, p = 16, "l0.mlp."
    mc = O.moe_cfg(ff=8, experts=experts, top=top, identity=identity, shared_ff=12)
    W = O.random_weights(O.model_cfg([O.layer(O.mixer_cfg(), mlp=mc)], width=width), seed=6)
    mod, shared = build_moe(mc, width, W, p, device)
    h = torch.randn(rows, width, generator=torch.Generator().manual_seed(7), dtype=F64)
    want = O.feed_forward(h, W, p, mc)
    hd = h.float().to(device)
    with torch.no_grad():
        idx, wts = KF.moe_route(hd, mod.router, top, 1.0, mode=KF.ROUTE_SOFTMAX_ALL, correction=mod._fp32("correction"))
        for t in range(rows):
            chosen, weights = O.route(h[t], W, p, mc)
            assert idx[t].tolist() == chosen and torch.allclose(wts[t].cpu().double(), torch.tensor(weights, dtype=F64), atol=1e-6)
        for graph_safe in (False, True):                           # sorted form (many rows) and pair form
            r = mod.run(hd, graph_safe=graph_safe)
            y = r.y if r.pos is None else (r.y[r.pos.clamp(min=0).long()] * (r.wts * (r.pos >= 0))[:, :, None]).sum(1)
            if identity:
                y = y + r.keep[:, None] * hd
            else:
                assert r.keep is None
            y = y + torch.sigmoid(hd @ shared.sg[0])[:, None] * shared(hd)
            assert torch.allclose(y.cpu().double(), want, atol=3e-5)
    if experts + identity > top:                                   # the correction takes part in the choice …
        other = O.feed_forward(h, {**W, p + "correction": torch.roll(W[p + "correction"] * 4, 1)}, p, mc)
        assert not torch.allclose(other, want, atol=1e-3)
    else:                                                          # … and not in the weights
        assert torch.allclose(O.feed_forward(h, {**W, p + "correction": -W[p + "correction"]}, p, mc), want)


# ---------------------------------------------------------------------------------------------------------- whole model
@pytest.mark.parametrize("device", DEVICES)
def test_whole_prompt_with_residuals(device, tmp_path):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device)
    toks = tokens(19)
    residuals, taps = [], []
    want = O.forward(W, cfg, toks, lambda i, x: residuals.append(x.clone()))
    cache = model.state_cache()
    slots = cache.allocate(1)
    got = model.step(torch.tensor(toks, device=device), RaggedBatch([len(toks)], slots, [0], device),
                     tap=lambda i, x: taps.append(x.detach().cpu().double().clone()))
    cache.free(slots)
    assert len(taps) == len(residuals) == len(cfg["layers"])
    for i, (a, b) in enumerate(zip(taps, residuals)):
        assert torch.allclose(a, b, atol=2e-4), f"residual after block {i}"
    assert rel_err(got, want) < 1e-4
    assert rel_err(O.forward(W, dict(cfg, logit_scale=1.4), toks), want) > 0.5 and rel_err(O.forward(W, dict(cfg, embedding={"scale": 1.0}), toks), want) > 1e-2


@pytest.mark.parametrize("device", DEVICES)
def test_prefill_against_token_by_token(device, tmp_path):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device)
    toks = tokens(26, seed=3)
    want = O.forward(W, cfg, toks)
    whole, = run_schedule(model, [toks], [[len(toks)]])
    single, = run_schedule(model, [toks], [[1] * len(toks)])
    mixed, = run_schedule(model, [toks], [[9] + [1] * 17])
    for got in (whole, single, mixed):
        assert rel_err(got, want) < 1e-4
    assert rel_err(single, whole.cpu()) < 1e-4


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cuts", [[2] * 15, [3, 7, 2, 11, 7], [13, 2, 2, 13], [1, 29], [29, 1], [10, 20]])
def test_prompt_portions(device, tmp_path, cuts):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device)
    toks = tokens(30, seed=5)
    want = O.forward(W, cfg, toks)
    for absorb in (16, 0):                                          # short portions in either form
        for blk in model.model.layers:
            blk.mix.absorb_max_tokens = absorb
        got, = run_schedule(model, [toks], [cuts])
        assert rel_err(got, want) < 1e-4


@pytest.mark.parametrize("device", DEVICES)
def test_ragged_batches_against_each_alone(device, tmp_path):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device)
    prompts = [tokens(n, seed=n) for n in (1, 17, 4, 30, 9)]
    want = [O.forward(W, cfg, p) for p in prompts]
    cuts = [[1], [12] + [1] * 5, [2, 1, 1], [21] + [1] * 9, [9]]
    together = run_schedule(model, prompts, cuts)
    for i, p in enumerate(prompts):
        alone, = run_schedule(model, [p], [cuts[i]])
        assert rel_err(together[i], want[i]) < 1e-4
        assert rel_err(together[i], alone.cpu()) < 1e-5
    cuts2 = [[1], [5, 12], [1, 3], [2, 20, 8], [4, 1, 4]]          # unequal portions in one step
    for got, w in zip(run_schedule(model, prompts, cuts2), want):
        assert rel_err(got, w) < 1e-4


@pytest.mark.parametrize("device", DEVICES)
def test_pages_and_slots_are_reused_without_clearing(device, tmp_path):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device, page_size=4)
    sched = RequestScheduler(model)
    cache = sched.cache
    a, b, c = tokens(23, seed=1), tokens(8, seed=2), tokens(15, seed=3)
    sched.step([("a", a, []), ("b", b, [])])
    slot_a, pages_a = sched.slot_of["a"], list(cache._pages[sched.slot_of["a"]])
    sched.finish(["a"])
    got = sched.step([("c", c[:6], list(range(6)))])               # takes a's slot and a's first pages
    assert sched.slot_of["c"] == slot_a and cache._pages[slot_a] == pages_a[:2]
    got = torch.cat([got] + [sched.step([("c", [t], [0]), ("b", [1], [])]) for t in c[6:]])
    assert rel_err(got, O.forward(W, cfg, c)) < 1e-4
    before, pages_before = cache.capacity, cache.num_pages
    many = [(("m", i), tokens(3 + i, seed=10 + i), [2 + i]) for i in range(before + 3)]      # more requests than slots, more rows than pages
    logits = sched.step(many)
    assert cache.capacity > before and cache.num_pages > pages_before
    for row, (_, p, _) in enumerate(many):
        assert rel_err(logits[row:row + 1], O.forward(W, cfg, p)[-1:]) < 1e-4
    got = sched.step([("c", [7], [0])])                            # a request that lived through the growth goes on
    assert rel_err(got, O.forward(W, cfg, c + [7])[-1:]) < 1e-4
    sched.finish(["b", "c"] + [("m", i) for i in range(before + 3)])
    assert cache.live() == 0 and len(cache._free_pages) == cache.num_pages       # every page came back


# ------------------------------------------------------------------------------------------- far keys, page borders, starts
def sharp_weights(by_position, distance):
    """One block, one head, built by hand on one-hot embeddings (token 0: filler, 1: the probe that asks, 2: the needle with a value
    unlike every other).  The probe's query finds the needle by its content (the unrotated parts agree) or — ``by_position`` — finds
    whatever token lies ``distance`` back: all keys carry the same rotated part, so the angle alone decides."""
    width, R = 16, 4
    m = O.mixer_cfg(heads=1, dim=8, rot_dim=R, vdim=8, kv_rank=8, scale=1.0, base=10000.0)
    cfg = O.model_cfg([O.layer(m)], vocab=8, width=width, embedding_scale=1.0, logit_scale=1.0, eps=1e-6)
    W = O.random_weights(cfg, seed=9)
    p = "l0.mix."
    W["embed"] = torch.zeros(8, width, dtype=F64)
    for t in range(8):
        W["embed"][t, t] = 1.0
    dkv, q, uk, uv = torch.zeros(8 + R, width, dtype=F64), torch.zeros(8 + R, width, dtype=F64), torch.zeros(8, 8, dtype=F64), torch.zeros(8, 8, dtype=F64)
    for t in range(8):
        dkv[t, t] = 1.0                                            # token t's latent is the t-th unit vector, normed
    uv[:, :3] = torch.tensor([[1.0, 0.2, 0], [0.1, 0.5, 0], [0, 0, 0], [0, 0, 4], [0, 0, -3], [0, 0.1, 0], [0, 0, 0], [0, 0, 0]], dtype=F64)
    if by_position:
        dkv[8:, :8] = torch.tensor([1.0, 0, 1.0, 0], dtype=F64)[:, None]
        for i, (f, size) in enumerate(((1.0, 200.0), (0.01, 2000.0))):
            q[8 + 2 * i, 1], q[9 + 2 * i, 1] = size * math.cos(distance * f), -size * math.sin(distance * f)
    else:
        uk[0, 2] = 1.0
        q[0, 1] = 8.0
    W[p + "dkv"], W[p + "dkv.norm"], W[p + "q"], W[p + "uk"], W[p + "uv"] = dkv, torch.ones(8, dtype=F64), q, uk, uv
    W[p + "sink"] = torch.tensor([-2.0], dtype=F64)
    return cfg, {k: v.to(torch.bfloat16).to(F64) for k, v in W.items()}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("by_position", [False, True], ids=["content", "position"])
@pytest.mark.parametrize("key_at,page_size", [(0, 8), (7, 8), (8, 8), (63, 8), (64, 8), (150, 64), (127, 64), (128, 64), (1, 3), (198, 5)])
def test_one_far_key_decides_the_last_position(device, tmp_path, by_position, key_at, page_size):
    n = 200
    cfg, W = sharp_weights(by_position, n - 1 - key_at)
    toks = [0] * n
    toks[key_at], toks[-1] = 2, 1
    want = O.forward(W, cfg, toks)[-1:]
    for other in {key_at - 1, key_at + 1, 0} - {-1, key_at, n - 1}:      # the key is decisive, and so is its place where position decides
        moved = list(toks)
        moved[key_at], moved[other] = 0, 2 if by_position else 0
        assert rel_err(O.forward(W, cfg, moved)[-1:], want) > 0.2
    model, _ = make(tmp_path, cfg, device, weights=W, page_size=page_size)
    for cuts in ([n], [n - 1, 1], [key_at + 1] + [1] * (n - key_at - 1) if key_at > 100 else [n - 40] + [1] * 40, [n - 2, 2], [n - 30, 30]):
        got, = run_schedule(model, [toks], [cuts])
        assert rel_err(got[-1:], want) < 1e-3, cuts


@pytest.mark.parametrize("device", DEVICES)
def test_the_first_tokens_of_a_sequence(device, tmp_path):
    """The first positions see few keys beside the sink, whatever the slot and its pages held before."""
    cfg = O.model_cfg([O.layer(O.mixer_cfg(), mlp=O.moe_cfg()), O.layer(O.mixer_cfg(q_rank=6), mlp=None)])
    W = O.random_weights(cfg, seed=4)
    W["l0.mix.sink"] = (W["l0.mix.sink"] + 2.0).to(torch.bfloat16).to(F64)                       # the sink takes most of the first positions' weight
    model, _ = make(tmp_path, cfg, device, weights=W)
    sched = RequestScheduler(model)
    sched.step([("old", tokens(11, seed=8), [])])                  # leaves rows behind in the pages that come next
    sched.finish(["old"])
    toks = tokens(6, seed=9)
    want = O.forward(W, cfg, toks)
    assert rel_err(O.forward({**W, "l0.mix.sink": W["l0.mix.sink"] - 40.0}, cfg, toks)[:1], want[:1]) > 1e-3
    for cuts in ([6], [1] * 6, [2, 1, 3]):
        got, = run_schedule(model, [toks], [cuts])
        assert rel_err(got, want) < 1e-4, cuts


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device, tmp_path):
    cfg = O.model_cfg([O.layer(O.mixer_cfg(scaling=YARN), mlp=O.moe_cfg()), O.layer(O.mixer_cfg(q_rank=6), mlp=O.moe_cfg())])
    model, W = make(tmp_path, cfg, device, page_size=16)
    toks = tokens(150, seed=4)
    want = O.forward(W, cfg, toks)
    got, = run_schedule(model, [toks], [[10] + [1] * 140])
    assert rel_err(got, want) < 2e-4


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", ["one_head", "wide_latent", "all_experts", "only_identity", "wide_values", "odd_sizes", "many_heads", "no_ff", "no_yarn_blend"])
def test_other_sizes(device, tmp_path, case):
    m1, m2, mlp, kw = O.mixer_cfg(scaling=YARN), O.mixer_cfg(q_rank=10), O.moe_cfg(), {}
    if case == "one_head":
        m1, m2 = O.mixer_cfg(heads=1, dim=16, vdim=16), O.mixer_cfg(heads=1, q_rank=3)
    elif case == "wide_latent":
        m1, m2 = O.mixer_cfg(kv_rank=300, rot_dim=10), O.mixer_cfg(kv_rank=140, q_rank=70)
    elif case == "all_experts":
        mlp = O.moe_cfg(experts=3, top=3, identity=0, shared_ff=0)
    elif case == "only_identity":
        mlp = O.moe_cfg(experts=1, top=4, identity=3)
    elif case == "wide_values":
        m1, m2 = O.mixer_cfg(dim=4, vdim=70), O.mixer_cfg(dim=20, vdim=2, q_rank=5)
    elif case == "odd_sizes":
        m1, m2, kw = O.mixer_cfg(heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=11), O.mixer_cfg(heads=5, dim=3, rot_dim=2, vdim=9, kv_rank=13, q_rank=15), dict(width=20, vocab=37)
        mlp = O.moe_cfg(ff=5, experts=7, top=3, identity=3, shared_ff=9)
    elif case == "many_heads":
        m1, m2 = O.mixer_cfg(heads=20, dim=4, vdim=4), O.mixer_cfg(heads=33, dim=2, rot_dim=2, vdim=3, kv_rank=8, q_rank=8)
    elif case == "no_ff":
        mlp = None
    elif case == "no_yarn_blend":
        m1 = O.mixer_cfg(scaling={"factor": 1.0, "original": 64, "fast": 4.0, "slow": 1.0})
    cfg = O.model_cfg([O.layer(m1, mlp=mlp), O.layer(m2, mlp=mlp)], **kw)
    model, W = make(tmp_path, cfg, device, seed=11)
    prompts = [tokens(n, vocab=cfg["vocab"], seed=n) for n in (13, 22)]
    want = [O.forward(W, cfg, p) for p in prompts]
    for got, w in zip(run_schedule(model, prompts, [[9] + [1] * 4, [22]]), want):
        assert rel_err(got, w) < 1e-4


def test_yarn_constants_reach_the_model(tmp_path):
    """Every constant of the frequency blending changes the logits of a long prompt, and the model follows each."""
    base = dict(YARN)
    toks = tokens(40, seed=2)
    first = None
    for change in ({}, {"factor": 9.0}, {"original": 300}, {"fast": 1.5}, {"slow": 0.2}):
        cfg = O.model_cfg([O.layer(O.mixer_cfg(rot_dim=12, base=400.0, scaling={**base, **change}))])
        model, W = make(tmp_path, cfg, "cpu", seed=2)
        want = O.forward(W, cfg, toks)
        got, = run_schedule(model, [toks], [[40]])
        assert rel_err(got, want) < 1e-4
        if first is None:
            first = want
        else:
            assert rel_err(want, first) > 1e-3, change


# ------------------------------------------------------------------------------------------------------------- generation
@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_through_the_entry_points(device, tmp_path):
    cfg = mixed_cfg()
    W = O.random_weights(cfg, seed=2)
    path = save_model(tmp_path, cfg, W)
    model = load_pretrained(path, dtype=torch.float32, device=device)
    model.kv_page_size = 8
    prompts = [tokens(7, seed=1), tokens(12, seed=2), tokens(3, seed=3)]
    want = [O.greedy(cfg, W, p, 9) for p in prompts]
    assert RequestScheduler(model).generate(prompts, max_new_tokens=9) == want
    assert model.state_cache().live() == 0
    width = max(len(p) for p in prompts)                           # the Generator protocol of the other causal LMs: a left-padded batch
    ids = torch.tensor([[0] * (width - len(p)) + p for p in prompts], device=device)
    mask = torch.tensor([[0] * (width - len(p)) + [1] * len(p) for p in prompts], device=device)
    out = model.generate(ids, attention_mask=mask, max_length=width + 9, do_sample=False, use_cache=True, eos_token_id=None,
                         pad_token_id=0)
    assert [row[width:].tolist() for row in out] == want
    spec = importlib.util.spec_from_file_location("generate_tool", os.path.join(REPO, "tools", "generate.py"))
    tool = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(tool)
    out = tool.main(["--model", path, "--prompts", ";".join(" ".join(map(str, p)) for p in prompts), "--max-new-tokens", "9",
                     "--dtype", "float32", "--device", device])
    assert out == want


@pytest.mark.parametrize("device", DEVICES)
def test_random_init_from_the_config_record(device):
    from libai_b200.config import LazyConfig, instantiate

    node = LazyConfig.load(os.path.join(REPO, "configs", "common", "models", "voduzen.py")).model
    node.cfg.width, node.cfg.vocab = 32, 90
    for lc in node.cfg.layers:
        m = lc["mixer"]
        m.update(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=16)
        if "q_rank" in m:
            m["q_rank"] = 12
        m["rot"]["dims"] = 4
        lc["mlp"]["expert"]["ff"] = lc["mlp"]["shared"]["ff"] = 8
    with param_defaults(dtype=torch.float32, device=device, seed=3):
        model = instantiate(node).eval()
    out = RequestScheduler(model).generate([[1, 2, 3, 4, 5], [7]], max_new_tokens=5)
    assert [len(o) for o in out] == [5, 5] and all(0 <= t < 90 for o in out for t in o)


def test_a_checkpoint_that_lacks_a_tensor_is_refused(tmp_path):
    cfg = O.model_cfg([O.layer(O.mixer_cfg(), mlp=O.moe_cfg())])
    for name in ("l0.mix.sink", "l0.mlp.correction", "l0.mlp.shared.sg"):
        W = O.random_weights(cfg, seed=1)
        del W[name]
        with pytest.raises(RuntimeError, match="lacks tensors"):
            load_pretrained(save_model(tmp_path, cfg, W), dtype=torch.float32, device="cpu")


def test_trace_runner_replays_steps(tmp_path):
    """``bin/trace_run`` on a tiny checkpoint (CPU): a prompt step for two requests, single-token steps, one request ending early;
    the files it writes hold the wanted logits in the order of the entries."""
    import subprocess
    import sys

    import numpy as np

    cfg = mixed_cfg()
    W = O.random_weights(cfg, seed=8)
    path = save_model(tmp_path, cfg, W)
    a, b = tokens(9, seed=4), tokens(6, seed=5)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [0, 6]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[7:8], "want": []}, {"id": "b", "tokens": b[5:6], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[8:9], "want": [0]}], "end": ["a"]}]
    out = os.path.join(str(tmp_path), "out")
    res = subprocess.run([sys.executable, os.path.join(REPO, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", out,
                          "--max-tokens", "64", "--device", "cpu"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [ln for ln in res.stdout.split("\n") if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = O.forward(W, cfg, a), O.forward(W, cfg, b)
    read = lambda s: torch.from_numpy(np.fromfile(os.path.join(out, f"{s}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    assert rel_err(read(0), torch.stack([wa[0], wa[6], wb[4]])) < 1e-4
    assert rel_err(read(1), wb[5:6]) < 1e-4
    assert rel_err(read(2), wa[8:9]) < 1e-4


# ------------------------------------------------------------------------------------------------------ kernels (GPU only)
def cached_rows(dtype, lens, past, C, R, page_size=16):
    """A cache entry whose rows are random, and the step's descriptor."""
    cache = SequenceStateCache("cuda", dtype, page_size=page_size)
    handle = cache.register("paged", channels=LF.row_channels(C, R), taps=1, conv_channels=0)
    slots = cache.allocate(len(lens))
    cache.prepare(slots, [a + b for a, b in zip(lens, past)])
    bufs = cache.buffers(handle)
    bufs["pool"].copy_(torch.randn(bufs["pool"].shape, device="cuda").to(dtype))
    return bufs["pool"], bufs["table"], RaggedBatch(lens, slots, past, "cuda")


SIZES = [(8, 64, 16, 48, 104), (3, 32, 24, 40, 56), (16, 128, 64, 128, 512), (5, 48, 24, 80, 40), (2, 96, 32, 128, 256), (1, 16, 8, 16, 24),
         (18, 24, 8, 40, 136), (2, 192, 64, 256, 72), (4, 64, 64, 192, 640)]


@pytest.mark.gpu
@pytest.mark.parametrize("H,D,R,V,C", SIZES)
@pytest.mark.parametrize("sink", [False, True])
def test_every_form_of_the_attention_agrees(H, D, R, V, C, sink):
    """Expanded (generic and tensor-core) and absorbed (generic and tensor-core, one part and many) attention on the same cache, in
    fp32 and in bf16: ragged lengths, continued sequences, tiles that end inside a page."""
    torch.manual_seed(0)
    lens, past = [70, 1, 37], [0, 45, 90]
    T = sum(lens)
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 2.5e-2)):
        pool, table, rb = cached_rows(dtype, lens, past, C, R)
        q = (1.5 * torch.randn(T, H * (D + R), device="cuda")).to(dtype)
        uk, uv = (torch.randn(H * D, C, device="cuda") / C ** 0.5).to(dtype), (torch.randn(H * V, C, device="cuda") / C ** 0.5).to(dtype)
        ang = torch.rand(T, R // 2, device="cuda") * 6
        cs = torch.stack([ang.cos(), ang.sin()], -1).contiguous()
        sk = torch.randn(H, device="cuda") + 1 if sink else None
        args = (H, D, R, V, C, (D + R) ** -0.5)
        lat, off = LF.latent_rows(pool, table, rb, None)
        kv = torch.nn.functional.linear(lat[:, :C].float(), torch.cat([uk, uv]).float()).to(dtype)
        new = lambda: torch.full((T, H * V), float("nan"), device="cuda", dtype=dtype)
        want = LF.latent_prompt(q, kv, lat, off, cs, rb, new(), *args, sink=sk, mma=False).float()
        assert bool(torch.isfinite(want).all())
        forms = {f"absorbed {parts} {mma}": LF.latent_absorbed(q, uk, uv, cs, pool, table, rb, new(), *args, sink=sk, parts=parts, mma=mma)
                 for parts in (1, 3, 40, None) for mma in ((False, True) if dtype == torch.bfloat16 else (False,))}
        if dtype == torch.bfloat16:
            assert LF.prompt_mma_eligible(q, kv, lat, want.to(dtype), D, R, V, C)
            forms["prompt mma"] = LF.latent_prompt(q, kv, lat, off, cs, rb, new(), *args, sink=sk, tc=False)
        for name, got in forms.items():
            assert torch.allclose(got.float(), want, atol=tol, rtol=tol), (name, dtype, float((got.float() - want).abs().max()))
            assert float((got.float() - want).abs().mean()) < tol / 8, name


@pytest.mark.gpu
@pytest.mark.parametrize("H,D,R,V,C", [(3, 64, 16, 64, 40), (2, 64, 64, 128, 96), (4, 128, 24, 64, 72), (5, 128, 64, 128, 256), (1, 64, 8, 64, 16)])
@pytest.mark.parametrize("gain", [1.0, 8.0])
def test_tcgen05_prompts_match_the_generic_kernel(H, D, R, V, C, gain):
    """bf16 prompts on the tcgen05 kernel: several key tiles, tiles that end inside a sequence, continued sequences, a sequence of one
    token, scores that grow along the sequence so that running maxima move, with and without a sink."""
    torch.manual_seed(1)
    lens, past = [300, 1, 129, 128, 70], [0, 250, 383, 0, 61]
    T = sum(lens)
    pool, table, rb = cached_rows(torch.bfloat16, lens, past, C, R)
    lat, off = LF.latent_rows(pool, table, rb, None)
    kv = torch.randn(lat.shape[0], H * (D + V), device="cuda")
    kv[:, :H * D] *= torch.linspace(0.2, 1.5, lat.shape[0], device="cuda")[:, None]
    kv = kv.to(torch.bfloat16)
    q = (gain * torch.randn(T, H * (D + R), device="cuda")).to(torch.bfloat16)
    ang = torch.rand(T, R // 2, device="cuda") * 6
    cs = torch.stack([ang.cos(), ang.sin()], -1).contiguous()
    if gain > 1:                                                    # large scores: quarter turns, so that no kernel rounds a rotated query
        cs = cs.round().where(cs.abs() == cs.abs().amax(-1, keepdim=True), torch.zeros_like(cs)).sign().contiguous()
    for sk in (None, torch.randn(H, device="cuda") + 2):
        args = (H, D, R, V, C, (D + R) ** -0.5)
        new = lambda: torch.full((T, H * V), float("nan"), device="cuda", dtype=torch.bfloat16)
        want = LF.latent_prompt(q, kv, lat, off, cs, rb, new(), *args, sink=sk, mma=False).float()
        assert LF.prompt_tc_eligible(q, kv, lat, new(), D, R, V, C, 0.1)
        got = LF.latent_prompt(q, kv, lat, off, cs, rb, new(), *args, sink=sk, tc=True).float()
        other = LF.latent_prompt(q, kv, lat, off, cs, rb, new(), *args, sink=sk, tc=False).float()
        for name, g in (("tcgen05", got), ("mma.sync", other)):
            assert torch.allclose(g, want, atol=3e-2, rtol=3e-2), (name, float((g - want).abs().max()))
            assert float((g - want).abs().mean()) < 3e-3, name
        assert not torch.equal(got, other)                          # the two did run different kernels


@pytest.mark.gpu
def test_bf16_model_on_the_tcgen05_path(tmp_path, monkeypatch):
    """A whole bf16 model whose sizes the tcgen05 prompt kernel takes: against the oracle, and against the same model kept off it."""
    cfg = O.model_cfg([O.layer(O.mixer_cfg(heads=2, dim=64, rot_dim=16, vdim=64, kv_rank=40, scale=0.11, scaling=YARN)),
                       O.layer(O.mixer_cfg(heads=3, dim=64, rot_dim=32, vdim=64, kv_rank=48, q_rank=40, scale=0.1))], width=64)
    W = O.random_weights(cfg, seed=5)
    model = load_pretrained(save_model(tmp_path, cfg, W), dtype=torch.bfloat16, device="cuda")
    model.kv_page_size = 16
    prompts = [tokens(170, seed=1), tokens(33, seed=2)]
    want = [O.forward(W, cfg, p) for p in prompts]
    cuts = [[140, 20] + [1] * 10, [33]]
    fast = run_schedule(model, prompts, cuts)
    monkeypatch.setattr(LF, "prompt_tc_eligible", lambda *a: False)
    slow = run_schedule(model, prompts, cuts)
    for f, s_, w in zip(fast, slow, want):
        assert rel_err(f, w) < 1e-1 and rel_err(s_, w) < 1e-1
        assert rel_err(f, s_.float().cpu()) < 5e-2
    assert not torch.equal(fast[0], slow[0])                       # the two paths did run different kernels


@pytest.mark.gpu
@pytest.mark.parametrize("experts,identity,top,ff,shared", [(8, 2, 3, 64, 48), (5, 1, 2, 40, 0), (12, 4, 6, 32, 64)])
def test_bf16_experts_on_the_grouped_products(experts, identity, top, ff, shared):
    """The bf16 forms (grouped tensor-core products on sorted rows; pairs) with identity experts, against the oracle on the same
    rounded inputs, through the residual kernel."""
    width, rows, p = 64, 300, "l0.mlp."
    mc = O.moe_cfg(ff=ff, experts=experts, top=top, identity=identity, shared_ff=shared)
    W = O.random_weights(O.model_cfg([O.layer(O.mixer_cfg(), mlp=mc)], width=width), seed=8)
    mod, sh = build_moe(mc, width, W, p, "cuda", torch.bfloat16)
    h = torch.randn(rows, width, generator=torch.Generator().manual_seed(3)).to(torch.bfloat16)
    want = h.double() + O.centred_norm(O.feed_forward(h.double(), W, p, mc), W["l0.norm2"], 1e-5)
    hd = h.cuda()
    norm = W["l0.norm2"].to(torch.bfloat16).cuda()
    for graph_safe in (False, True):
        with torch.no_grad():
            x = h.float().cuda()
            r = mod.run(hd, graph_safe=graph_safe)
            gate = (hd.float() @ sh.sg[0].float()) if sh is not None else None
            PF.outnorm_residual(x, norm, 1e-5, y=sh(hd) if sh is not None else None, gate=gate, y2=r.y, pos=r.pos, cw=r.wts, keep=r.keep)
        assert float((x.cpu().double() - want).abs().max()) < 6e-2 and float((x.cpu().double() - want).abs().mean()) < 5e-3


@pytest.mark.gpu
def test_serving_precision_and_graphed_steps(tmp_path):
    """bf16 against the oracle (no experts: a close router call would flip a position), on sizes that the tensor-core kernels take and on
    sizes they refuse; a replayed single-token step computes exactly what an eager one does."""
    for name, m1, m2 in (("mma", O.mixer_cfg(heads=4, dim=32, rot_dim=16, vdim=24, kv_rank=40, scale=0.14, scaling=YARN),
                          O.mixer_cfg(heads=2, dim=24, rot_dim=8, vdim=32, kv_rank=48, q_rank=40, scale=0.18)),
                         ("generic", O.mixer_cfg(heads=3, dim=7, rot_dim=6, vdim=9, kv_rank=13), O.mixer_cfg(heads=2, dim=9, rot_dim=2, vdim=5, kv_rank=11, q_rank=10))):
        cfg = O.model_cfg([O.layer(m1), O.layer(m2), O.layer(m1)], width=64)
        W = O.random_weights(cfg, seed=3)
        model = load_pretrained(save_model(tmp_path, cfg, W, name), dtype=torch.bfloat16, device="cuda")
        model.kv_page_size = 8
        prompts = [tokens(n, seed=n) for n in (24, 9, 90)]
        want = [O.forward(W, cfg, p) for p in prompts]
        cuts = [[10] + [1] * 14, [5] + [1] * 4, [75] + [1] * 15]
        eager = run_schedule(model, prompts, cuts, cuda_graphs=False)
        graphed = run_schedule(model, prompts, cuts, cuda_graphs=True)
        for e, g_, w in zip(eager, graphed, want):
            assert rel_err(e, w) < 1e-1
            assert float(torch.tensor([rel_err(e[i:i + 1], w[i:i + 1]) for i in range(len(w))]).median()) < 3e-2
            assert rel_err(g_, e.float().cpu()) < 1e-6


@pytest.mark.gpu
def test_graphed_steps_with_experts(tmp_path):
    """Single-token steps with experts replay from a CUDA graph, also across a page border and while the cache grows."""
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, "cuda", page_size=4)
    prompts = [tokens(n, seed=n) for n in (40, 33)]
    cuts = [[5] + [1] * 35, [3] + [1] * 30]
    for got, p in zip(run_schedule(model, prompts, cuts, cuda_graphs=True), prompts):
        assert rel_err(got, O.forward(W, cfg, p)) < 1e-4
