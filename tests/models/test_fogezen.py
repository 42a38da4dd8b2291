"""Fogezen against a plain float64 oracle (``fogezen_oracle.py``): every mechanism alone, whole prompts, decoding through pages, rings and
recurrent state, prompt portions, ragged batches, pages and slots that are freed and used again, keys far away, at page borders and at
the edges of chunks, the first tokens of a sequence, long decoding, loops, other sizes, generation.

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
from libai_b200.layers import GatedFeedForward, MatrixMemory, PagedAttention, RingAttention
from libai_b200.layers._param import param_defaults
from libai_b200.models.utils.model_loader.auto import load_pretrained
from libai_b200.ops import kv_functional as KF
from libai_b200.ops import lin_functional as LF
from libai_b200.ops import paged_functional as PF
from libai_b200.ops import seq_functional as SF

from . import fogezen_oracle as O

DEVICES = [pytest.param("cpu", id="cpu"), pytest.param("cuda", id="cuda", marks=pytest.mark.gpu)]
REPO = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
F64 = torch.float64


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


def make(tmp_path, cfg, device, dtype=torch.float32, seed=0, weights=None, page_size=4, name="m"):
    """The loaded model (pages of ``page_size`` positions: small, so that short prompts cross many page borders) and its weights."""
    weights = weights if weights is not None else O.random_weights(cfg, seed)
    model = load_pretrained(save_model(tmp_path, cfg, weights, name), dtype=dtype, device=device)
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
    """Every branch once: both mixers in several sizes, with and without temperature, rotation on none / some / all channels, a block
    without a feed-forward, a loop that takes in both kinds of blocks."""
    layers = [O.layer(O.parallel_cfg()),
              O.layer(O.attention_cfg()),
              O.layer(O.parallel_cfg(heads=2, kv_heads=1, dim=6, vdim=9, size=5, rot=0, mheads=1, mdim=7, mvdim=3, cap=4.0), ff=None),
              O.layer(O.attention_cfg(heads=3, kv_heads=3, dim=5, vdim=8, every=0), ff=13),
              O.layer(O.parallel_cfg(heads=3, kv_heads=1, dim=4, vdim=4, size=11, rot=4, base=40.0, mheads=2, mdim=4, mvdim=8))]
    return O.model_cfg(layers, **{"loop": (1, 4, 2), **kw})


# ------------------------------------------------------------------------------------------------------- modules alone
def build_attention(m, width, W, p, device, dtype=torch.float32):
    qt = m.get("q_temp")
    with param_defaults(dtype=dtype, device=device):
        mod = PagedAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], scale=m["scale"], qk_norm=False, bias=True,
                             q_temp=(qt["coef"], qt["every"]) if qt else None)
    return fill(mod, W, p)


def build_chunked(m, width, W, p, eps, device, dtype=torch.float32):
    with param_defaults(dtype=dtype, device=device):
        mod = RingAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], chunk=m["mask"]["size"], scale=m["scale"], rot_dims=m["rot"]["dims"],
                            rot_base=m["rot"]["base"], rot_pairs="interleaved", qk_norm="head", out_gate="channel", eps=eps)
    return fill(mod, W, p)


def build_memory(m, width, W, p, eps, device, dtype=torch.float32):
    with param_defaults(dtype=dtype, device=device):
        mod = MatrixMemory(width, m["heads"], m["dim"], m["vdim"], gate_cap=m["gate_cap"], eps=eps)
    return fill(mod, W, p)


def fill(mod, W, p):
    with torch.no_grad():
        for name, t in mod.named_parameters():
            t.copy_(W[p + name.replace("_norm", ".norm").replace("_b", ".b")])
    return mod


def run_mixer(mod, h, device, lens, page_size=4, dtype=torch.float32, dirty=False):
    """A mixer module alone on one sequence ``h`` ``[n, width]`` fed in the portions ``lens``; returns ``[n, width]``.  ``dirty``: the slot and
    its pages hold numbers of an earlier sequence."""
    cache = SequenceStateCache(device, dtype, page_size=page_size)
    kind, shape = mod.state_spec()
    handle = cache.register(kind, **shape)
    slot = cache.allocate(3)[1:2]                                   # not slot 0
    out, at = [], 0
    for n in lens:
        cache.prepare(slot, [n])
        if dirty and at == 0:
            for name, t in cache.buffers(handle).items():
                if name != "table":
                    t.fill_(7.0)
        rb = RaggedBatch([n], slot, [at], device)
        with torch.no_grad():
            x = h[at:at + n].to(dtype).to(device)
            args = ({},) if isinstance(mod, RingAttention) else ()
            out.append(mod(x, rb, cache.buffers(handle), *args).cpu().double())
        cache.advance(slot, [n])
        at += n
    return torch.cat(out)


PORTIONS = [[21], [1] * 21, [5, 1, 9, 2, 4], [3, 18], [20, 1]]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("lens", PORTIONS)
@pytest.mark.parametrize("m", [O.attention_cfg(), O.attention_cfg(heads=1, kv_heads=1, dim=3, vdim=7, coef=1.5, every=1), O.attention_cfg(every=0),
                               O.attention_cfg(heads=18, kv_heads=1, dim=8, vdim=4, every=5), O.attention_cfg(heads=2, kv_heads=2, dim=70, vdim=140, scale=0.1)],
                         ids=["grouped", "one_head", "no_temperature", "many_heads", "wide"])
def test_attention_alone(device, lens, m):
    width, p = 16, "l0.mix."
    W = O.random_weights(O.model_cfg([O.layer(m)], width=width), seed=3)
    mod = build_attention(m, width, W, p, device)
    h = torch.randn(21, width, generator=torch.Generator().manual_seed(1), dtype=F64)
    want = O.attention(h, W, p, m)
    assert torch.allclose(run_mixer(mod, h, device, lens, dirty=True), want, atol=3e-5)
    far = lambda Wx, mx=m: not torch.allclose(O.attention(h, Wx, p, mx), want, atol=1e-2)      # each ingredient is visible in the result
    for b in ("q.b", "v.b"):
        assert far({**W, p + b: W[p + b] * 0})
    if m.get("q_temp"):
        assert far(W, {**m, "q_temp": None}) and far(W, {**m, "q_temp": dict(m["q_temp"], every=m["q_temp"]["every"] + 1)})


def test_temperature_steps():
    """The floor: the temperature is 1 up to position every − 2, then rises in steps of ``every`` positions."""
    for every, coef in ((1, 0.7), (4, 0.3), (10, 2.0)):
        for p in range(45):
            want = 1 + coef * math.log((p + 1) // every + 1)
            assert KF.query_temperature(p, (coef, float(every))) == pytest.approx(want, rel=1e-12)
            assert O.temperature(p, {"coef": coef, "every": every}) == pytest.approx(want, rel=1e-12)
    assert KF.query_temperature(1000, None) == 1.0


@pytest.mark.gpu
def test_temperature_of_the_kernels():
    """Two keys whose scores differ by a known amount: the attention weight reveals the temperature of every position, over many steps of
    the floor, in the prompt kernels and in the single-token kernels, with ``every`` a power of two and not."""
    for every in (1.0, 3.0, 64.0, 100.0):
        n, D = 700, 16
        q = torch.zeros(n, D, device="cuda")
        q[:, 0] = 0.7
        k, v = torch.zeros(n, D, device="cuda"), torch.zeros(n, D, device="cuda")
        k[0, 0], v[0, 0] = 1.0, 1.0                                 # position 0 stands out by 0.7 · temperature
        pos = torch.arange(n, dtype=F64)
        s = torch.tensor([0.7 * KF.query_temperature(p, (0.9, every)) for p in range(n)], dtype=F64)
        want = s.exp() / (s.exp() + pos)
        rb = RaggedBatch([n], [0], [0], "cuda")
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 6e-3)):
            for kw in ({}, {"tc": False}, {"mma": False}):
                y = torch.empty(n, D, device="cuda", dtype=dtype)
                KF.masked_attention(q.to(dtype), k.to(dtype), v.to(dtype), rb.kv_ext([(0, 0, 0)]), None, rb, y, 1, 1, D, D, 0, 0, 0, 1.0, temp=(0.9, every), **kw)
                s_ = s if dtype == torch.float32 else s * float(q.to(dtype)[0, 0] / 0.7)
                w = want if dtype == torch.float32 else s_.exp() / (s_.exp() + pos)
                assert torch.allclose(y[:, 0].cpu().double(), w, atol=tol, rtol=tol), (every, dtype, kw)
            pool = torch.cat([k, v], 1).to(dtype).view(-1, 7, 2 * D)
            table = torch.arange(pool.shape[0], dtype=torch.int32, device="cuda")[None]
            for p in (0, 1, 2, 62, 63, 64, 98, 99, 100, 127, 128, 299, 300, 699):
                one = RaggedBatch([1], [0], [p], "cuda")
                for splits in (0, 1, 5, None):
                    y = torch.empty(1, D, device="cuda", dtype=dtype)
                    KF.page_attention(q[p:p + 1].to(dtype), pool, table, None, one, y, 1, 1, D, D, 1.0, splits=splits, temp=(0.9, every))
                    assert float(y[0, 0]) == pytest.approx(float(want[p]), rel=3 * tol), (every, dtype, p, splits)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("lens", PORTIONS)
@pytest.mark.parametrize("m", [O.parallel_cfg()["left"], O.parallel_cfg(size=1)["left"], O.parallel_cfg(heads=3, kv_heads=3, dim=7, vdim=5, rot=2, size=4)["left"],
                               O.parallel_cfg(heads=12, kv_heads=1, dim=8, vdim=12, rot=8, size=30)["left"], O.parallel_cfg(rot=0, size=10)["left"],
                               O.parallel_cfg(heads=2, kv_heads=1, dim=132, vdim=36, rot=128, size=9, scale=0.09)["left"]],
                         ids=["grouped", "chunk_of_one", "odd", "chunk_beyond_the_end", "no_rotation", "wide"])
def test_chunked_attention_alone(device, lens, m):
    width, eps, p = 16, 1e-4, "l0.mix.left."
    mx = dict(left=m, right=O.parallel_cfg()["right"])
    W = O.random_weights(O.model_cfg([O.layer(mx)], width=width), seed=4)
    W[p + "q.norm"], W[p + "k.norm"] = (2.0 * W[p + n] for n in ("q.norm", "k.norm"))
    mod = build_chunked(m, width, W, p, eps, device)
    h = torch.randn(21, width, generator=torch.Generator().manual_seed(2), dtype=F64)
    want = O.chunk_attention(h, W, p, m, eps)
    assert torch.allclose(run_mixer(mod, h, device, lens, dirty=True), want, atol=3e-5)
    far = lambda Wx, mx=m: not torch.allclose(O.chunk_attention(h, Wx, p, mx, eps), want, atol=1e-2)
    assert far({**W, p + "g": W[p + "g"] * 0})
    if m["mask"]["size"] > 1:
        assert far({**W, p + "k.norm": W[p + "k.norm"].flip(0)}) and far(W, dict(m, scale=2 * m["scale"]))
        if m["mask"]["size"] < 21:
            assert far(W, dict(m, mask={"size": m["mask"]["size"] + 1}))
        if m["rot"]["dims"]:
            assert far(W, dict(m, rot={"dims": 0})) and far(W, dict(m, rot=dict(m["rot"], base=m["rot"]["base"] * 9 + 3.0))) == (m["rot"]["dims"] > 2)
        assert not far({**W, p + "k": 3.0 * W[p + "k"]})                                            # (keys are normed)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("pairs", [True, False], ids=["interleaved", "half"])
@pytest.mark.parametrize("H,G,D,V,rot,norm", [(3, 1, 8, 8, 8, True), (2, 2, 12, 4, 4, True), (1, 1, 5, 3, 2, False), (9, 3, 64, 48, 64, True), (2, 1, 256, 16, 200, True),
                                              (4, 2, 16, 20, 0, True), (4, 4, 6, 10, 6, False)])
def test_head_preparation(device, pairs, H, G, D, V, rot, norm):
    """Norm, rotation in both pairings and the cache rows (ring that wraps inside the step, pages), for two sequences of which one goes on."""
    g = torch.Generator().manual_seed(1)
    lens, past, eps, L, ps = [5, 9], [0, 6], 1e-3, 6, 3
    T = sum(lens)
    proj = torch.randn(T, (H + G) * D + G * V + 3, generator=g)
    qn, kn = torch.rand(D, generator=g) + 0.5, torch.rand(D, generator=g) + 0.5
    freq, _ = KF.rotary_frequencies(rot, 20.0) if rot else (torch.zeros(0), 1.0)
    for paged in (False, True):
        cache = SequenceStateCache(device, torch.float32, page_size=ps)
        C = G * (D + V)
        handle = cache.register("paged", channels=C, taps=1, conv_channels=0) if paged else cache.register("kv", ring_len=L, first_len=0, channels=C)
        slots = cache.allocate(2)
        cache.prepare(slots, [a + b for a, b in zip(lens, past)])
        bufs = cache.buffers(handle)
        rb = RaggedBatch(lens, slots, past, device)
        d = proj.clone().to(device)
        q, k, v = d[:, :H * D], d[:, H * D:(H + G) * D], d[:, (H + G) * D:(H + G) * D + G * V]
        KF.heads_prepare(q, k, v, qn.to(device) if norm else None, kn.to(device) if norm else None, freq.to(device), eps, rb, H, G, D, V, pairs=pairs,
                         **(dict(pool=bufs["pool"], table=bufs["table"]) if paged else dict(ring=bufs["ring"])))
        p64 = proj.double()
        for b in range(2):
            rows = p64[rb.offsets[b]:rb.offsets[b + 1]]
            for got, heads, w, lo in ((q, H, qn, 0), (k, G, kn, H * D)):
                want = rows[:, lo:lo + heads * D].view(-1, heads, D)
                if norm:
                    want = O.plain_norm(want, w.double(), eps)
                if not pairs and rot:                                # the same rotation on channels put next to each other
                    order = [c for i in range(rot // 2) for c in (i, i + rot // 2)] + list(range(rot, D))
                    want[..., order] = O.rotate_pairs(want[..., order], past[b], rot, 20.0)
                else:
                    want = O.rotate_pairs(want, past[b], rot, 20.0)
                assert torch.allclose(got[rb.offsets[b]:rb.offsets[b + 1]].cpu().double(), want.reshape(-1, heads * D), atol=2e-5)
            full = torch.cat([k, v], 1).cpu()[rb.offsets[b]:rb.offsets[b + 1]]
            for i in range(lens[b]):
                pos = past[b] + i
                if paged:
                    assert torch.equal(bufs["pool"][int(bufs["table"][slots[b], pos // ps]), pos % ps].cpu(), full[i])
                elif lens[b] - i <= L:
                    assert torch.equal(bufs["ring"][slots[b], pos % L].cpu(), full[i])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("lens", PORTIONS)
@pytest.mark.parametrize("m", [O.parallel_cfg()["right"], O.parallel_cfg(mheads=1, mdim=1, mvdim=1)["right"], O.parallel_cfg(mheads=2, mdim=40, mvdim=12, cap=3.0)["right"],
                               O.parallel_cfg(mheads=9, mdim=8, mvdim=20)["right"], O.parallel_cfg(mheads=1, mdim=100, mvdim=130)["right"],
                               O.parallel_cfg(mheads=1, mdim=200, mvdim=140)["right"], O.parallel_cfg(mheads=2, mdim=16, mvdim=65, cap=1.0)["right"]],
                         ids=["small", "ones", "wide_keys", "many_heads", "wide", "several_column_tiles", "odd_values"])
def test_memory_alone(device, lens, m):
    width, eps, p = 16, 1e-5, "l0.mix.right."
    W = O.random_weights(O.model_cfg([O.layer(dict(left=O.parallel_cfg()["left"], right=m))], width=width), seed=5)
    W[p + "i"], W[p + "f"], W[p + "i.b"] = 2.0 * W[p + "i"], 2.0 * W[p + "f"], W[p + "i.b"] + 1.0
    mod = build_memory(m, width, W, p, eps, device)
    h = torch.randn(21, width, generator=torch.Generator().manual_seed(3), dtype=F64)
    want = O.memory(h, W, p, m, eps)
    assert torch.allclose(run_mixer(mod, h, device, lens, dirty=True), want, atol=1e-4)
    far = lambda Wx, mx=m: not torch.allclose(O.memory(h, Wx, p, mx, eps), want, atol=1e-3)
    if m["dim"] > 1:
        assert far({**W, p + "f.b": W[p + "f.b"] - 3.0}) and far({**W, p + "i": -W[p + "i"]}) and far({**W, p + "norm": W[p + "norm"].flip(0) + 0.1})
        assert far({**W, p + "g": W[p + "g"] * 0})


def reader(H, D, V, n, seed, i_shift=0.0, f_shift=1.5):
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(n, H, D, generator=g) * D ** -0.5, torch.randn(n, H, D, generator=g), torch.randn(n, H, V, generator=g)
    return q, k, v, torch.randn(n, 2 * H, generator=g) * 3 + torch.tensor([i_shift] * H + [f_shift] * H)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", ["denominator_by_floor", "denominator_by_keys", "peak_below_zero", "peaks_far_apart", "forgets", "keeps"])
def test_memory_gates_and_normaliser(device, case):
    """The branches of the cell: which of |z·q| and e^(−m) divides, a running maximum that stays at 0 because every gate is below it
    or jumps by the gates' whole range, states that are forgotten at once or kept over 150 tokens — in one step and continued."""
    H, D, V, n, cap = 2, 6, 5, 150, 11.0
    q, k, v, z = reader(H, D, V, n, 7)
    if case == "denominator_by_floor":
        q, z = 0.01 * q, z - torch.tensor([9.0] * H + [0.0] * H)
    elif case == "denominator_by_keys":
        q, k = q.abs() + 0.5, k.abs() + 0.5
        z = z + torch.tensor([5.0] * H + [3.0] * H)
    elif case == "peak_below_zero":
        z = z - torch.tensor([14.0] * H + [-9.0] * H)
    elif case == "peaks_far_apart":
        z[:, :H] = -30.0
        z[40, :H] = z[90, :H] = 30.0
        z[:, H:] += 6.0
    elif case == "forgets":
        z[:, H:] = -40.0
    else:
        z[:, H:] = 60.0
        z[:, :H] -= 4.0
        z[0, :H] = 30.0                                             # the first token is what every later read-out sees most of
    zz = (z / cap).double()
    li, lf = cap * torch.tanh(zz[:, :H]), torch.nn.functional.logsigmoid(cap * torch.tanh(zz[:, H:]))
    want = O.memory_read(q.double(), k.double(), v.double(), li, lf).reshape(n, H * V)
    cell = lambda qx: O.memory_read(qx.double(), k.double(), v.double(), li, lf).reshape(n, H * V)
    if case == "denominator_by_floor":                              # the read-out grows with the query …
        assert torch.allclose(100 * cell(0.01 * q), want, rtol=1e-6)
    if case == "denominator_by_keys":                               # … or its size does not matter
        assert torch.allclose(cell(3 * q), want, rtol=1e-4)
    if case == "keeps":
        gone = v.double().clone()
        gone[0] = 0
        assert float((O.memory_read(q.double(), k.double(), gone, li, lf).reshape(n, -1)[-1] - want[-1]).abs().max()) > 0.1 * float(want[-1].abs().max())
    qd, kd, vd, zd, zb = (t.reshape(n, -1).to(device) for t in (q, k, v, z, torch.zeros(n, 2 * H)))
    zb = torch.zeros(2 * H, device=device)
    for lens in ([n], [31, 1, 1, 32, 33, 52], [100] + [1] * 50):
        cache = SequenceStateCache(device, torch.float32)
        handle = cache.register("recurrent", heads=H, dim=D, vdim=V, taps=1, conv_channels=0, peaks=True)
        slot, at, out = cache.allocate(2)[1:], 0, []
        for t in cache.buffers(handle).values():
            t.fill_(3.0)
        for m in lens:
            rb = RaggedBatch([m], slot, [at], device)
            s = slice(at, at + m)
            out.append(LF.memory_scan(qd[s], kd[s], vd[s], zd[s], zb, H, cap, 1.0, cache.buffers(handle), rb).cpu().double())
            at += m
        err = (torch.cat(out) - want).abs().max(-1).values / want.abs().max()
        # (where |z·q| is small by cancellation, the quotient carries rounding errors of z·q many times enlarged)
        assert float(err.max()) < 1e-3 and float(err.median()) < 2e-6, (case, lens, float(err.max()), float(err.median()))
        ones = torch.ones(H * V, device=device)                     # single tokens through the fused form
        y = torch.empty(1, H * V, device=device)
        rb = RaggedBatch([1], slot, [n], device)
        q2, k2, v2, z2 = (torch.randn(1, t.shape[1], generator=torch.Generator().manual_seed(i)).to(device) for i, t in enumerate((qd, kd, vd, zd)))
        LF.memory_step(q2, k2, v2, z2, zb, H, cap, 0.7, cache.buffers(handle), rb, ones, None, 1e-6, y)
        zc = torch.cat([zd, z2]).cpu().double() / cap
        cat = lambda t, u, w: torch.cat([t.double(), u.cpu().double().view(1, H, w)])
        last = O.memory_read(cat(q, 0.7 * q2, D), cat(k, k2, D), cat(v, v2, V), cap * torch.tanh(zc[:, :H]),
                             torch.nn.functional.logsigmoid(cap * torch.tanh(zc[:, H:])))[-1]
        assert torch.allclose(y.cpu().double().view(H, V), O.unit_rms(last, 1e-6), atol=1e-4)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("n", [24, 19, 1100, 2050])
def test_sandwich_residual(device, n):
    g = torch.Generator().manual_seed(5)
    rows, eps = 7, 1e-2
    x, y, y2 = (torch.randn(rows, n, generator=g) for _ in range(3))
    post, nxt, add, w1, w2 = (0.3 * torch.randn(n, generator=g) for _ in range(5))
    d = lambda t: t.to(device)
    x64 = x.double()
    for two in (False, True):
        for enters in (False, True):
            for opens in (False, True):
                xd, h = d(x.clone()), torch.empty(rows, n, device=device) if opens else None
                v = y.double() if not two else 0.25 * (O.plain_norm(y.double(), w1.double(), eps) + O.plain_norm(y2.double(), w2.double(), eps))
                want = x64 + 0.6 * O.centred_norm(v, post.double(), eps) + (add.double() if enters else 0)
                PF.sandwich_residual(xd, eps, y=d(y), post=d(post), mult=0.6, y2=d(y2) if two else None, branch=(d(w1), d(w2)) if two else None,
                                     branch_scale=0.25, add=d(add) if enters else None, nxt=d(nxt) if opens else None, h=h)
                assert torch.allclose(xd.cpu().double(), want, atol=2e-5)
                if opens:
                    assert torch.allclose(h.cpu().double(), O.centred_norm(want, nxt.double(), eps), atol=2e-5)
    xd, h = d(x.clone()), torch.empty(rows, n, device=device)      # nothing to close
    PF.sandwich_residual(xd, eps, nxt=d(nxt), h=h)
    assert torch.equal(xd.cpu(), x) and torch.allclose(h.cpu().double(), O.centred_norm(x64, nxt.double(), eps), atol=2e-5)
    PF.sandwich_residual(xd, eps, add=d(add), nxt=d(nxt), h=h)
    assert torch.allclose(xd.cpu().double(), x64 + add.double(), atol=1e-6)
    assert torch.allclose(h.cpu().double(), O.centred_norm(x64 + add.double(), nxt.double(), eps), atol=2e-5)


@pytest.mark.parametrize("device", DEVICES)
def test_feed_forward_alone(device):
    W = {k: torch.randn(*s, generator=torch.Generator().manual_seed(i), dtype=F64) * 0.4
         for i, (k, s) in enumerate({"m.gate": (13, 10), "m.up": (13, 10), "m.down": (10, 13)}.items())}
    with param_defaults(dtype=torch.float32, device=device):
        mod = GatedFeedForward(10, 13, "gelu_tanh")
    with torch.no_grad():
        mod.gate_up.copy_(torch.cat([W["m.gate"], W["m.up"]]))
        mod.down.copy_(W["m.down"])
        h = torch.randn(9, 10, generator=torch.Generator().manual_seed(9), dtype=F64) * 2
        got = mod(h.float().to(device)).cpu().double()
    assert torch.allclose(got, O.feed_forward(h, W, "m."), atol=1e-4)
    z = h @ W["m.gate"].T
    erf = (0.5 * z * (1 + torch.erf(z / 2 ** 0.5)) * (h @ W["m.up"].T)) @ W["m.down"].T
    assert not torch.allclose(got, erf, atol=1e-4)


@pytest.mark.parametrize("device", DEVICES)
def test_biases_ride_in_the_stacked_product(device):
    where_ws = [("a", torch.randn(5, 12)), ("b", torch.randn(8, 12)), ("c", torch.randn(3, 12))]
    w, where = SF.fuse_rows(where_ws)
    b = SF.fuse_biases({"a": torch.arange(5.0), "c": torch.arange(3.0) + 10}, where)
    h = torch.randn(4, 12)
    out = SF.linear(h.to(device), w.to(device), b.to(device)).cpu()
    for name, m in where_ws:
        lo, n = where[name]
        bias = {"a": torch.arange(5.0), "b": 0.0, "c": torch.arange(3.0) + 10}[name]
        assert torch.allclose(out[:, lo:lo + n], h @ m.T + bias, atol=1e-5)


# ---------------------------------------------------------------------------------------------------------- whole model
@pytest.mark.parametrize("device", DEVICES)
def test_whole_prompt_with_residuals(device, tmp_path):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device)
    toks = tokens(19)
    residuals, taps = [], []
    want = O.forward(toks, W, cfg, residuals)
    cache = model.state_cache()
    slots = cache.allocate(1)
    got = model.step(torch.tensor(toks, device=device), RaggedBatch([len(toks)], slots, [0], device),
                     tap=lambda i, x: taps.append(x.detach().cpu().double().clone()))
    cache.free(slots)
    assert len(taps) == len(residuals) == 8
    for i, (a, b) in enumerate(zip(taps, residuals)):
        assert torch.allclose(a, b, atol=3e-4), f"residual after block run {i}"
    assert rel_err(got, want) < 1e-4
    plain, = run_schedule(model, [toks], [[19]])                     # without the tap the row that enters a pass rides in the closing kernel
    assert rel_err(plain, want) < 1e-4 and rel_err(plain, got.cpu()) < 1e-6
    for change in (dict(residual_mult=0.5), dict(embedding={"scale": 1.0}), dict(loop=dict(start=1, stop=4, times=1)), dict(norm={"eps": 0.5})):
        assert rel_err(O.forward(toks, W, {**cfg, **change}), want) > 1e-2, change
    assert rel_err(O.forward(toks, {**W, "loop.step": W["loop.step"].flip(0)}, cfg), want) > 1e-2


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("loop", [None, (0, 1, 3), (0, 5, 2), (3, 5, 2), (2, 3, 1), (4, 5, 4)], ids=str)
def test_loops(device, tmp_path, loop):
    """No loop, one that starts at the first block, takes in every block, ends at the last one, runs once."""
    cfg = mixed_cfg(loop=loop)
    model, W = make(tmp_path, cfg, device)
    toks = tokens(14, seed=1)
    want = O.forward(toks, W, cfg)
    for cuts in ([14], [5, 2, 7], [6] + [1] * 8):
        got, = run_schedule(model, [toks], [cuts])
        assert rel_err(got, want) < 1e-4
    assert len(model._handles) == len(O.runs(cfg))                   # every pass has a state of its own


@pytest.mark.parametrize("device", DEVICES)
def test_prefill_against_token_by_token(device, tmp_path):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device)
    toks = tokens(26, seed=3)
    want = O.forward(toks, W, cfg)
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
    got, = run_schedule(model, [toks], [cuts])
    assert rel_err(got, O.forward(toks, W, cfg)) < 1e-4


@pytest.mark.parametrize("device", DEVICES)
def test_ragged_batches_against_each_alone(device, tmp_path):
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, device)
    prompts = [tokens(n, seed=n) for n in (1, 17, 4, 30, 9)]
    want = [O.forward(p, W, cfg) for p in prompts]
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
    assert rel_err(got, O.forward(c, W, cfg)) < 1e-4
    before, pages_before = cache.capacity, cache.num_pages
    many = [(("m", i), tokens(3 + i, seed=10 + i), [2 + i]) for i in range(before + 3)]      # more requests than slots, more rows than pages
    logits = sched.step(many)
    assert cache.capacity > before and cache.num_pages > pages_before
    for row, (_, p, _) in enumerate(many):
        assert rel_err(logits[row:row + 1], O.forward(p, W, cfg)[-1:]) < 1e-4
    got = sched.step([("c", [7], [0])])                            # a request that lived through the growth goes on
    assert rel_err(got, O.forward(c + [7], W, cfg)[-1:]) < 1e-4
    sched.finish(["b", "c"] + [("m", i) for i in range(before + 3)])
    assert cache.live() == 0 and len(cache._free_pages) == cache.num_pages       # every page came back


# ------------------------------------------------------------------------------- far keys, page borders, chunk edges, starts
def sharp_attention(every=0):
    """One attention block built by hand on one-hot embeddings (token 0: filler, 1: the probe that asks, 2: the needle with a value unlike
    every other): the probe's query finds the needle by its content."""
    width = 16
    m = O.attention_cfg(heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, coef=0.2, every=every)
    cfg = O.model_cfg([O.layer(m, ff=None)], vocab=8, width=width, mult=1.0, scale=1.0, eps=1e-6)
    W = O.random_weights(cfg, seed=9)
    W["embed"] = torch.zeros(8, width, dtype=F64)
    for t in range(8):
        W["embed"][t, t] = 1.0
    W["embed"][:, 8:] = 0.2 * torch.randn(8, 8, generator=torch.Generator().manual_seed(1), dtype=F64)
    p = "l0.mix."
    q, k, v = torch.zeros(16, width, dtype=F64), torch.zeros(8, width, dtype=F64), torch.zeros(8, width, dtype=F64)
    q[0, 1] = q[8, 1] = 3.0                                        # the probe looks at channel 0 of the keys …
    k[0, 2] = 2.5                                                  # … which only the needle has (score ≈ 60 above the others after the norm)
    v[0, 0], v[1, 1], v[2, 2], v[3, 2] = 0.5, 0.5, 3.0, -2.0
    W[p + "q"], W[p + "k"], W[p + "v"] = q, k, v
    for b in ("q.b", "k.b", "v.b"):
        W[p + b] = torch.zeros_like(W[p + b])
    W[p + "v.b"] += 0.1
    return cfg, {n: t.to(torch.bfloat16).to(F64) for n, t in W.items()}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("key_at,page_size", [(0, 8), (7, 8), (8, 8), (63, 8), (64, 8), (150, 64), (127, 64), (128, 64), (1, 3), (198, 5)])
def test_one_far_key_decides_the_last_position(device, tmp_path, key_at, page_size):
    n = 200
    cfg, W = sharp_attention(every=50)
    toks = [0] * n
    toks[key_at], toks[-1] = 2, 1
    want = O.forward(toks, W, cfg)[-1:]
    gone = list(toks)
    gone[key_at] = 0
    assert rel_err(O.forward(gone, W, cfg)[-1:], want) > 0.2
    model, _ = make(tmp_path, cfg, device, weights=W, page_size=page_size)
    for cuts in ([n], [n - 1, 1], [key_at + 1] + [1] * (n - key_at - 1) if key_at > 100 else [n - 40] + [1] * 40, [n - 2, 2], [n - 30, 30]):
        got, = run_schedule(model, [toks], [cuts])
        assert rel_err(got[-1:], want) < 1e-3, cuts


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("size", [5, 16, 75])
def test_edges_of_a_chunk(device, tmp_path, size):
    """A needle just inside and just outside the probe's chunk, at its first and last position and in its middle, in prompts, decoded alone,
    with the prompt cut at the edge or elsewhere: only a needle inside is found, and a mask one position off would show."""
    width, p = 16, "l0.mix.left."
    m = O.parallel_cfg(heads=2, kv_heads=1, dim=8, vdim=8, size=size, rot=4, scale=1.0, base=1e4, mheads=1, mdim=2, mvdim=2)
    cfg = O.model_cfg([O.layer(m, ff=None)], vocab=8, width=width, mult=1.0, scale=1.0, eps=1e-6)
    W = O.random_weights(cfg, seed=9)
    W["embed"] = torch.zeros(8, width, dtype=F64)
    for t in range(8):
        W["embed"][t, t] = 1.0
    q, k, v = torch.zeros(16, width, dtype=F64), torch.zeros(8, width, dtype=F64), torch.zeros(8, width, dtype=F64)
    q[5, 1] = q[13, 1] = k[5, 2] = 3.0                             # an unrotated channel; every other token's key points elsewhere
    q[6, 0] = q[14, 0] = k[6, 0] = k[7, 1] = k[6, 3] = 1.0
    v[0, 0], v[1, 1], v[2, 2], v[3, 2] = 0.5, 0.5, 3.0, -2.0
    W[p + "q"], W[p + "k"], W[p + "v"] = q, k, v
    W[p + "q.norm"], W[p + "k.norm"] = torch.full((8,), 2.0, dtype=F64), torch.full((8,), 2.0, dtype=F64)
    for n_ in ("q", "k", "v"):                                     # the recurrent side stays out of the way
        W["l0.mix.right." + n_] = W["l0.mix.right." + n_] * 0
    W = {n_: t.to(torch.bfloat16).to(F64) for n_, t in W.items()}
    model, _ = make(tmp_path, cfg, device, weights=W)
    last = 3 * size - 1
    for ask in (2 * size, 2 * size + 1, last):                     # first, second and last position of the third chunk
        for key_at in sorted({2 * size - 1, 2 * size, size, ask - 1} - {ask}):
            toks = [0] * (ask + 1)
            toks[key_at] = 2
            toks[ask] = 1
            want = O.forward(toks, W, cfg)[-1:]
            gone = list(toks)
            gone[key_at] = 0
            inside = 2 * size <= key_at < ask
            effect = rel_err(O.forward(gone, W, cfg)[-1:], want)
            assert effect > 0.2 if inside else effect < 1e-9, (ask, key_at)
            for cuts in ([ask + 1], [ask, 1], [2 * size, ask + 1 - 2 * size], [2 * size - 2] + [1] * (ask + 3 - 2 * size), [size + 1, ask - size]):
                got, = run_schedule(model, [toks], [cuts])
                assert rel_err(got[-1:], want) < 1e-3, (ask, key_at, cuts)


@pytest.mark.parametrize("device", DEVICES)
def test_the_first_tokens_of_a_sequence(device, tmp_path):
    """The first positions see few keys, a state at zero and a running maximum at 0, whatever the slot and its pages held before."""
    cfg = mixed_cfg()
    W = O.random_weights(cfg, seed=4)
    for i in (0, 2, 4):                                            # strongly negative input gates: the maximum stays at its start for a while
        W[f"l{i}.mix.right.i.b"] = (W[f"l{i}.mix.right.i.b"] - 3.0).to(torch.bfloat16).to(F64)
    model, _ = make(tmp_path, cfg, device, weights=W)
    sched = RequestScheduler(model)
    sched.step([("old", tokens(11, seed=8), [])])                  # leaves rows, states and maxima behind in what comes next
    sched.finish(["old"])
    toks = tokens(6, seed=9)
    want = O.forward(toks, W, cfg)
    for cuts in ([6], [1] * 6, [2, 1, 3]):
        got, = run_schedule(model, [toks], [cuts])
        assert rel_err(got, want) < 1e-4, cuts


@pytest.mark.parametrize("device", DEVICES)
def test_a_far_token_through_the_memory(device, tmp_path):
    """Forget gates near one: the first token reaches the last logits through the matrix memory alone (chunks of 8), 200 positions on."""
    cfg = O.model_cfg([O.layer(O.parallel_cfg(size=8, cap=30.0)), O.layer(O.parallel_cfg(size=8, cap=30.0))])
    W = O.random_weights(cfg, seed=12)
    for i in (0, 1):
        W[f"l{i}.mix.right.f"] *= 0.05
        W[f"l{i}.mix.right.f.b"] = torch.full_like(W[f"l{i}.mix.right.f.b"], 12.0)
        W[f"l{i}.mix.right.i"] *= 0.05
    W = {n: t.to(torch.bfloat16).to(F64) for n, t in W.items()}
    model, _ = make(tmp_path, cfg, device, weights=W)
    toks = tokens(200, seed=6)
    other = [(toks[0] + 1) % 50] + toks[1:]
    want, moved = O.forward(toks, W, cfg), O.forward(other, W, cfg)
    effect = rel_err(moved[-1:], want[-1:])
    assert effect > 1e-3
    for cuts in ([200], [150] + [1] * 50, [63, 64, 2, 71]):
        got, = run_schedule(model, [toks], [cuts])
        assert rel_err(got[-1:], want[-1:]) < effect / 10, cuts


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding(device, tmp_path):
    """Many chunk wraps of the ring, many pages, a long-lived running maximum."""
    cfg = O.model_cfg([O.layer(O.parallel_cfg(size=9)), O.layer(O.attention_cfg(every=20)), O.layer(O.parallel_cfg(size=40))], loop=(0, 2, 2))
    model, W = make(tmp_path, cfg, device, page_size=16)
    toks = tokens(150, seed=4)
    want = O.forward(toks, W, cfg)
    got, = run_schedule(model, [toks], [[10] + [1] * 140])
    assert rel_err(got, want) < 2e-4


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("case", ["one_head", "ungrouped", "many_query_heads", "wide_values", "odd_sizes", "no_ff", "ones", "large_heads", "extra_norms"])
def test_other_sizes(device, tmp_path, case):
    a, b, ff, kw = O.attention_cfg(), O.parallel_cfg(), 20, {}
    if case == "one_head":
        a, b = O.attention_cfg(heads=1, kv_heads=1), O.parallel_cfg(heads=1, kv_heads=1, mheads=1)
    elif case == "ungrouped":
        a, b = O.attention_cfg(kv_heads=4), O.parallel_cfg(kv_heads=4)
    elif case == "many_query_heads":
        a, b = O.attention_cfg(heads=20, kv_heads=2), O.parallel_cfg(heads=16, kv_heads=1, mheads=12)
    elif case == "wide_values":
        a, b = O.attention_cfg(dim=4, vdim=40), O.parallel_cfg(dim=4, rot=4, vdim=70, mdim=3, mvdim=90)
    elif case == "odd_sizes":
        a, b = O.attention_cfg(heads=3, kv_heads=1, dim=5, vdim=7), O.parallel_cfg(heads=3, kv_heads=3, dim=9, vdim=11, rot=2, mheads=5, mdim=3, mvdim=7)
        ff, kw = 11, dict(width=21, vocab=37)
    elif case == "no_ff":
        ff = None
    elif case == "ones":
        a, b, kw = O.attention_cfg(coef=1.0, every=1, scale=1.0), O.parallel_cfg(scale=1.0, size=1, cap=1.0, base=1.0), dict(mult=1.0, scale=1.0)
    elif case == "large_heads":
        a, b = O.attention_cfg(heads=2, kv_heads=1, dim=128, vdim=128, scale=0.1), O.parallel_cfg(heads=2, kv_heads=1, dim=128, vdim=128, rot=64, scale=0.1, mheads=1, mdim=128, mvdim=128)
    cfg = O.model_cfg([O.layer(b, ff), O.layer(a, ff)], **kw)
    W = O.random_weights(cfg, seed=11)
    if case == "extra_norms":                                      # a block without a feed-forward whose checkpoint still carries the norms around it
        cfg["layers"][1]["mlp"] = None
        W = {n: t for n, t in W.items() if not n.startswith("l1.mlp")}
    model, _ = make(tmp_path, cfg, device, weights=W)
    prompts = [tokens(n, vocab=cfg["vocab"], seed=n) for n in (13, 22)]
    want = [O.forward(p, W, cfg) for p in prompts]
    for got, w in zip(run_schedule(model, prompts, [[9] + [1] * 4, [22]]), want):
        assert rel_err(got, w) < 1e-4


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

    node = LazyConfig.load(os.path.join(REPO, "configs", "common", "models", "fogezen.py")).model
    node.cfg.width, node.cfg.vocab = 32, 90
    for lc in node.cfg.layers:
        lc["mlp"]["ff"] = 24
        a = lc["mixer"]["left"] if "left" in lc["mixer"] else lc["mixer"]
        a.update(heads=2, kv_heads=1, dim=8, vdim=8)
        if "left" in lc["mixer"]:
            a["rot"]["dims"], a["mask"]["size"] = 8, 4
            lc["mixer"]["right"].update(heads=2, dim=8, vdim=8)
    with param_defaults(dtype=torch.float32, device=device, seed=3):
        model = instantiate(node).eval()
    out = RequestScheduler(model).generate([[1, 2, 3, 4, 5], [7]], max_new_tokens=5)
    assert [len(o) for o in out] == [5, 5] and all(0 <= t < 90 for o in out for t in o)


def test_a_checkpoint_that_lacks_a_tensor_is_refused(tmp_path):
    cfg = mixed_cfg()
    for name in ("l0.mix.left.q.norm", "l0.mix.right.f.b", "l1.mix.v.b", "l0.mix.left.out", "loop.step", "l1.norm2b"):
        W = O.random_weights(cfg, seed=1)
        del W[name]
        with pytest.raises(RuntimeError, match="lacks tensors"):
            load_pretrained(save_model(tmp_path, cfg, W), dtype=torch.float32, device="cpu")
    with pytest.raises(ValueError, match="loop"):
        bad = mixed_cfg(loop=(1, 6, 2))
        load_pretrained(save_model(tmp_path, bad, O.random_weights(bad, seed=1)), dtype=torch.float32, device="cpu")


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
    wa, wb = O.forward(a, W, cfg), O.forward(b, W, cfg)
    read = lambda s: torch.from_numpy(np.fromfile(os.path.join(out, f"{s}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    assert rel_err(read(0), torch.stack([wa[0], wa[6], wb[4]])) < 1e-4
    assert rel_err(read(1), wb[5:6]) < 1e-4
    assert rel_err(read(2), wa[8:9]) < 1e-4


# ------------------------------------------------------------------------------------------------------ kernels (GPU only)
@pytest.mark.gpu
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 64, 64), (3, 1, 128, 128), (2, 2, 64, 48), (6, 3, 48, 80), (8, 1, 16, 128), (1, 1, 128, 16), (5, 5, 112, 96), (2, 1, 32, 64)])
@pytest.mark.parametrize("mask", [(0, 0), (0, 72), (0, 130), (0, 1), (100, 0), (129, 0)], ids=["causal", "chunk72", "chunk130", "chunk1", "window100", "window129"])
def test_tcgen05_prompts_match_the_generic_kernel(H, G, D, V, mask):
    """bf16 prompts on the tcgen05 kernel: several key tiles, tiles that end inside a sequence or across a chunk's edge, continued
    sequences, a sequence of one token, scores that grow along the sequence so that running maxima move, all kinds of gates,
    temperature, strided operands."""
    torch.manual_seed(1)
    window, chunk = mask
    lens, past = [300, 1, 129, 128, 70], [0, 250, 383, 0, 61]
    T = sum(lens)
    rb = RaggedBatch(lens, [4, 0, 2, 1, 3], past, "cuda")
    ext = rb.kv_ext([(window, chunk, 0)])
    rows = torch.randn(ext.rows, G * (D + V) + 8, device="cuda")
    rows[:, :G * D] *= torch.linspace(0.2, 1.5, ext.rows, device="cuda")[:, None]
    rows = rows.to(torch.bfloat16)
    kmat, vmat = rows[:, :G * D], rows[:, G * D:G * (D + V)]
    qg = torch.randn(T, H * (D + V), device="cuda").to(torch.bfloat16)
    q, wide, narrow = 3 * qg[:, :H * D], qg[:, H * D:], torch.randn(T, H, device="cuda").to(torch.bfloat16)
    new = lambda: torch.full((T, H * V + 8), float("nan"), device="cuda", dtype=torch.bfloat16)[:, :H * V]
    for gate, kw in ((None, {}), (wide, dict(gate_wide=True, out_scale=0.5)), (narrow, dict(temp=(0.4, 60.0))), (None, dict(temp=(0.2, 7.0), out_scale=2.0))):
        args = (q, kmat, vmat, ext, gate, rb)
        sizes = (H, G, D, V, window, chunk, 0, D ** -0.5)
        want = KF.masked_attention(*args, new(), *sizes, mma=False, **kw).float()
        assert KF.tc_eligible(q, kmat, vmat, gate if kw.get("gate_wide") else None, new(), D, V, 0, 0.1, 0.0, False, kw.get("temp"))
        got = KF.masked_attention(*args, new(), *sizes, tc=True, **kw).float()
        assert torch.allclose(got, want, atol=3e-2, rtol=3e-2), float((got - want).abs().max())
        assert float((got - want).abs().mean()) < 3e-3
    if chunk != 1:
        assert not torch.equal(got, want)                           # the two did run different kernels


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,D,V", [(4, 2, 64, 64), (8, 1, 64, 80), (16, 1, 32, 32), (3, 3, 20, 24), (6, 2, 128, 128), (2, 1, 9, 200)])
def test_paged_single_tokens(H, G, D, V):
    """Single-token steps over pages, any number of parts, against the same attention as a prompt step on gathered rows."""
    torch.manual_seed(2)
    past, ps = [0, 1, 63, 64, 500, 2], 16
    B = len(past)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        cache = SequenceStateCache("cuda", dtype, page_size=ps)
        handle = cache.register("paged", channels=G * (D + V), taps=1, conv_channels=0)
        slots = cache.allocate(B + 2)[2:]
        cache.prepare(slots, [p + 1 for p in past])
        bufs = cache.buffers(handle)
        bufs["pool"].copy_(torch.randn(bufs["pool"].shape, device="cuda").to(dtype))
        rb = RaggedBatch([1] * B, slots, past, "cuda")
        q, gate = torch.randn(B, H * D, device="cuda").to(dtype), torch.randn(B, H * V, device="cuda").to(dtype)
        fresh = torch.empty(B, G * D, device="cuda", dtype=dtype)
        kmat, vmat, ext = PF.page_rows(bufs["pool"], bufs["table"], rb, fresh, fresh)
        kw = dict(gate_wide=True, temp=(0.3, 20.0), out_scale=0.7)
        want = KF.masked_attention(q, kmat, vmat, ext, gate, rb, torch.empty(B, H * V, device="cuda", dtype=dtype), H, G, D, V, 0, 0, 0, 0.2, mma=False, **kw)
        for splits in (0, 1, 3, 32, None):
            if splits and not KF.grouped_decode_ok(H, G, D, V):
                continue
            got = KF.page_attention(q, bufs["pool"], bufs["table"], gate, rb, torch.empty_like(want), H, G, D, V, 0.2, splits=splits, **kw)
            assert torch.allclose(got.float(), want.float(), atol=tol, rtol=tol), (dtype, splits)


@pytest.mark.gpu
@pytest.mark.parametrize("H,D,V", [(2, 64, 64), (1, 128, 128), (3, 32, 48), (2, 16, 128), (1, 64, 200), (4, 48, 96), (8, 8, 8), (6, 64, 128), (5, 120, 72)])
def test_memory_prompts_in_bf16(H, D, V):
    """bf16 prompts through the memory against the float64 cell on the same rounded inputs: ragged lengths, continued from a state, with
    gates that move the maximum and gates that keep everything."""
    torch.manual_seed(3)
    lens, past, cap = [200, 1, 64, 130] + 12 * [3], [0, 7, 0, 5] + 12 * [0], 10.0
    T = sum(lens)
    for shift in (0.0, 5.0):
        q, k, v = (torch.randn(T, H * n, device="cuda").to(torch.bfloat16) for n in (D, D, V))
        z = torch.randn(T, 16, device="cuda") * 4
        z[:, 8:] += shift
        zb = torch.zeros(16, device="cuda")
        cache = SequenceStateCache("cuda", torch.bfloat16)
        handle = cache.register("recurrent", heads=H, dim=D, vdim=V, taps=1, conv_channels=0, peaks=True)
        slots = cache.allocate(len(lens) + 1)[1:]
        bufs = cache.buffers(handle)
        prior = {}
        for b, p in enumerate(past):                                # a past of its own for the continued sequences
            if p:
                qp, kp, vp = (torch.randn(p, H * n, device="cuda").to(torch.bfloat16) for n in (D, D, V))
                zp = torch.randn(p, 16, device="cuda")
                LF.memory_scan(qp, kp, vp, zp, zb, 8, cap, D ** -0.5, bufs, RaggedBatch([p], [slots[b]], [0], "cuda"))
                prior[b] = (qp, kp, vp, zp)
        rb = RaggedBatch(lens, slots, past, "cuda")
        start = {n: t.clone() for n, t in bufs.items()}
        assert LF.load_lin_ext().memory_chunk_blocks(q, k, v, rb.B, H, D, V) > 0
        serial = LF.memory_scan(q, k, v, z, zb, 8, cap, D ** -0.5, bufs, rb, chunks=False)
        left = {n: t.clone() for n, t in bufs.items()}
        for n, t in bufs.items():
            t.copy_(start[n])
        got = LF.memory_scan(q, k, v, z, zb, 8, cap, D ** -0.5, bufs, rb).cpu().double()
        assert not torch.equal(got, serial.cpu().double())         # the two did run different kernels …
        for n in ("S", "keys", "peak"):                             # … and leave the same state
            scale = left[n][slots].abs().amax()
            assert float((bufs[n][slots] - left[n][slots]).abs().max()) < 1e-5 * float(scale), n
        for n, t in bufs.items():
            t.copy_(start[n])
        gate, w = torch.randn(T, H * V + 4, device="cuda").to(torch.bfloat16)[:, :H * V], torch.rand(H * V, device="cuda").to(torch.bfloat16)
        y = LF.memory_prompt(q, k, v, z, zb, 8, cap, D ** -0.5, bufs, rb, w, gate, 1e-5, torch.empty(T, H * V, device="cuda", dtype=torch.bfloat16), 0.5)
        want_y = 0.5 * O.unit_rms(got.view(T, H, V), 1e-5).view(T, -1) * w.cpu().double() * torch.sigmoid(gate.cpu().double())
        assert torch.allclose(y.cpu().double(), want_y, atol=2e-2, rtol=1e-2)
        for b in range(len(lens)):
            s = slice(rb.offsets[b], rb.offsets[b + 1])
            parts = [torch.cat([prior[b][i], t[s]]) if b in prior else t[s] for i, t in enumerate((q, k, v, z))]
            q64, k64, v64, z64 = (t.cpu().double() for t in parts)
            n = q64.shape[0]
            li = cap * torch.tanh(z64[:, :H] / cap)
            lf = torch.nn.functional.logsigmoid(cap * torch.tanh(z64[:, 8:8 + H] / cap))
            want = O.memory_read(q64.view(n, H, D) * D ** -0.5, k64.view(n, H, D), v64.view(n, H, V), li, lf)[past[b]:]
            g_ = got[s].view(-1, H, V)
            err = (g_ - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
            assert float(err.max()) < 3e-3 and float(err.median()) < 3e-6, (shift, b, float(err.max()), float(err.median()))


@pytest.mark.gpu
def test_serving_precision_and_graphed_steps(tmp_path):
    """bf16 against the oracle on sizes that the tensor-core kernels take and on sizes they refuse; a replayed single-token step computes
    exactly what an eager one does, also across page borders and chunk edges."""
    tc = [O.layer(O.parallel_cfg(heads=4, kv_heads=2, dim=64, vdim=48, rot=32, size=40, scale=0.12, mheads=2, mdim=32, mvdim=64), 64),
          O.layer(O.attention_cfg(heads=4, kv_heads=1, dim=64, vdim=64, scale=0.12, every=16), 64)]
    generic = [O.layer(O.parallel_cfg(heads=3, kv_heads=1, dim=7, vdim=9, rot=6, size=13), 30), O.layer(O.attention_cfg(heads=3, kv_heads=3, dim=9, vdim=5), 30)]
    for name, layers in (("tc", tc), ("generic", generic)):
        cfg = O.model_cfg(layers, width=64, loop=(0, 2, 2))
        W = O.random_weights(cfg, seed=3)
        model, _ = make(tmp_path, cfg, "cuda", dtype=torch.bfloat16, weights=W, page_size=8, name=name)
        prompts = [tokens(n, seed=n) for n in (24, 9, 170)]
        want = [O.forward(p, W, cfg) for p in prompts]
        cuts = [[10] + [1] * 14, [5] + [1] * 4, [120, 35] + [1] * 15]
        eager = run_schedule(model, prompts, cuts, cuda_graphs=False)
        graphed = run_schedule(model, prompts, cuts, cuda_graphs=True)
        for e, g_, w in zip(eager, graphed, want):
            assert rel_err(e, w) < 6e-2
            assert float(torch.tensor([rel_err(e[i:i + 1], w[i:i + 1]) for i in range(len(w))]).median()) < 2.5e-2
            assert rel_err(g_, e.float().cpu()) < 1e-6


@pytest.mark.gpu
def test_bf16_model_on_and_off_the_tcgen05_path(tmp_path, monkeypatch):
    cfg = O.model_cfg([O.layer(O.parallel_cfg(heads=2, kv_heads=1, dim=64, vdim=64, rot=64, size=100, scale=0.12, mheads=1, mdim=64, mvdim=64), 48),
                       O.layer(O.attention_cfg(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.1, every=32), 48)], width=64)
    model, W = make(tmp_path, cfg, "cuda", dtype=torch.bfloat16, page_size=16)
    prompts = [tokens(170, seed=1), tokens(73, seed=2)]
    want = [O.forward(p, W, cfg) for p in prompts]
    cuts = [[140, 20] + [1] * 10, [73]]
    fast = run_schedule(model, prompts, cuts)
    monkeypatch.setattr(KF, "tc_eligible", lambda *a: False)
    slow = run_schedule(model, prompts, cuts)
    for f, s_, w in zip(fast, slow, want):
        assert rel_err(f, w) < 6e-2 and rel_err(s_, w) < 6e-2
        assert rel_err(f, s_.float().cpu()) < 3e-2
    assert not torch.equal(fast[0], slow[0])                       # the two paths did run different kernels


@pytest.mark.gpu
def test_graphed_steps_of_a_mixed_model(tmp_path):
    """Single-token steps replay from a CUDA graph, also across a page border and while the cache grows."""
    cfg = mixed_cfg()
    model, W = make(tmp_path, cfg, "cuda", page_size=4)
    prompts = [tokens(n, seed=n) for n in (40, 33)]
    cuts = [[5] + [1] * 35, [3] + [1] * 30]
    for got, p in zip(run_schedule(model, prompts, cuts, cuda_graphs=True), prompts):
        assert rel_err(got, O.forward(p, W, cfg)) < 1e-4
