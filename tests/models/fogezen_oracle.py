"""A plain float64 implementation of Fogezen, one function per mechanism, written from the model's equations only: whole sequences
at once, no cache, no batching, no code shared with the framework.  The tests compare the framework with it.

Notation: ``h`` ``[n, width]`` are the inputs of one sequence, ``W`` the dictionary of checkpoint tensors (float64), ``p`` a tensor name
prefix, ``m`` the part of the configuration that describes the mechanism."""
import math

import torch

F64 = torch.float64


# ---------------------------------------------------------------------------------------------------------------- helpers
def unit_rms(t, eps):
    return t / torch.sqrt((t * t).mean(-1, keepdim=True) + eps)


def centred_norm(t, w, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return unit_rms(t, eps) * (1.0 + w)


def plain_norm(t, w, eps):
    return unit_rms(t, eps) * w


def rotate_pairs(t, first, dims, base):
    """``t`` ``[n, heads, D]`` at the positions ``first …``: the channels (2i, 2i + 1) turn together."""
    out = t.clone()
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        for r in range(t.shape[0]):
            a = (first + r) * f
            u, v = t[r, :, 2 * i], t[r, :, 2 * i + 1]
            out[r, :, 2 * i] = u * math.cos(a) - v * math.sin(a)
            out[r, :, 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return out


def temperature(pos, qt):
    return 1.0 + qt["coef"] * math.log(math.floor((pos + 1) / qt["every"]) + 1.0) if qt else 1.0


def softmax_over(q, k, v, visible, scale):
    """``q`` ``[n, H, D]``, ``k`` ``[n, G, D]``, ``v`` ``[n, G, V]``; ``visible(i)`` = first position that the query at i sees."""
    n, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for i in range(n):
        lo = visible(i)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[lo:i + 1, g]
    return out.reshape(n, -1)


# ----------------------------------------------------------------------------------------------------------------- mixers
def attention(h, W, p, m):
    """Softmax attention over the whole past, biased projections, no rotation, queries scaled by their position."""
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(n, H, D)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(n, G, D)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(n, G, V)
    q = q * torch.tensor([temperature(i, m.get("q_temp")) for i in range(n)], dtype=F64)[:, None, None]
    return softmax_over(q, k, v, lambda i: 0, m["scale"]) @ W[p + "o"].T


def chunk_attention(h, W, p, m, eps):
    """Softmax attention inside chunks of the sequence, normed and rotated heads, channel-wise output gate."""
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {}
    turn = lambda t: rotate_pairs(t, 0, rot.get("dims", 0), rot.get("base", 1.0))
    q = turn(plain_norm((h @ W[p + "q"].T).view(n, H, D), W[p + "q.norm"], eps))
    k = turn(plain_norm((h @ W[p + "k"].T).view(n, G, D), W[p + "k.norm"], eps))
    v = (h @ W[p + "v"].T).view(n, G, V)
    size = m["mask"]["size"]
    o = softmax_over(q, k, v, lambda i: (i // size) * size, m["scale"])
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def memory_gates(h, W, p, m):
    """Log input and log forget gates, ``[n, H]`` each."""
    cap = m["gate_cap"]
    i = cap * torch.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = cap * torch.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap)
    return i, torch.where(f > 0, -torch.log1p(torch.exp(-f)), f - torch.log1p(torch.exp(f)))


def memory_read(q, k, v, i, f):
    """The matrix memory of xLSTM, token by token: ``q``, ``k`` ``[n, H, D]``, ``v`` ``[n, H, V]``, log gates ``[n, H]`` → ``[n, H, V]``."""
    n, H, D = q.shape
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for h in range(H):
        S, z, mx = torch.zeros(D, v.shape[2], dtype=F64), torch.zeros(D, dtype=F64), 0.0
        for t in range(n):
            new = max(float(f[t, h]) + mx, float(i[t, h]))
            keep, put = math.exp(float(f[t, h]) + mx - new), math.exp(float(i[t, h]) - new)
            S = keep * S + put * torch.outer(k[t, h], v[t, h])
            z = keep * z + put * k[t, h]
            mx = new
            out[t, h] = (S.T @ q[t, h]) / (max(abs(float(z @ q[t, h])), math.exp(-mx)) + 1e-6)
    return out


def memory(h, W, p, m, eps):
    n = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(n, H, D) * D ** -0.5
    k = (h @ W[p + "k"].T).view(n, H, D)
    v = (h @ W[p + "v"].T).view(n, H, V)
    o = unit_rms(memory_read(q, k, v, *memory_gates(h, W, p, m)), eps).reshape(n, H * V)
    return (o * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(h, W, p, m, eps):
    a = plain_norm(chunk_attention(h, W, p + "left.", m["left"], eps), W[p + "left.out"], eps)
    b = plain_norm(memory(h, W, p + "right.", m["right"], eps), W[p + "right.out"], eps)
    return 0.5 * (a + b)


# ----------------------------------------------------------------------------------------------------------- feed-forward
def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ------------------------------------------------------------------------------------------------------------------ model
def block(x, W, p, lc, mult, eps):
    h = centred_norm(x, W[p + "norm1"], eps)
    y = attention(h, W, p + "mix.", lc["mixer"]) if lc["type"] == "attention" else parallel(h, W, p + "mix.", lc["mixer"], eps)
    x = x + mult * centred_norm(y, W[p + "norm1b"], eps)
    if lc.get("mlp"):
        y = feed_forward(centred_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
        x = x + mult * centred_norm(y, W[p + "norm2b"], eps)
    return x


def runs(cfg):
    """``(layer, pass or None)`` in execution order; ``pass`` is set on the first layer of a pass."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(toks, W, cfg, collect=None):
    """Logits ``[n, vocab]``; ``collect`` receives the residual after every layer run."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(toks)] * cfg["embedding"]["scale"]
    for i, t in runs(cfg):
        if t is not None:
            x = x + W["loop.step"][t]
        x = block(x, W, f"l{i}.", cfg["layers"][i], cfg["residual_mult"], eps)
        if collect is not None:
            collect.append(x.clone())
    return centred_norm(x, W["final.norm"], eps) @ W["embed"].T


# -------------------------------------------------------------------------------------------------------- random models
def attention_cfg(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, coef=0.5, every=3):
    out = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if every:
        out["q_temp"] = {"coef": coef, "every": every}
    return out


def parallel_cfg(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.35, size=7, rot=6, base=500.0, mheads=3, mdim=5, mvdim=4, cap=9.0):
    return dict(left=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask={"size": size}, rot={"dims": rot, "base": base}),
                right=dict(heads=mheads, dim=mdim, vdim=mvdim, gate_cap=cap))


def layer(mixer, ff=20):
    return dict(type="parallel" if "left" in mixer else "attention", mixer=mixer, mlp={"kind": "dense", "ff": ff} if ff else None)


def model_cfg(layers, vocab=50, width=24, mult=0.4, scale=5.0, eps=1e-5, loop=None):
    out = dict(architecture="Fogezen", vocab=vocab, width=width, layers=layers, residual_mult=mult, embedding={"scale": scale}, norm={"eps": eps})
    if loop:
        out["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return out


def shapes(cfg):
    """Name → shape of every tensor of a model."""
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "final.norm": (w,)}
    if cfg.get("loop"):
        out["loop.step"] = (cfg["loop"]["times"], w)
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        out.update({p + "norm1": (w,), p + "norm1b": (w,)})
        if lc.get("mlp"):
            ff = lc["mlp"]["ff"]
            out.update({p + "norm2": (w,), p + "norm2b": (w,), p + "mlp.gate": (ff, w), p + "mlp.up": (ff, w), p + "mlp.down": (w, ff)})
        q = p + "mix."
        a = m if lc["type"] == "attention" else m["left"]
        H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        r = q if lc["type"] == "attention" else q + "left."
        out.update({r + "q": (H * D, w), r + "k": (G * D, w), r + "v": (G * V, w), r + "o": (w, H * V)})
        if lc["type"] == "attention":
            out.update({r + "q.b": (H * D,), r + "k.b": (G * D,), r + "v.b": (G * V,)})
            continue
        out.update({r + "q.norm": (D,), r + "k.norm": (D,), r + "g": (H * V, w), r + "out": (w,)})
        b, r = m["right"], q + "right."
        H, D, V = b["heads"], b["dim"], b["vdim"]
        out.update({r + "q": (H * D, w), r + "k": (H * D, w), r + "v": (H * V, w), r + "g": (H * V, w), r + "o": (w, H * V), r + "norm": (H * V,),
                    r + "i": (H, w), r + "i.b": (H,), r + "f": (H, w), r + "f.b": (H,), r + "out": (w,)})
    return out


def random_weights(cfg, seed=0):
    """bfloat16 numbers as float64."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(*shape, generator=g)
        last = name.split(".")[-1]
        if name.endswith(("q.norm", "k.norm", "right.norm", ".out")):
            t = 1.0 + 0.3 * t
        elif last in ("norm", "norm1", "norm1b", "norm2", "norm2b"):
            t = 0.2 * t
        elif name.endswith("f.b"):
            t = 1.5 + t
        elif name.endswith(".b") or name == "loop.step":
            t = 0.5 * t
        elif name == "embed":
            t = 0.3 * t
        else:
            t = t * 1.2 / math.sqrt(shape[-1])
        W[name] = t.to(torch.bfloat16).to(F64)
    return W


def greedy(cfg, W, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(toks, W, cfg)[-1].argmax()))
    return toks[len(prompt):]
