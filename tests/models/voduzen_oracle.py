"""A plain float64 implementation of Voduzen, one function per mechanism, written from the model's equations only: whole
sequences at once, no cache, no batching, no code shared with the framework.  The tests compare the framework with it.

Notation: ``x`` ``[n, width]`` is the residual of one sequence, ``W`` the dictionary of checkpoint tensors (float64), ``p`` a tensor
name prefix, ``m`` the part of the configuration that describes the mechanism."""
import math

import torch

F64 = torch.float64


# ---------------------------------------------------------------------------------------------------------------- helpers
def unit_rms(t, eps):
    return t / torch.sqrt((t * t).mean(-1, keepdim=True) + eps)


def centred_norm(t, w, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return unit_rms(t, eps) * (1.0 + w)


def pair_frequencies(dims, base, scaling=None):
    """Angular frequency of every rotated pair and the factor on cos and sin (YaRN blending when ``scaling`` is given)."""
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freq, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def dim_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(t, rot):
    """``t`` ``[n, heads, R]``, row j at position j: channel 2i turns with channel 2i + 1 for i < dims / 2; the rest passes."""
    dims = (rot or {}).get("dims", 0)
    if not dims:
        return t
    freq, mag = pair_frequencies(dims, rot["base"], rot.get("scaling"))
    out = t.clone()
    for pos in range(t.shape[0]):
        for i, f in enumerate(freq):
            c, s = mag * math.cos(pos * f), mag * math.sin(pos * f)
            u, v = t[pos, :, 2 * i], t[pos, :, 2 * i + 1]
            out[pos, :, 2 * i] = u * c - v * s
            out[pos, :, 2 * i + 1] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------------------------ mixers
def attention_inputs(x, W, p, m, eps):
    """Queries and keys ``[n, H, dim + rot_dim]`` and values ``[n, H, vdim]``."""
    n, H, D, R, V = x.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    if "q_rank" in m:
        q = (unit_rms(x @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T
    else:
        q = x @ W[p + "q"].T
    q = q.view(n, H, D + R)
    down = x @ W[p + "dkv"].T
    c = unit_rms(down[:, :m["kv_rank"]], eps) * W[p + "dkv.norm"]
    kr = rotate_pairs(down[:, None, m["kv_rank"]:], m.get("rot"))
    k = torch.cat([(c @ W[p + "uk"].T).view(n, H, D), kr.expand(n, H, R)], -1)
    q = torch.cat([q[..., :D], rotate_pairs(q[..., D:], m.get("rot"))], -1)
    return q, k, (c @ W[p + "uv"].T).view(n, H, V)


def mixer(x, W, p, m, eps, sink):
    n, H, V = x.shape[0], m["heads"], m["vdim"]
    q, k, v = attention_inputs(x, W, p, m, eps)
    out = torch.zeros(n, H, V, dtype=F64)
    for i in range(n):
        for h in range(H):
            s = (k[: i + 1, h] @ q[i, h]) * m["scale"]
            top = s.max()
            e = torch.exp(s - top)
            denom = e.sum() + (torch.exp(W[p + "sink"][h] - top) if sink else 0.0)
            out[i, h] = (e / denom) @ v[: i + 1, h]
    return out.reshape(n, H * V) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------------------ feed-forward
def square_ff(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def route(h, W, p, m):
    """One token ``h`` ``[width]``: the chosen expert numbers and their weights."""
    r = m["router"]
    z = W[p + "router"] @ h
    e = torch.exp(z - z.max())
    s = e / e.sum()
    order = torch.sort(s + W[p + "correction"], descending=True, stable=True).indices[: r["top"]]
    return [int(i) for i in order], [float(s[i]) for i in order]


def feed_forward(x, W, p, m):
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        chosen, weights = route(x[t], W, p, m)
        for e, w in zip(chosen, weights):
            out[t] += w * (square_ff(x[t], W, p + f"e{e}.") if e < m["router"]["experts"] else x[t])
        if m.get("shared"):
            gate = 1.0 / (1.0 + math.exp(-float(W[p + "shared.sg"][0] @ x[t])))
            out[t] += gate * square_ff(x[t], W, p + "shared.")
    return out


# ------------------------------------------------------------------------------------------------------------------- model
def forward(W, cfg, tokens, tap=None):
    """Logits ``[n, vocab]`` of one sequence; ``tap(layer, x)`` sees the residual after every layer."""
    W = {k: v.to(F64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(list(tokens))] * cfg["embedding"]["scale"]
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = mixer(x, W, p + "mix.", lc["mixer"], eps, sink=lc["type"] == "latent_attention")
        x = x + centred_norm(y, W[p + "norm1"], eps)
        if lc.get("mlp"):
            x = x + centred_norm(feed_forward(x, W, p + "mlp.", lc["mlp"]), W[p + "norm2"], eps)
        if tap is not None:
            tap(i, x)
    return centred_norm(x, W["final.norm"], eps) @ W["head"].T * cfg["logit_scale"]


# ------------------------------------------------------------------------------------------------- small models for tests
def mixer_cfg(heads=3, dim=6, rot_dim=4, vdim=10, kv_rank=12, q_rank=None, scale=0.3, base=50.0, scaling=None, rot_dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dim if rot_dims is None else rot_dims, "base": base}}
    if q_rank is not None:
        m["q_rank"] = q_rank
    if scaling:
        m["rot"]["scaling"] = dict(scaling)
    return m


def moe_cfg(ff=10, experts=5, top=2, identity=2, shared_ff=7):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}}
    if shared_ff:
        m["shared"] = {"ff": shared_ff}
    return m


def layer(m, mlp=None):
    return {"type": "latent_attention_2" if "q_rank" in m else "latent_attention", "mixer": m, "mlp": mlp}


def model_cfg(layers, vocab=50, width=16, eps=1e-5, embedding_scale=3.0, logit_scale=0.7):
    return {"architecture": "Voduzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embedding_scale},
            "logit_scale": logit_scale, "layers": layers}


def random_weights(cfg, seed=0):
    """bf16-representable float64 weights of a configuration."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, gain=1.0, mean=0.0):
        fan = shape[-1] if len(shape) > 1 else 1
        return (torch.randn(*shape, generator=g) * gain / math.sqrt(fan) + mean).to(torch.bfloat16).to(F64)

    n = cfg["width"]
    W = {"embed": rnd(cfg["vocab"], n, gain=math.sqrt(n) * 0.4), "final.norm": rnd(n, gain=0.2), "head": rnd(cfg["vocab"], n, gain=2.0)}
    for i, lc in enumerate(cfg["layers"]):
        m, p = lc["mixer"], f"l{i}.mix."
        H, D, R, V, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        W[f"l{i}.norm1"] = rnd(n, gain=0.2)
        if "q_rank" in m:
            W[p + "dq"], W[p + "dq.norm"] = rnd(m["q_rank"], n), rnd(m["q_rank"], gain=0.2, mean=1.0)
            W[p + "uq"] = rnd(H * (D + R), m["q_rank"], gain=1.5)
        else:
            W[p + "q"] = rnd(H * (D + R), n, gain=1.5)
            W[p + "sink"] = rnd(H, gain=1.5)
        W[p + "dkv"], W[p + "dkv.norm"] = rnd(C + R, n, gain=1.5), rnd(C, gain=0.2, mean=1.0)
        W[p + "uk"], W[p + "uv"], W[p + "o"] = rnd(H * D, C, gain=1.5), rnd(H * V, C), rnd(n, H * V)
        if lc.get("mlp"):
            f, p = lc["mlp"], f"l{i}.mlp."
            r = f["router"]
            total = r["experts"] + r.get("identity", 0)
            W[f"l{i}.norm2"] = rnd(n, gain=0.2)
            W[p + "router"], W[p + "correction"] = rnd(total, n, gain=2.0), rnd(total, gain=0.15)
            for e in range(r["experts"]):
                W[p + f"e{e}.up"], W[p + f"e{e}.down"] = rnd(f["expert"]["ff"], n, gain=1.5), rnd(n, f["expert"]["ff"])
            if f.get("shared"):
                W[p + "shared.up"], W[p + "shared.down"] = rnd(f["shared"]["ff"], n, gain=1.5), rnd(n, f["shared"]["ff"])
                W[p + "shared.sg"] = rnd(1, n, gain=1.5)
    return W


def greedy(cfg, W, prompt, n):
    """The ``n`` tokens that greedy decoding appends."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(W, cfg, toks)[-1].argmax()))
    return toks[len(prompt):]
