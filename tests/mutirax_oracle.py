"""Plain float64 restatement of the Mutirax design: one function per mechanism, whole sequences, no caches, no batching, no
code shared with the served path.  Slow on purpose: loops over tokens and heads where that is clearest.

Shapes: a sequence is [n, ...]; weights are [out, in] and applied as x @ W.T.  Positions are 0 .. n-1.
"""
import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------ elementary pieces
def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def lin(x, w):
    return x @ w.to(F64).T


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.to(F64)


def dyt(x, W, name):
    """tanh of the scaled input, then weight and bias: no statistics."""
    return torch.tanh(W[name + ".alpha"].to(F64) * x) * W[name].to(F64) + W[name + ".b"].to(F64)


def causal_conv(u, w, b=None):
    """u [n, c], w [c, taps]: the last tap belongs to the token itself; zeros before the sequence."""
    n, taps = u.shape[0], w.shape[1]
    w, out = w.to(F64), torch.zeros_like(u)
    for t in range(n):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += w[:, j] * u[src]
    return out if b is None else out + b.to(F64)


# ------------------------------------------------------------------ rotary positions (halves layout)
def frequencies(dims, base, scaling=None):
    """(frequencies, magnitude of cos and sin)."""
    i = torch.arange(dims // 2, dtype=F64)
    f = float(base) ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim_of(scaling["fast"])), 0), min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, f, mag=1.0):
    """x [n, ..., >= 2 len(f)]: column i of row t is paired with column i + len(f); the others pass."""
    out, m = x.clone(), f.shape[0]
    for t, p in enumerate(positions):
        c, s = mag * torch.cos(float(p) * f), mag * torch.sin(float(p) * f)
        u, v = x[t, ..., :m], x[t, ..., m:2 * m]
        out[t, ..., :m] = u * c - v * s
        out[t, ..., m:2 * m] = v * c + u * s
    return out


# ------------------------------------------------------------------ hyper-connections
def hyper_read(streams, w_in):
    """streams [s, n, d] -> what a sublayer reads [n, d]."""
    return torch.einsum("s,snd->nd", w_in.to(F64), streams)


def hyper_write(streams, mix, w_out, y, m):
    """New stream t = sum over the old streams s of mix[s, t] x_s, plus m out[t] y."""
    return torch.einsum("st,snd->tnd", mix.to(F64), streams) + m * w_out.to(F64)[:, None, None] * y


# ------------------------------------------------------------------ attention kernels of one head
def softmax_attention(q, k, v, scale, sink=None, first=0):
    """q [n - first, d] (positions first ..), k [n, d], v [n, e]; sink: a logit that only joins the denominator."""
    n = k.shape[0]
    out = torch.zeros(n - first, v.shape[1], dtype=F64)
    for i in range(first, n):
        s = (k[:i + 1] @ q[i - first]) * scale
        top = float(s.max()) if sink is None else max(float(s.max()), float(sink))
        e = torch.exp(s - top)
        den = e.sum() + (0.0 if sink is None else math.exp(float(sink) - top))
        out[i - first] = (e @ v[:i + 1]) / den
    return out


# ------------------------------------------------------------------ mixers
def gla_scan(q, k, a, v):
    """q, k, a [n, H, d], v [n, H, e]: S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, S zero at the start."""
    n, H, d = q.shape
    o = torch.zeros(n, H, v.shape[-1], dtype=F64)
    for h in range(H):
        S = torch.zeros(d, v.shape[-1], dtype=F64)
        for t in range(n):
            S = a[t, h][:, None] * S + torch.outer(k[t, h], v[t, h])
            o[t, h] = S.T @ q[t, h]
    return o


def gla_operands(h, W, p, m):
    n, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    z = lin(lin(h, W[p + "a1"]), W[p + "a2"]) + W[p + "a2.b"].to(F64)
    a = sigmoid(z) ** (1.0 / m["tau"])
    return lin(h, W[p + "q"]).view(n, H, d) / math.sqrt(d), lin(h, W[p + "k"]).view(n, H, d), a.view(n, H, d), lin(h, W[p + "v"]).view(n, H, e)


def gla_mixer(h, W, p, m, eps):
    o = rms(gla_scan(*gla_operands(h, W, p, m)), W[p + "norm"], eps).reshape(h.shape[0], -1)
    return lin(o * silu(lin(h, W[p + "g"])), W[p + "o"])


def latent_mixer(h, W, p, m, eps):
    n, H, d, r, e, c = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = list(range(n))
    f, mag = frequencies(r, m["rot"]["base"], m["rot"].get("scaling"))
    q = lin(rms(lin(h, W[p + "dq"]), W[p + "dq.norm"], eps), W[p + "uq"]).view(n, H, d + r)
    kv = lin(h, W[p + "dkv"])
    lat, kr = rms(kv[:, :c], W[p + "dkv.norm"], eps), rotate(kv[:, c:], pos, f, mag)
    k, v = lin(lat, W[p + "uk"]).view(n, H, d), lin(lat, W[p + "uv"]).view(n, H, e)
    qr = rotate(q[..., d:], pos, f, mag)
    gate = sigmoid(lin(h, W[p + "g"]))
    outs = [softmax_attention(torch.cat([q[:, i, :d], qr[:, i]], -1), torch.cat([k[:, i], kr], -1), v[:, i], m["scale"]) * gate[:, i:i + 1]
            for i in range(H)]
    return lin(torch.cat(outs, -1), W[p + "o"])


def conv_attention(h, W, p, m, eps):
    """Keys and queries through a short convolution, normed over the whole projection and rotated; the values are the keys
    as they leave the convolution; a softmax sink per head."""
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = list(range(n))
    f, mag = frequencies(m["rot"]["dims"], m["rot"]["base"])
    q, k = causal_conv(lin(h, W[p + "q"]), W[p + "q.conv"]), causal_conv(lin(h, W[p + "k"]), W[p + "k.conv"])
    v = k.view(n, G, d)
    q = rotate(rms(q, W[p + "q.norm"], eps).view(n, H, d), pos, f, mag)
    k = rotate(rms(k, W[p + "k.norm"], eps).view(n, G, d), pos, f, mag)
    outs = [softmax_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], W[p + "sink"][i]) for i in range(H)]
    return lin(torch.cat(outs, -1), W[p + "o"])


def lru_gates(u, W, p, blocks):
    """u [n, width] -> (a, i): the decay and the input gate of every channel."""
    n, width = u.shape
    ub = u.view(n, blocks, width // blocks)
    gate = lambda name: sigmoid(torch.einsum("nbk,bjk->nbj", ub, W[p + name].to(F64)) + W[p + name + ".b"].to(F64)).reshape(n, width)
    return torch.exp(-8.0 * gate("ra") * softplus(W[p + "lam"].to(F64))), gate("ri")


def lru_scan(a, x):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) x_t, S zero at the start."""
    S, out = torch.zeros(x.shape[1], dtype=F64), torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = a[t] * S + torch.sqrt(1.0 - a[t] ** 2) * x[t]
        out[t] = S
    return out


def lru_block(h, W, p, m, eps):
    y = gelu_tanh(lin(h, W[p + "y"]) + W[p + "y.b"].to(F64))
    u = causal_conv(lin(h, W[p + "x"]) + W[p + "x.b"].to(F64), W[p + "conv"], W[p + "conv.b"])
    a, i = lru_gates(u, W, p, m["blocks"])
    return lin(lru_scan(a, i * u) * y, W[p + "o"])


def parallel_mixer(h, W, p, m, eps):
    left = conv_attention(h, W, p + "left.", m["left"], eps)
    right = lru_block(h, W, p + "right.", m["right"], eps)
    return 0.5 * (rms(left, W[p + "left.out"], eps) + rms(right, W[p + "right.out"], eps))


MIXERS = {"gla": gla_mixer, "latent_attention": latent_mixer, "parallel": parallel_mixer}


# ------------------------------------------------------------------ feed-forward
def clamped_ff(h, W, p, limit):
    g = lin(h, W[p + "gate"]).clamp(max=limit)
    u = lin(h, W[p + "up"]).clamp(-limit, limit)
    return lin(g * sigmoid(1.702 * g) * (u + 1.0), W[p + "down"])


def expert_ff(h, W, p):
    return lin(silu(lin(h, W[p + "gate"])) * lin(h, W[p + "up"]), W[p + "down"])


def route(h, W, p, top):
    """(experts, weights) [n, top]: the largest logits, softmax over the chosen ones."""
    z = lin(h, W[p + "router"]) + W[p + "router.b"].to(F64)
    best, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(best, -1)


def moe_ff(h, W, p, ml):
    idx, w = route(h, W, p, ml["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t].tolist(), w[t]):
            out[t] += we * expert_ff(h[t:t + 1], W, f"{p}e{e}.")[0]
    return out


# ------------------------------------------------------------------ the model
def run_order(cfg):
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(cfg, W, tokens, layers_out=None):
    """Logits [n, vocab] (float64) of one sequence; layers_out (a list) receives the sum of the streams after each layer run."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    emb = W["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)]
    x = emb[None].repeat(cfg["streams"], 1, 1)
    for i in run_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        subs = [("1", lambda h: MIXERS[L["type"]](h, W, p + "mix.", L["mixer"], eps))]
        if L.get("mlp") is not None:
            ml = L["mlp"]
            subs.append(("2", lambda h: clamped_ff(h, W, p + "mlp.", ml["limit"]) if ml["kind"] == "dense" else moe_ff(h, W, p + "mlp.", ml)))
        for q, f in subs:
            hc = p + "hc" + q + "."
            y = f(dyt(hyper_read(x, W[hc + "in"]), W, p + "norm" + q))
            x = hyper_write(x, W[hc + "mix"], W[hc + "out"], y, m)
        if layers_out is not None:
            layers_out.append(x.sum(0))
    return lin(dyt(x.sum(0), W, "final.norm"), W["head"])


# ------------------------------------------------------------------ configurations and random checkpoints for tests
def gla(heads, dim, vdim, tau=8.0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale=None, base=10000.0, scaling=(4.0, 64, 8.0, 1.0)):
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                  "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": rot}}


def parallel(heads, kv_heads, dim, width, blocks, conv=4, rconv=4, rot_dims=None, base=10000.0, scale=None):
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv, "scale": scale if scale is not None else dim ** -0.5,
                 "rot": {"dims": dim if rot_dims is None else rot_dims, "base": base}},
        "right": {"width": width, "blocks": blocks, "conv": rconv}}}


def dense(ff, limit=2.0):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def make_config(width, vocab, layers, loop=None, streams=3, m=0.8, eps=1e-5):
    cfg = {"architecture": "Mutirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "residual_mult": m,
           "layers": layers}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def make_checkpoint(cfg, seed=0, dtype=torch.bfloat16, rank=12):
    """Random weights rounded to `dtype` (so a 16-bit engine holds exactly the same numbers), returned as float32; `rank` is
    the width of the decay's inner projection."""
    g = torch.Generator().manual_seed(seed)
    D, V, s = cfg["width"], cfg["vocab"], cfg["streams"]

    def mat(rows, cols, gain=1.0):
        return (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(dtype).float()

    def vec(n, mean=0.0, dev=0.2):
        return (mean + dev * torch.randn(n, generator=g)).to(dtype).float()

    def norm(name, alpha):
        return {name: vec(D, 1.0), name + ".b": vec(D, 0.0, 0.1), name + ".alpha": torch.tensor(alpha).to(dtype).float()}

    def hyper(p):
        mix = torch.eye(s) * 0.6 + 0.4 / s + 0.1 * torch.randn(s, s, generator=g)
        return {p + "in": vec(s, 1.0 / s, 0.15), p + "out": vec(s, 0.8, 0.3), p + "mix": mix.to(dtype).float()}

    W = {"embed": torch.randn(V, D, generator=g).to(dtype).float(), "head": mat(V, D, 1.5)}
    W.update(norm("final.norm", 0.3))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        x = p + "mix."
        W.update(norm(p + "norm1", 0.7))
        W.update(hyper(p + "hc1."))
        if L["type"] == "gla":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            W.update({x + "q": mat(H * d, D, 1.5), x + "k": mat(H * d, D, 1.5), x + "v": mat(H * e, D, 1.5), x + "g": mat(H * e, D, 1.5),
                      x + "o": mat(D, H * e, 1.5), x + "norm": vec(e, 1.0), x + "a1": mat(rank, D), x + "a2": mat(H * d, rank, 2.0),
                      x + "a2.b": vec(H * d, 0.0, 1.5)})
        elif L["type"] == "latent_attention":
            H, d, r, e, qr, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            W.update({x + "dq": mat(qr, D), x + "dq.norm": vec(qr, 1.0), x + "uq": mat(H * (d + r), qr, 1.5), x + "dkv": mat(kr + r, D, 1.5),
                      x + "dkv.norm": vec(kr, 1.0), x + "uk": mat(H * d, kr, 1.5), x + "uv": mat(H * e, kr, 1.5), x + "g": mat(H, D, 1.5),
                      x + "o": mat(D, H * e, 1.5)})
        else:
            a, b = m["left"], m["right"]
            nq, nk, w, bs = a["heads"] * a["dim"], a["kv_heads"] * a["dim"], b["width"], b["width"] // b["blocks"]
            l, r = x + "left.", x + "right."
            W.update({l + "q": mat(nq, D), l + "k": mat(nk, D), l + "q.norm": vec(nq, 1.0), l + "k.norm": vec(nk, 1.0),
                      l + "q.conv": mat(nq, a["conv"], 1.5), l + "k.conv": mat(nk, a["conv"], 1.5), l + "sink": vec(a["heads"], 0.5, 1.0),
                      l + "o": mat(D, nq, 1.5), l + "out": vec(D, 1.0),
                      r + "y": mat(w, D), r + "y.b": vec(w), r + "x": mat(w, D), r + "x.b": vec(w, 0.0, 0.4), r + "conv": mat(w, b["conv"], 1.5),
                      r + "conv.b": vec(w), r + "ra": mat(w, bs).view(b["blocks"], bs, bs), r + "ra.b": vec(w, 0.0, 0.5).view(b["blocks"], bs),
                      r + "ri": mat(w, bs).view(b["blocks"], bs, bs), r + "ri.b": vec(w, 0.0, 0.5).view(b["blocks"], bs),
                      r + "lam": vec(w, -3.0, 1.5), r + "o": mat(D, w, 1.5), r + "out": vec(D, 1.0)})
        ml = L.get("mlp")
        if ml is None:
            continue
        f = p + "mlp."
        W.update(norm(p + "norm2", 0.7))
        W.update(hyper(p + "hc2."))
        if ml["kind"] == "dense":
            W.update({f + "gate": mat(ml["ff"], D, 1.5), f + "up": mat(ml["ff"], D, 1.5), f + "down": mat(D, ml["ff"])})
        else:
            E, ff = ml["router"]["experts"], ml["expert"]["ff"]
            W.update({f + "router": mat(E, D, 2.0), f + "router.b": vec(E, 0.0, 0.5)})
            for e in range(E):
                W.update({f"{f}e{e}.gate": mat(ff, D, 1.5), f"{f}e{e}.up": mat(ff, D, 1.5), f"{f}e{e}.down": mat(D, ff)})
    return W
