"""Plain float64 restatement of the Ranesun design: one function per mechanism, whole sequences, no caches, no
batching, no code shared with the served path.  Slow on purpose: loops over tokens and heads where that is clearest.

Shapes: a sequence is [n, ...]; weights are [out, in] and applied as x @ W.T.  Positions are 0 .. n-1.
"""
import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------ elementary pieces
def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def lin(x, w):
    return x @ w.to(F64).T


def layer_norm(x, w, b, eps):
    mean = x.mean(-1, keepdim=True)
    var = ((x - mean) ** 2).mean(-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * w.to(F64) + b.to(F64)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ------------------------------------------------------------------ rotary positions (halves layout)
def frequencies(dims, base):
    i = torch.arange(dims // 2, dtype=F64)
    return float(base) ** (-2.0 * i / dims)


def rotate(x, positions, f):
    """x [n, ..., >= 2 len(f)]: column i of row t is paired with column i + len(f); the others pass."""
    out = x.clone()
    m = f.shape[0]
    for t, p in enumerate(positions):
        c, s = torch.cos(float(p) * f), torch.sin(float(p) * f)
        u, v = x[t, ..., :m], x[t, ..., m:2 * m]
        out[t, ..., :m] = u * c - v * s
        out[t, ..., m:2 * m] = v * c + u * s
    return out


# ------------------------------------------------------------------ retention
def retention_scan(q, k, v, decay):
    """q, k [n, H, d], v [n, H, e]: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, S zero at the start."""
    n, H, d = q.shape
    o = torch.zeros(n, H, v.shape[-1], dtype=F64)
    for h in range(H):
        S = torch.zeros(d, v.shape[-1], dtype=F64)
        for t in range(n):
            S = float(decay[h]) * S + torch.outer(k[t, h], v[t, h])
            o[t, h] = S.T @ q[t, h]
    return o


def retention_operands(h, W, p, m):
    n, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = list(range(n))
    q, k = lin(h, W[p + "q"]).view(n, H, d), lin(h, W[p + "k"]).view(n, H, d)
    if m.get("rot"):
        f = frequencies(m["rot"]["dims"], m["rot"]["base"])
        q, k = rotate(q, pos, f), rotate(k, pos, f)
    return q, k / math.sqrt(d), lin(h, W[p + "v"]).view(n, H, e)


def retention_mixer(h, W, p, m, eps):
    q, k, v = retention_operands(h, W, p, m)
    o = unit_rms(retention_scan(q, k, v, m["decay"]), eps).reshape(h.shape[0], -1)
    return lin(o * silu(lin(h, W[p + "g"])), W[p + "o"])


# ------------------------------------------------------------------ attention
def query_temperature(p, coef, every):
    return 1.0 + coef * math.log((p + 1) // every + 1)


def cap(s, softcap):
    return softcap * torch.tanh(s / softcap) if softcap else s


def tied_attention(q, k, scale, softcap, temp, sink, first=0):
    """q [n - first, d] (positions first ..), k [n, d] of ONE head; the values are the keys.  temp = (coef, every)."""
    n = k.shape[0]
    out = torch.zeros(n - first, k.shape[1], dtype=F64)
    for i in range(first, n):
        qi = q[i - first] * query_temperature(i, *temp)
        s = cap((k[:i + 1] @ qi) * scale, softcap)
        top = max(float(s.max()), float(sink))
        e = torch.exp(s - top)
        out[i - first] = (e @ k[:i + 1]) / (e.sum() + math.exp(float(sink) - top))
    return out


def attention_mixer(h, W, p, m, eps):
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = lin(h, W[p + "q"]).view(n, H, d), lin(h, W[p + "k"]).view(n, G, d)
    t = m.get("q_temp")
    temp = (t["coef"], t["every"]) if t else (0.0, 1)
    outs = [tied_attention(q[:, hd], k[:, hd // (H // G)], m["scale"], m.get("softcap"), temp, W[p + "sink"][hd])
            for hd in range(H)]
    return lin(torch.cat(outs, -1), W[p + "o"])


MIXERS = {"retention": retention_mixer, "attention": attention_mixer}


# ------------------------------------------------------------------ feed-forward
def dense_ff(h, W, p):
    return lin(gelu_tanh(lin(h, W[p + "gate"])) * lin(h, W[p + "up"]), W[p + "down"])


def expert_ff(h, W, p):
    return lin(torch.relu(lin(h, W[p + "up"])) ** 2, W[p + "down"])


def table_moe_ff(h, W, p, tokens):
    table = W[p + "table"]
    out = torch.zeros(h.shape[0], h.shape[1], dtype=F64)
    for t, tok in enumerate(tokens):
        experts = table[int(tok)].tolist()
        for e in experts:
            out[t] += expert_ff(h[t:t + 1], W, f"{p}e{e}.")[0] / len(experts)
    return out


# ------------------------------------------------------------------ the model
def run_order(cfg):
    """(layer, number of the pass that it opens or None) for every layer run, in order."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        for i in range(lp["start"], lp["stop"]):
            order.append((i, t if i == lp["start"] else None))
    return order + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg, W, tokens, layers_out=None):
    """Logits [n, vocab] (float64) of one sequence; layers_out (a list) receives the residual stream after each layer run."""
    eps = cfg["norm"]["eps"]
    emb = W["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)]
    x = emb.clone()
    for i, opens in run_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        if opens is not None:
            if opens > 0:
                x = x + emb
            x = x + W["loop.step"].to(F64)[opens]
        x = x + MIXERS[L["type"]](layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps), W, p + "mix.", L["mixer"], eps)
        if L.get("mlp") is not None:
            h = layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps)
            x = x + (dense_ff(h, W, p + "mlp.") if L["mlp"]["kind"] == "dense" else table_moe_ff(h, W, p + "mlp.", tokens))
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(layer_norm(x, W["final.norm"], W["final.norm.b"], eps), W["embed"]) * cfg["logit_scale"]


# ------------------------------------------------------------------ configurations and random checkpoints for tests
def retention(heads, dim, vdim, decay=None, rot_dims=None, base=10000.0):
    if decay is None:
        decay = [1.0 - 2.0 ** (-2.0 - 5.0 * h / max(heads - 1, 1)) for h in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                           "rot": {"dims": dim if rot_dims is None else rot_dims, "base": base}}}


def attention(heads, kv_heads, dim, softcap=15.0, coef=0.4, every=32, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
                                           "scale": scale if scale is not None else 1.0 / math.sqrt(dim), "softcap": softcap,
                                           "q_temp": {"coef": coef, "every": every}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def make_config(width, vocab, layers, loop=None, eps=1e-5, logit_scale=1.0):
    cfg = {"architecture": "Ranesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
           "layers": layers}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def make_checkpoint(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights rounded to `dtype` (so a 16-bit engine holds exactly the same numbers), returned as float32;
    the expert tables are int32."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(rows, cols, gain=1.0):
        return (torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)).to(dtype).float()

    def vec(n, mean=0.0, dev=0.2):
        return (mean + dev * torch.randn(n, generator=g)).to(dtype).float()

    W = {"embed": torch.randn(V, D, generator=g).to(dtype).float(), "final.norm": vec(D, 1.0), "final.norm.b": vec(D)}
    if cfg.get("loop"):
        W["loop.step"] = (0.5 * torch.randn(cfg["loop"]["times"], D, generator=g)).to(dtype).float()
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        W.update({p + "norm1": vec(D, 1.0), p + "norm1.b": vec(D, 0.1)})
        if L["type"] == "retention":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            W.update({p + "mix.q": mat(H * d, D, 1.5), p + "mix.k": mat(H * d, D, 1.5), p + "mix.v": mat(H * e, D, 1.5),
                      p + "mix.g": mat(H * e, D, 1.5), p + "mix.o": mat(D, H * e, 1.5)})
        else:
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            W.update({p + "mix.q": mat(H * d, D, 2.0), p + "mix.k": mat(G * d, D, 2.0), p + "mix.sink": vec(H, 0.5, 1.0),
                      p + "mix.o": mat(D, H * d, 1.5)})
        ml = L.get("mlp")
        if ml is None:
            continue
        f = p + "mlp."
        W.update({p + "norm2": vec(D, 1.0), p + "norm2.b": vec(D, 0.1)})
        if ml["kind"] == "dense":
            W.update({f + "gate": mat(ml["ff"], D, 1.5), f + "up": mat(ml["ff"], D, 1.5), f + "down": mat(D, ml["ff"])})
        else:
            E, top, ff = ml["router"]["experts"], ml["router"]["top"], ml["expert"]["ff"]
            for e in range(E):
                W.update({f"{f}e{e}.up": mat(ff, D, 1.5), f"{f}e{e}.down": mat(D, ff)})
            W[f + "table"] = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(V)]).to(torch.int32)
    return W
