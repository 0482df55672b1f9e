"""Mutirax: a decoder-only language model whose residual stream is several copies joined by hyper-connections, normed by
dynamic tanh, whose mixers are gated linear attention, latent attention with a gate per head, or a pair of parallel branches
(attention over convolved keys that are also the values, beside a gated linear recurrent unit), with dense or
mixture-of-experts feed-forwards and a block of layers that runs several times with the same weights.

Design (every size and every constant that can differ between checkpoints comes from config.json):

  x_s[t]     = embed[token_t] for every stream s = 1 .. streams              fp32 residual streams
  schedule   : layers 0 .. start-1 once, layers start .. stop-1 `times` times in a row (same weights, but every pass has a
               cache / state of its own), then stop .. n-1 once.  A layer run is one (layer, pass) pair.
  sublayer   : u = sum_s in[s] x_s ;  y = F(N(u)) ;  x_t <- sum_s mix[s, t] x_s + residual_mult out[t] y   (all t at once);
               F is the mixer, then the feed-forward (which may be absent), each with in / mix / out and a norm of its own
  N(u)       = tanh(alpha u) * w + b
  gla        : q = Wq h dim^(-1/2), k = Wk h, v = Wv h; a = sigmoid(Wa2 Wa1 h + b)^(1/tau) per key channel;
               S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t;  Wo (concat_h(RMS(o) w) * silu(Wg h))
  latent     : `latent.py`: rotary pairs (i, i + rot_dim/2) with YaRN-scaled frequencies, no sink, gate sigmoid(Wg h) per head
  parallel   : left:  q, k = conv(Wq h), conv(Wk h) (causal, per channel); v = k; q, k <- RMS over the whole projection,
                      rotary on the first rot.dims columns of every head (pairs (i, i + dims/2)); causal softmax with a sink; Wo
               right: y = gelu_tanh(Wy h + b), u = conv(Wx h + b) + b'; r, i = sigmoid of block-diagonal products of u;
                      log a = -8 r softplus(lam), S_t = a S_(t-1) + sqrt(1 - a^2) i u;  Wo (S * y)
               half the sum of RMS(left) w_left and RMS(right) w_right
  ff dense   : g = min(Wgate h, limit), u = clamp(Wup h, -limit, limit);  Wdown (g sigmoid(1.702 g) (u + 1))
  ff moe     : z = Wrouter h + b; the `top` largest, weighted by the softmax over them; expert: Wdown (silu(Wgate h) * Wup h)
  output     : logits = Whead N_final(sum_s x_s)

fp32: the residual streams and their mixing, every norm, positions and angles, attention scores and weights, the router, and
in both recurrences everything but the projections and the convolution: decays, gates, state, unit norms.  Model dtype (fp32
accumulation): projections, convolved inputs, caches, the feed-forward.

One row kernel does everything between two sublayers (hyper.cu): it takes the sublayer's output in whatever form it was left
(dense rows, expert rows with their places and weights, the two branches of a parallel mixer before their norms), mixes the
streams and writes the next sublayer's operand.  The streams are not written before the first sublayer's output exists.

The engine owns the repacked weights (one fused projection per mixer), one paged latent pool per run of a latent layer, one
paged key / value pool pair per run of a parallel layer and, through the scheduler's slot table, the per-sequence state of every
run: [heads, dim, vdim] of gated linear attention, [width] of the recurrent unit and the last projected inputs of both branches'
convolutions.  The step function, page pool, scheduler and sampling are the framework's (`ragged_engine.RaggedEngine`,
`scheduler.SlotKV` / `SlotState` / `RaggedBatcher`).
"""
from __future__ import annotations

import warnings
from dataclasses import dataclass, field
from typing import Dict, List, Mapping, Optional

import torch

from . import _cabi as cabi
from ._cabi import ptr
from .latent import LatentAttentionMixin, latent_cfg, pack_latent
from .ragged_engine import LoopCfg, RaggedEngine, RotaryCfg, Run, StepInputs, _stack_rows, layer_runs, loop_cfg, rotary_pairs
from .registry import register

GLU_ALPHA = 1.702                 # the sigmoid's slope in the dense feed-forward: fixed by the design
LRU_C = 8.0                       # the factor in the recurrent unit's log decay: fixed by the design
PAIR_SCALE = 0.5                  # a parallel mixer is the mean of its branches


@dataclass
class GlaCfg:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass
class ConvAttnCfg:
    heads: int
    kv_heads: int
    dim: int                      # of queries, keys and (the keys before norm and rotation) values
    scale: float
    taps: int
    rot: Optional[RotaryCfg]


@dataclass
class LruCfg:
    width: int
    blocks: int
    taps: int


@dataclass
class ParallelCfg:
    left: ConvAttnCfg
    right: LruCfg


@dataclass
class MlpCfg:
    kind: str                     # "dense" | "moe"
    ff: int                       # dense width / expert width
    limit: float = 0.0
    experts: int = 0
    top: int = 0


@dataclass
class LayerCfg:
    kind: str                     # "gla" | "latent_attention" | "parallel"
    mixer: object
    mlp: Optional[MlpCfg]


def _conv_attn_cfg(i: int, m: Mapping) -> ConvAttnCfg:
    heads, dim, rot = int(m["heads"]), int(m["dim"]), m.get("rot")
    a = ConvAttnCfg(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=dim, scale=float(m["scale"]), taps=int(m["conv"]),
                    rot=RotaryCfg(int(rot["dims"]), float(rot["base"])) if rot and int(rot["dims"]) else None)
    if a.heads % a.kv_heads or a.taps < 1:
        raise ValueError(f"layer {i}: {a.heads} heads over {a.kv_heads} key heads, {a.taps} taps")
    if int(m.get("vdim", dim)) != dim:
        raise ValueError(f"layer {i}: the values are the keys, so vdim {m['vdim']} must be dim {dim}")
    if a.rot and (a.rot.dims % 2 or a.rot.dims > dim or rot.get("scaling")):
        raise ValueError(f"layer {i}: {a.rot.dims} rotated columns of {dim}, frequency scaling {rot.get('scaling')}")
    return a


def _mixer_cfg(i: int, kind: str, m: Mapping):
    if kind == "gla":
        return GlaCfg(int(m["heads"]), int(m["dim"]), int(m.get("vdim", m["dim"])), float(m["tau"]))
    if kind == "latent_attention":
        return latent_cfg(i, m, halves=True)
    if kind == "parallel":
        r = m["right"]
        right = LruCfg(int(r["width"]), int(r["blocks"]), int(r["conv"]))
        if right.blocks < 1 or right.width % right.blocks or right.taps < 1:
            raise ValueError(f"layer {i}: {right.width} channels in {right.blocks} blocks, {right.taps} taps")
        return ParallelCfg(_conv_attn_cfg(i, m["left"]), right)
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def _mlp_cfg(i: int, ml: Optional[Mapping]) -> Optional[MlpCfg]:
    if ml is None:
        return None
    if ml.get("kind") == "dense":
        return MlpCfg("dense", int(ml["ff"]), float(ml["limit"]))
    if ml.get("kind") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {ml.get('kind')!r}")
    c = MlpCfg("moe", int(ml["expert"]["ff"]), 0.0, int(ml["router"]["experts"]), int(ml["router"]["top"]))
    if not 1 <= c.top <= c.experts:
        raise ValueError(f"layer {i}: top {c.top} of {c.experts} experts")
    return c


@dataclass
class MutiraxConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    residual_mult: float
    layers: List[LayerCfg] = field(default_factory=list)
    loop: Optional[LoopCfg] = None

    def runs(self) -> List[Run]:
        """The layer runs of one forward pass, in order."""
        return layer_runs(len(self.layers), self.loop)

    @staticmethod
    def from_dict(cfg: Mapping) -> "MutiraxConfig":
        layers = [LayerCfg(L.get("type"), _mixer_cfg(i, L.get("type"), L["mixer"]), _mlp_cfg(i, L.get("mlp")))
                  for i, L in enumerate(cfg["layers"])]
        c = MutiraxConfig(vocab=int(cfg["vocab"]), width=int(cfg["width"]), eps=float((cfg.get("norm") or {})["eps"]),
                          streams=int(cfg["streams"]), residual_mult=float(cfg["residual_mult"]), layers=layers,
                          loop=loop_cfg(cfg.get("loop"), len(layers)))
        if c.streams < 1:
            raise ValueError(f"{c.streams} residual streams")
        return c


@register("Mutirax")
class MutiraxEngine(LatentAttentionMixin, RaggedEngine):
    """Weights + paged pools + recurrent state shapes + the launch sequence of one step over a ragged token batch."""

    def __init__(self, config, weights: Mapping[str, torch.Tensor], *, device="cuda", dtype=torch.bfloat16,
                 page_size: int = 64, kv_pool_tokens: int = 65536, gemm_impl: int = 0, strict: bool = False):
        self.cfg = config if isinstance(config, MutiraxConfig) else MutiraxConfig.from_dict(config)
        self.strict = bool(strict)      # True: tensors the config does not call for raise instead of being reported
        self._init_common(device=device, dtype=dtype, page_size=page_size, gemm_impl=gemm_impl)
        self.runs = self.cfg.runs()
        self.needs_segments = any(lc.kind != "latent_attention" for lc in self.cfg.layers)
        self.lru_impl = 0               # recurrent unit: 0 picks, 1 token by token, 2 chunked
        self.route_gemm_min = 256       # tokens from which the router's logits are a GEMM of their own
        self._repack(weights)
        L_ = cabi.lib()
        for w, lc in zip(self.layers, self.cfg.layers):     # prompt portions of layers whose sizes the tensor-core kernel takes
            w["attn_tc"] = False
            if lc.kind == "latent_attention":
                w["attn_tc"] = self._latent_tc_ok(lc.mixer)
            elif lc.kind == "parallel":
                a = lc.mixer.left
                w["attn_tc"] = bool(L_.pg_attention_ragged_tc_ok8(a.dim, a.dim, self.page_size, a.heads * a.dim, a.heads * a.dim, 8,
                                                                  self.dt))
        self._attn_tc_any = any(w["attn_tc"] for w in self.layers)
        self._init_runtime(kv_pool_tokens)
        # pools per RUN of a layer: a layer that runs twice keeps two caches
        self.c_pools: Dict[int, torch.Tensor] = {}
        self.k_pools: Dict[int, torch.Tensor] = {}
        self.v_pools: Dict[int, torch.Tensor] = {}
        for ri, r in enumerate(self.runs):
            lc = self.cfg.layers[r.layer]
            pool = lambda cols: torch.zeros((self.num_pages, self.page_size, cols), dtype=dtype, device=self.device)
            if lc.kind == "latent_attention":
                self.c_pools[ri] = pool(self.layers[r.layer]["ld_pool"])
            elif lc.kind == "parallel":
                cols = lc.mixer.left.kv_heads * lc.mixer.left.dim
                self.k_pools[ri], self.v_pools[ri] = pool(cols), pool(cols)

    # ------------------------------------------------------------------ weights
    def _repack(self, weights: Mapping[str, torch.Tensor]) -> None:
        c, D, S, f32 = self.cfg, self.cfg.width, self.cfg.streams, torch.float32
        used = set()

        def W(name, shape=None, dtype=None):
            if name not in weights:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            used.add(name)
            t = weights[name]
            if shape is not None and tuple(t.shape) != tuple(shape):
                raise ValueError(f"tensor {name}: shape {tuple(t.shape)}, the config wants {tuple(shape)}")
            return t.to(device=self.device, dtype=dtype or self.dtype).contiguous()

        def reader(name, w_in):         # what the row kernel needs to write a sublayer's operand: stream weights and alpha, w, b
            alpha = W(name + ".alpha", (), f32).reshape(1)
            return torch.cat([w_in, alpha]).contiguous(), W(name, (D,)), W(name + ".b", (D,))

        def writer(p):                  # ... and to take its output into the streams: mix, residual_mult * out
            return W(p + "mix", (S, S), f32), (W(p + "out", (S,), f32) * c.residual_mult).contiguous()

        self.emb, self.head = W("embed", (c.vocab, D)), W("head", (c.vocab, D))
        self.final_read = reader("final.norm", torch.ones(S, dtype=f32, device=self.device))
        self.layers: List[dict] = []
        for i, L in enumerate(c.layers):
            p, m, a = f"l{i}.", f"l{i}.mix.", L.mixer
            w = dict(read1=reader(p + "norm1", W(p + "hc1.in", (S,), f32)), write1=writer(p + "hc1."))
            if L.kind == "gla":
                nk, nv = a.heads * a.dim, a.heads * a.vdim
                a1 = W(m + "a1")
                if a1.dim() != 2 or a1.shape[1] != D:
                    raise ValueError(f"tensor {m}a1: shape {tuple(a1.shape)}, the config wants (.., {D})")
                w["rank"] = int(a1.shape[0])
                w["proj"], w["at"] = _stack_rows([("q", W(m + "q", (nk, D))), ("k", W(m + "k", (nk, D))), ("v", W(m + "v", (nv, D))),
                                                  ("g", W(m + "g", (nv, D))), ("a", a1)], self.device, self.dtype)
                w.update(a2=W(m + "a2", (nk, w["rank"])), a2_b=W(m + "a2.b", (nk,)), o=W(m + "o", (D, nv)),
                         onorm=W(m + "norm", (a.vdim,)).repeat(a.heads).contiguous())
            elif L.kind == "latent_attention":
                w.update(pack_latent(W, m, a, D, self.device, self.dtype, gated=False, sink=False, head_gate=True))
            else:
                self._repack_parallel(W, m, a, w)
            ml = L.mlp
            if ml is not None:
                f = p + "mlp."
                w.update(read2=reader(p + "norm2", W(p + "hc2.in", (S,), f32)), write2=writer(p + "hc2."))
                if ml.kind == "dense":
                    w.update(gu=torch.cat([W(f + "gate", (ml.ff, D)), W(f + "up", (ml.ff, D))], 0).contiguous(),
                             down=W(f + "down", (D, ml.ff)))
                else:
                    w.update(router=W(f + "router", (ml.experts, D)), router_b=W(f + "router.b", (ml.experts,)),
                             gu=torch.stack([torch.cat([W(f"{f}e{e}.gate", (ml.ff, D)), W(f"{f}e{e}.up", (ml.ff, D))], 0)
                                             for e in range(ml.experts)], 0).contiguous(),
                             dn=torch.stack([W(f"{f}e{e}.down", (D, ml.ff)) for e in range(ml.experts)], 0).contiguous())
            self.layers.append(w)
        extra = sorted(set(weights) - used)
        if extra:
            text = f"checkpoint holds {len(extra)} tensor(s) the config does not call for: {extra[:8]}"
            if self.strict:
                raise ValueError(text)
            warnings.warn(text + " (not used)")

    def _repack_parallel(self, W, m: str, a: ParallelCfg, w: dict) -> None:
        D, f32, lf, rt = self.cfg.width, torch.float32, a.left, a.right
        l, r = m + "left.", m + "right."
        nq, nk, bs = lf.heads * lf.dim, lf.kv_heads * lf.dim, rt.width // rt.blocks
        # the convolved columns first and together: q | k | x, so that one state holds the earlier inputs of both branches
        w["proj"], w["at"] = _stack_rows([("q", W(l + "q", (nq, D))), ("k", W(l + "k", (nk, D))), ("x", W(r + "x", (rt.width, D))),
                                          ("y", W(r + "y", (rt.width, D)))], self.device, self.dtype)
        at = w["at"]
        conv = torch.zeros((lf.taps, at["k"] + nk), dtype=self.dtype, device=self.device)   # [taps][columns], the current token last
        conv[:, :nq] = W(l + "q.conv", (nq, lf.taps)).T
        conv[:, at["k"]:] = W(l + "k.conv", (nk, lf.taps)).T
        w.update(conv=conv, q_norm=W(l + "q.norm", (nq,)), k_norm=W(l + "k.norm", (nk,)), sink=W(l + "sink", (lf.heads,), f32),
                 freq=rotary_pairs(lf.rot).to(self.device) if lf.rot else None, o=W(l + "o", (D, nq)), left_out=W(l + "out", (D,)))
        gates = torch.cat([W(r + "ra", (rt.blocks, bs, bs)), W(r + "ri", (rt.blocks, bs, bs))], 1).contiguous()
        w.update(x_b=W(r + "x.b", (rt.width,)), y_b=W(r + "y.b", (rt.width,)), gates=gates,
                 r_conv=W(r + "conv", (rt.width, rt.taps)).T.contiguous(), r_conv_b=W(r + "conv.b", (rt.width,)),
                 ra_b=W(r + "ra.b", (rt.blocks, bs)).reshape(-1), ri_b=W(r + "ri.b", (rt.blocks, bs)).reshape(-1),
                 lam=W(r + "lam", (rt.width,), f32), r_o=W(r + "o", (D, rt.width)), right_out=W(r + "out", (D,)),
                 conv_len=max(lf.taps, rt.taps) - 1, conv_cols=at["x"] + rt.width)

    # ------------------------------------------------------------------ per-sequence state
    def new_slot_state(self, slots: int):
        from .scheduler import SlotState
        shapes = {}
        for ri, r in enumerate(self.runs):
            L, w = self.cfg.layers[r.layer], self.layers[r.layer]
            if L.kind == "gla":
                shapes[("gla", ri)] = (L.mixer.heads, L.mixer.dim, L.mixer.vdim)
            elif L.kind == "parallel":
                shapes[("lru", ri)] = (L.mixer.right.width,)
                if w["conv_len"]:
                    shapes[("conv", ri)] = (w["conv_len"], w["conv_cols"])
        return SlotState(slots, shapes, self.device) if shapes else None

    # ------------------------------------------------------------------ one step
    def _connect(self, inp: StepInputs, x, y, write, out, read, *, emb: bool, rows_idx=None) -> None:
        """The sublayer output y (None, dense rows, {"experts": ..} or {"pair": ..}) into the streams with `write`, then the
        operand that `read` asks for into `out` (None: no operand).  emb: the old streams are still the embedding rows."""
        rows = x.shape[0] if rows_idx is None else rows_idx.shape[0]
        rows_y, pos, wts, top, y2, n1, n2 = y, None, None, 1, None, None, None
        if isinstance(y, dict):
            if "experts" in y:
                rows_y, pos, wts, top = y["experts"]
            else:
                rows_y, y2, n1, n2 = y["pair"]
        mix, w_out = write if write is not None else (None, None)
        w_in, w, b = read if read is not None else (None, None, None)
        with self._tm("connect_pair" if y2 is not None else ("connect_experts" if pos is not None else "connect")):
            cabi.check(cabi.lib().pg_hyper_connect(
                ptr(out), 0 if out is None else out.stride(0), ptr(x), self.cfg.streams, ptr(rows_y),
                0 if rows_y is None else rows_y.stride(0), ptr(pos), ptr(wts), top, ptr(y2), 0 if y2 is None else y2.stride(0),
                ptr(n1), ptr(n2), self.cfg.eps, PAIR_SCALE, ptr(inp.ids) if emb else None, ptr(self.emb), self.cfg.vocab, ptr(mix),
                ptr(w_out), ptr(w_in), ptr(w), ptr(b), ptr(rows_idx), rows, self.cfg.width, ptr(self.err_flag), self.dt,
                cabi.stream()), "hyper_connect")

    def _gla(self, kv, inp: StepInputs, ri: int, a: GlaCfg, w: dict, h) -> torch.Tensor:
        L, st, tm, T, at = cabi.lib(), cabi.stream(), self._tm, inp.T, w["at"]
        with tm("proj"):
            proj = self._linear(h, w["proj"])
        nv = a.heads * a.vdim
        rec = self._new(int(L.pg_gla_record_floats(T, a.heads, a.dim, a.vdim)), dtype=torch.float32)
        with tm("gla_prep"):
            cabi.check(L.pg_gla_prep(ptr(rec), ptr(proj), proj.stride(0), at["q"], at["k"], at["v"], at["a"], w["rank"], ptr(w["a2"]),
                                     ptr(w["a2_b"]), a.dim ** -0.5, 1.0 / a.tau, T, a.heads, a.dim, a.vdim, self.dt, st), "gla_prep")
        o = self._new(T, nv, dtype=torch.float32)
        with tm("gla"):
            cabi.check(L.pg_gla_attention(ptr(o), ptr(kv.state.layers[("gla", ri)]), ptr(rec), ptr(inp.segs), inp.n_segs, a.heads,
                                          a.dim, a.vdim, st), "gla_attention")
        g = self._new(T, nv)
        with tm("headnorm_gate"):
            cabi.check(L.pg_headnorm_gate_ex(ptr(g), nv, ptr(o), ptr(w["onorm"]), ptr(proj[:, at["g"]:]), proj.stride(0), 1, T,
                                             a.heads, a.vdim, self.cfg.eps, 1.0, self.dt, st), "headnorm_gate")
        with tm("o"):
            return self._linear(g, w["o"])

    def _conv_attention(self, kv, inp: StepInputs, ri: int, a: ConvAttnCfg, w: dict, proj, conv_state) -> torch.Tensor:
        L, st, tm, T, at = cabi.lib(), cabi.stream(), self._tm, inp.T, w["at"]
        q = self._new(T, a.heads * a.dim)
        kp, vp = self.k_pools[ri], self.v_pools[ri]
        with tm("conv_qk_append"):
            cabi.check(L.pg_conv_qk_append(ptr(q), ptr(proj), proj.stride(0), at["q"], a.heads, at["k"], a.kv_heads, a.dim, ptr(w["conv"]),
                                           a.taps, ptr(conv_state), w["conv_len"], w["conv_cols"], ptr(w["q_norm"]), ptr(w["k_norm"]),
                                           self.cfg.eps, ptr(w["freq"]), a.rot.dims if a.rot else 0, ptr(kp), ptr(vp),
                                           ptr(kv.page_table), kv.max_pages, self.page_size, ptr(inp.slot), ptr(inp.pos), T,
                                           self.dt, st), "conv_qk_append")
        att = self._new(T, a.heads * a.dim)
        with tm("attention"):
            if inp.n_tiles and w["attn_tc"]:
                cabi.check(L.pg_attention_ragged_tc_capped(
                    ptr(att), att.stride(0), ptr(q), q.stride(0), None, 0, 0, ptr(kp), 0, ptr(vp), 0, self.num_pages * self.page_size,
                    ptr(kv.page_table), kv.max_pages, self.page_size, ptr(inp.tiles), inp.n_tiles, T, a.heads, a.kv_heads, a.dim,
                    a.dim, a.scale, 0, 0, 0, None, 0, None, ptr(w["sink"]), 0.0, 0.0, 0, None, 0, 1.0, ptr(self.err_flag), self.dt,
                    st), "attention_ragged_tc_capped")
            else:
                cabi.check(L.pg_attention_ragged_capped(
                    ptr(att), att.stride(0), ptr(q), q.stride(0), None, 0, 0, ptr(kp), 0, ptr(vp), 0, ptr(kv.page_table),
                    kv.max_pages, self.page_size, ptr(inp.slot), ptr(inp.pos), T, a.heads, a.kv_heads, a.dim, a.dim, a.scale, 0,
                    0, 0, None, 0, None, ptr(w["sink"]), 0.0, 0.0, 0, None, 0, 1.0, ptr(self.attn_ws), self.attn_ws.numel(),
                    self.dt, st), "attention_ragged_capped")
        with tm("o"):
            return self._linear(att, w["o"])

    def _lru(self, kv, inp: StepInputs, ri: int, a: LruCfg, w: dict, proj, conv_state) -> torch.Tensor:
        L, st, tm, T, at = cabi.lib(), cabi.stream(), self._tm, inp.T, w["at"]
        bs = a.width // a.blocks
        u, z = self._new(T, a.width), self._new(T, 2 * a.width, dtype=torch.float32)
        with tm("lru_conv"):
            cabi.check(L.pg_lru_conv(ptr(u), ptr(proj), proj.stride(0), at["x"], ptr(w["x_b"]), ptr(w["r_conv"]), ptr(w["r_conv_b"]),
                                     a.taps, None if conv_state is None else conv_state.data_ptr() + 4 * at["x"], w["conv_len"],
                                     w["conv_cols"], ptr(inp.slot), ptr(inp.pos), T, a.width, self.dt, st), "lru_conv")
        with tm("lru_gates"):
            cabi.check(L.pg_head_gemm_f32(ptr(z), 2 * a.width, 2 * bs, ptr(u), a.width, bs, ptr(w["gates"]), T, a.blocks, 2 * bs, bs,
                                          self.head_impl, ptr(self.err_flag), self.dt, st), "head_gemm_f32")
        out, ws = self._new(T, a.width), self._new(int(L.pg_lru_ws_floats(T, inp.n_segs, a.width)), dtype=torch.float32)
        with tm("lru_scan"):
            cabi.check(L.pg_lru_scan(ptr(out), a.width, ptr(kv.state.layers[("lru", ri)]), ptr(z), ptr(u), ptr(proj[:, at["y"]:]),
                                     proj.stride(0), ptr(w["y_b"]), ptr(w["ra_b"]), ptr(w["ri_b"]), ptr(w["lam"]), LRU_C,
                                     ptr(inp.segs), inp.n_segs, T, a.width, a.blocks, ptr(ws), self.lru_impl, self.dt, st), "lru_scan")
        with tm("o"):
            return self._linear(out, w["r_o"])

    def _parallel(self, kv, inp: StepInputs, ri: int, a: ParallelCfg, w: dict, h) -> dict:
        L, st, tm = cabi.lib(), cabi.stream(), self._tm
        with tm("proj"):
            proj = self._linear(h, w["proj"])
        conv_state = kv.state.layers[("conv", ri)] if w["conv_len"] else None
        left = self._conv_attention(kv, inp, ri, a.left, w, proj, conv_state)
        right = self._lru(kv, inp, ri, a.right, w, proj, conv_state)
        if conv_state is not None:                          # after both readers
            with tm("conv_state"):
                cabi.check(L.pg_time_conv_state(ptr(conv_state), ptr(proj), proj.stride(0), 0, 0, ptr(inp.segs), inp.n_segs,
                                                w["conv_cols"], w["conv_len"] + 1, self.dt, st), "time_conv_state")
        return {"pair": (left, right, w["left_out"], w["right_out"])}

    def _dense(self, h, ml: MlpCfg, w: dict) -> torch.Tensor:
        L, st, tm, T = cabi.lib(), cabi.stream(), self._tm, h.shape[0]
        with tm("gate_up"):
            gu = self._linear(h, w["gu"])
        act = self._new(T, ml.ff)
        with tm("glu"):
            cabi.check(L.pg_glu_clamped(ptr(act), ptr(gu), T, ml.ff, ml.limit, GLU_ALPHA, self.dt, st), "glu_clamped")
        with tm("down"):
            return self._linear(act, w["down"])

    def _moe(self, h, ml: MlpCfg, w: dict) -> dict:
        T, D = h.shape
        idx, wts = self._new(T * ml.top, dtype=torch.int32), self._new(T * ml.top, dtype=torch.float32)
        L, st, z = cabi.lib(), cabi.stream(), None
        with self._tm("moe_route"):
            if T >= self.route_gemm_min and self.dtype != torch.float32 and D % 8 == 0 and ml.experts % 8 == 0:
                z = self._new(T, ml.experts, dtype=torch.float32)       # prompt portions: the fp32 logits on the tensor cores
                cabi.check(L.pg_head_gemm_f32(ptr(z), ml.experts, 0, ptr(h), h.stride(0), 0, ptr(w["router"]), T, 1, ml.experts, D, 0,
                                              ptr(self.err_flag), self.dt, st), "router logits")
            cabi.check(L.pg_moe_route_topk(ptr(idx), ptr(wts), ptr(z), ptr(h), h.stride(0), ptr(w["router"]), ptr(w["router_b"]), T, D,
                                           ml.experts, ml.top, self.dt, st), "moe_route_topk")
        y, pos = self._moe_experts(h, idx, ml.experts, ml.top, ml.ff, w["gu"], w["dn"], cabi.GLU_SILU)
        return {"experts": (y, pos, wts, ml.top)}

    def _forward_device(self, kv, inp: StepInputs, layer_sink: Optional[list]) -> torch.Tensor:
        c, tm = self.cfg, self._tm
        T, nw, D = inp.T, inp.nw, self.cfg.width
        if self.needs_segments and kv.state is None:
            raise RuntimeError("this step's slot table carries no per-sequence state for the model's recurrent layers")
        x = self._new(T, c.streams, D, dtype=torch.float32)
        y = write = None                                    # a sublayer's output that the next row kernel takes into the streams
        emb = True                                          # the streams are still the embedding rows
        for ri, run in enumerate(self.runs):
            lc, w = c.layers[run.layer], self.layers[run.layer]
            h = self._new(T, D)
            self._connect(inp, x, y, write, h, w["read1"], emb=emb)
            emb = emb and y is None
            if lc.kind == "gla":
                y = self._gla(kv, inp, ri, lc.mixer, w, h)
            elif lc.kind == "latent_attention":
                y = self._latent(kv, inp, self.c_pools[ri], lc.mixer, w, h)
            else:
                y = self._parallel(kv, inp, ri, lc.mixer, w, h)
            write = w["write1"]
            if lc.mlp is not None:
                self._connect(inp, x, y, write, h, w["read2"], emb=emb)
                emb = False
                y = self._dense(h, lc.mlp, w) if lc.mlp.kind == "dense" else self._moe(h, lc.mlp, w)
                write = w["write2"]
            if layer_sink is not None:
                self._connect(inp, x, y, write, None, None, emb=emb)
                y, write, emb = None, None, False
                layer_sink.append(x.sum(1))
        if nw == 0:
            return torch.empty((0, c.vocab), dtype=torch.float32, device=self.device)
        hf = self._new(nw, D)                               # only the wanted rows: the last sum over the streams and the norm
        self._connect(inp, x, y, write, hf, self.final_read, emb=emb, rows_idx=inp.want)
        with tm("head"):
            return self._linear(hf, self.head, out_f32=True)

    def weight_bytes(self) -> int:
        n = self.emb.numel() + self.head.numel()
        for w in self.layers:
            n += sum(t.numel() for t in w.values() if isinstance(t, torch.Tensor) and t.dtype == self.dtype)
        return n * torch.tensor([], dtype=self.dtype).element_size()
