"""Ranesun: a decoder-only language model with biased layer norms whose mixers are retention (linear attention with a
constant decay per head and rotary positions) or attention over tied keys and values (softcap, softmax sink, a query
temperature that grows with the position, no rotation), dense or mixture-of-experts feed-forwards whose experts are
looked up by token id, and a block of layers that runs several times with the same weights.

Design (every size and every constant that can differ between checkpoints comes from config.json):

  x_0[t]     = embed[token_t]                                                fp32 residual stream
  schedule   : layers 0 .. start-1 once, layers start .. stop-1 `times` times in a row (same weights, but every pass
               has a cache / state of its own), then stop .. n-1 once.  Right before the first layer of pass t:
               x <- x + (embed[token] for t > 0) + step[t].  A layer run is one (layer, pass) pair.
  layer      : x <- x + Mixer(LN1(x)) ;  x <- x + FF(LN2(x))                 (FF may be absent)
  LN(x)      = (x - mean) / sqrt(mean((x - mean)^2) + eps) * w + b
  retention  : q, k = Wq h, Wk h (heads x dim), v = Wv h (heads x vdim); q, k rotated over their first rot.dims columns
               (pairs (i, i + dims/2), angle p * base^(-2i/dims)), k times dim^(-1/2) after it;
               S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t (no softmax, no denominator), S zero at the start;
               Wo (concat_h(o / rms(o)) * silu(Wg h)).
  attention  : q = Wq h, k = Wk h (H query heads over G key heads), the values ARE the keys;
               q at position p times 1 + coef ln(floor((p + 1) / every) + 1); z = scale (q . k_j), j <= p;
               score = softcap tanh(z / softcap); softmax whose denominator also holds exp(sink_h); Wo.
  ff dense   : Wdown (gelu_tanh(Wgate h) * Wup h)
  ff moe     : table[token] names `top` experts, each with weight 1 / top; expert: Wdown relu(Wup h)^2
  output     : logits = embed LN_final(x) * logit_scale                      (the embedding table is the output matrix)

fp32: the residual stream and its sums, every norm, positions and angles, the rotated q and k, attention scores and
weights, decay, state and the recurrence's output with its norm.  Model dtype (fp32 accumulation): projections, the key
cache, the feed-forward.

What the design lets a step do: the experts of a token are known from its id, so the (token, expert) pairs of ALL
mixture layers are grouped in one launch before the first layer, the norm in front of such a layer writes its rows
straight into expert order (no gather), and the next norm sums the experts' rows through the same places (no combine
pass).  One row kernel does everything between two sublayers: sublayer output, embedding output, step vector, norm.
Queries are read by the attention kernels straight from the fused projection; one pool per attention run holds the keys,
which are the values too.  The output scale is folded into the last norm.

The engine owns the repacked weights (one fused projection per mixer), one paged key pool per run of an attention layer
and, through the scheduler's slot table, one fp32 state [slots, heads, dim, vdim] per run of a retention layer.  The step
function, page pool, scheduler and sampling are the framework's (`ragged_engine.RaggedEngine`, `scheduler.SlotKV` /
`SlotState` / `RaggedBatcher`); the recurrence is the decayed linear-attention kernel that Birizen and Gogivik use.
"""
from __future__ import annotations

import warnings
from dataclasses import dataclass, field
from typing import Dict, List, Mapping, Optional

import torch

from . import _cabi as cabi
from ._cabi import ptr
from .ragged_engine import (LoopCfg, RaggedEngine, RotaryCfg, Run, StepInputs, _stack_rows, layer_runs, loop_cfg,
                            rotary_pairs)
from .registry import register


@dataclass
class RetentionCfg:
    heads: int
    dim: int
    vdim: int
    decay: List[float]
    rot: Optional[RotaryCfg]


@dataclass
class TiedAttnCfg:
    heads: int
    kv_heads: int
    dim: int                      # of queries, keys and (the same rows) values
    scale: float
    softcap: float                # 0 = scores are not capped
    temp_coef: float
    temp_every: int               # 0 = no query temperature


@dataclass
class MlpCfg:
    kind: str                     # "dense" | "moe"
    ff: int                       # dense width / expert width
    experts: int = 0
    top: int = 0


@dataclass
class LayerCfg:
    kind: str                     # "retention" | "attention"
    mixer: object
    mlp: Optional[MlpCfg]


def _retention_cfg(i: int, m: Mapping) -> RetentionCfg:
    heads, dim, rot = int(m["heads"]), int(m["dim"]), m.get("rot")
    decay = [float(d) for d in m["decay"]]
    if len(decay) != heads:
        raise ValueError(f"layer {i}: {len(decay)} decays for {heads} heads")
    r = RetentionCfg(heads, dim, int(m.get("vdim", dim)), decay,
                     RotaryCfg(int(rot["dims"]), float(rot["base"])) if rot and int(rot["dims"]) else None)
    if r.rot and (r.rot.dims % 2 or r.rot.dims > dim):
        raise ValueError(f"layer {i}: {r.rot.dims} rotated columns of {dim}")
    return r


def _attention_cfg(i: int, m: Mapping) -> TiedAttnCfg:
    heads, dim, temp = int(m["heads"]), int(m["dim"]), m.get("q_temp") or {}
    a = TiedAttnCfg(heads=heads, kv_heads=int(m.get("kv_heads", heads)), dim=dim, scale=float(m["scale"]),
                    softcap=float(m.get("softcap") or 0.0), temp_coef=float(temp.get("coef", 0.0)),
                    temp_every=int(temp.get("every", 0)))
    if a.heads % a.kv_heads:
        raise ValueError(f"layer {i}: {a.heads} heads over {a.kv_heads} key heads")
    if int(m.get("vdim", dim)) != dim:
        raise ValueError(f"layer {i}: the values are the keys, so vdim {m['vdim']} must be dim {dim}")
    if a.softcap < 0 or a.temp_every < 0 or (temp and a.temp_every != float(temp["every"])):
        raise ValueError(f"layer {i}: softcap {a.softcap}, query temperature {dict(temp)}")
    return a


def _mlp_cfg(i: int, ml: Optional[Mapping]) -> Optional[MlpCfg]:
    if ml is None:
        return None
    if ml.get("kind") == "dense":
        return MlpCfg("dense", int(ml["ff"]))
    if ml.get("kind") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {ml.get('kind')!r}")
    c = MlpCfg("moe", int(ml["expert"]["ff"]), int(ml["router"]["experts"]), int(ml["router"]["top"]))
    if not 1 <= c.top <= c.experts:
        raise ValueError(f"layer {i}: top {c.top} of {c.experts} experts")
    return c


@dataclass
class RanesunConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: List[LayerCfg] = field(default_factory=list)
    loop: Optional[LoopCfg] = None

    def runs(self) -> List[Run]:
        """The layer runs of one forward pass, in order."""
        return layer_runs(len(self.layers), self.loop)

    @staticmethod
    def from_dict(cfg: Mapping) -> "RanesunConfig":
        layers = []
        for i, L in enumerate(cfg["layers"]):
            kind = L.get("type")
            if kind == "retention":
                mixer = _retention_cfg(i, L["mixer"])
            elif kind == "attention":
                mixer = _attention_cfg(i, L["mixer"])
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            layers.append(LayerCfg(kind, mixer, _mlp_cfg(i, L.get("mlp"))))
        return RanesunConfig(vocab=int(cfg["vocab"]), width=int(cfg["width"]), eps=float((cfg.get("norm") or {})["eps"]),
                             logit_scale=float(cfg.get("logit_scale", 1.0)), layers=layers,
                             loop=loop_cfg(cfg.get("loop"), len(layers)))


@register("Ranesun")
class RanesunEngine(RaggedEngine):
    """Weights + paged key pools + recurrent state shapes + the launch sequence of one step over a ragged batch."""

    def __init__(self, config, weights: Mapping[str, torch.Tensor], *, device="cuda", dtype=torch.bfloat16,
                 page_size: int = 64, kv_pool_tokens: int = 65536, gemm_impl: int = 0, strict: bool = False):
        self.cfg = config if isinstance(config, RanesunConfig) else RanesunConfig.from_dict(config)
        self.strict = bool(strict)      # True: tensors the config does not call for raise instead of being reported
        self._init_common(device=device, dtype=dtype, page_size=page_size, gemm_impl=gemm_impl)
        self.runs = self.cfg.runs()
        self.needs_segments = any(self.cfg.layers[r.layer].kind == "retention" for r in self.runs)
        self._repack(weights)
        L_ = cabi.lib()
        for w, lc in zip(self.layers, self.cfg.layers):     # prompt portions of layers whose sizes the tensor-core kernel takes
            a = lc.mixer
            w["attn_tc"] = lc.kind == "attention" and (a.softcap > 0 or a.temp_every == 0) and bool(L_.pg_attention_ragged_tc_ok8(
                a.dim, a.dim, self.page_size, w["proj"].shape[0], a.heads * a.dim, 8, self.dt))
        self._attn_tc_any = any(w["attn_tc"] for w in self.layers)
        self._init_runtime(kv_pool_tokens)
        # one key pool per RUN of an attention layer: a layer that runs twice keeps two caches
        self.k_pools: Dict[int, torch.Tensor] = {}
        for ri, r in enumerate(self.runs):
            lc = self.cfg.layers[r.layer]
            if lc.kind == "attention":
                self.k_pools[ri] = torch.zeros((self.num_pages, self.page_size, lc.mixer.kv_heads * lc.mixer.dim), dtype=dtype,
                                               device=self.device)

    # ------------------------------------------------------------------ weights
    def _repack(self, weights: Mapping[str, torch.Tensor]) -> None:
        c, D, f32 = self.cfg, self.cfg.width, torch.float32
        used = set()

        def W(name, shape=None, dtype=None):
            if name not in weights:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            used.add(name)
            t = weights[name]
            if shape is not None and tuple(t.shape) != tuple(shape):
                raise ValueError(f"tensor {name}: shape {tuple(t.shape)}, the config wants {tuple(shape)}")
            return t.to(device=self.device, dtype=dtype or self.dtype).contiguous()

        self.emb, self.final_norm, self.final_bias = W("embed", (c.vocab, D)), W("final.norm", (D,)), W("final.norm.b", (D,))
        self.loop_step = W("loop.step", (c.loop.times, D)) if c.loop is not None else None
        self.layers: List[dict] = []
        tables, desc = [], []                # of the mixture layers: expert tables, {start, experts, top, earlier top, earlier offsets}
        entries = tops = offs = 0
        for i, L in enumerate(c.layers):
            p, m, a = f"l{i}.", f"l{i}.mix.", L.mixer
            w = dict(norm1=W(p + "norm1", (D,)), norm1_b=W(p + "norm1.b", (D,)))
            if L.kind == "retention":
                nk, nv = a.heads * a.dim, a.heads * a.vdim
                w["proj"], w["at"] = _stack_rows([("q", W(m + "q", (nk, D))), ("k", W(m + "k", (nk, D))),
                                                  ("v", W(m + "v", (nv, D))), ("g", W(m + "g", (nv, D)))],
                                                 self.device, self.dtype)
                w.update(o=W(m + "o", (D, nv)), decay=torch.tensor(a.decay, dtype=f32, device=self.device),
                         freq=rotary_pairs(a.rot).to(self.device) if a.rot else None)
            else:
                nq, nk = a.heads * a.dim, a.kv_heads * a.dim
                w["proj"], w["at"] = _stack_rows([("q", W(m + "q", (nq, D))), ("k", W(m + "k", (nk, D)))], self.device, self.dtype)
                w.update(sink=W(m + "sink", (a.heads,), f32), o=W(m + "o", (D, nq)))
            ml = L.mlp
            if ml is not None:
                f = p + "mlp."
                w.update(norm2=W(p + "norm2", (D,)), norm2_b=W(p + "norm2.b", (D,)))
                if ml.kind == "dense":
                    w.update(gu=torch.cat([W(f + "gate", (ml.ff, D)), W(f + "up", (ml.ff, D))], 0).contiguous(),
                             down=W(f + "down", (D, ml.ff)))
                else:
                    w.update(up=torch.stack([W(f"{f}e{e}.up", (ml.ff, D)) for e in range(ml.experts)], 0).contiguous(),
                             dn=torch.stack([W(f"{f}e{e}.down", (D, ml.ff)) for e in range(ml.experts)], 0).contiguous())
                    t = W(f + "table", (c.vocab, ml.top), torch.int32)
                    if int(t.min()) < 0 or int(t.max()) >= ml.experts:
                        raise ValueError(f"tensor {f}table names experts outside 0 .. {ml.experts - 1}")
                    desc.append([entries, ml.experts, ml.top, tops, offs])
                    w["route"] = (tops, offs)
                    tables.append(t.reshape(-1))
                    entries, tops, offs = entries + t.numel(), tops + ml.top, offs + ml.experts + 1
            self.layers.append(w)
        self.tables = torch.cat(tables) if tables else None
        self.route_desc = torch.tensor(desc, dtype=torch.int32, device=self.device) if desc else None
        self.route_tops, self.route_offs = tops, offs
        self.max_experts = max((d[1] for d in desc), default=0)
        extra = sorted(set(weights) - used)
        if extra:
            text = f"checkpoint holds {len(extra)} tensor(s) the config does not call for: {extra[:8]}"
            if self.strict:
                raise ValueError(text)
            warnings.warn(text + " (not used)")

    # ------------------------------------------------------------------ recurrent state
    def new_slot_state(self, slots: int):
        from .scheduler import SlotState
        shapes = {}
        for ri, r in enumerate(self.runs):
            L = self.cfg.layers[r.layer]
            if L.kind == "retention":
                shapes[ri] = (L.mixer.heads, L.mixer.dim, L.mixer.vdim)
        return SlotState(slots, shapes, self.device) if shapes else None

    # ------------------------------------------------------------------ one step
    def _between(self, inp: StepInputs, x, y, out, w=None, b=None, *, emb=cabi.EMB_NONE, vec=None, out_route=None,
                 rows_idx=None, out_scale: float = 1.0) -> None:
        """x += y (a dense sublayer output, or (rows, places, top) of experts) + embedding row + vec; out = LN(x) w + b, its
        rows in token order or at the places out_route = (places, top) of the token's experts."""
        rows = x.shape[0] if rows_idx is None else rows_idx.shape[0]
        yt, y_pos, y_top = y if isinstance(y, tuple) else (y, None, 1)
        o_pos, o_top = out_route if out_route is not None else (None, 1)
        cabi.check(cabi.lib().pg_residual_layernorm(
            ptr(out), 0 if out is None else out.stride(0), ptr(x), ptr(yt), 0 if yt is None else yt.stride(0), ptr(y_pos), y_top,
            1.0 / y_top, ptr(inp.ids), ptr(self.emb), self.cfg.vocab, emb, ptr(vec), ptr(w), ptr(b), self.cfg.eps, out_scale,
            ptr(rows_idx), ptr(o_pos), o_top, rows, self.cfg.width, ptr(self.err_flag), self.dt, cabi.stream()),
            "residual_layernorm")

    def _retention(self, kv, inp: StepInputs, ri: int, a: RetentionCfg, w: dict, h) -> torch.Tensor:
        L, st, tm, T, at = cabi.lib(), cabi.stream(), self._tm, inp.T, w["at"]
        if kv.state is None or ri not in kv.state.layers:
            raise RuntimeError("this step's slot table carries no recurrent state for the model's retention layers")
        with tm("proj"):
            proj = self._linear(h, w["proj"])
        nv = a.heads * a.vdim
        rec = self._new(int(L.pg_lightning_record_floats(T, a.heads, a.dim, a.vdim)), dtype=torch.float32)
        with tm("retention_prep"):
            cabi.check(L.pg_retention_prep(ptr(rec), ptr(proj), proj.stride(0), at["q"], at["k"], at["v"], ptr(w["freq"]),
                                           a.rot.dims if a.rot else 0, 0, a.dim ** -0.5, ptr(inp.pos), T, a.heads, a.dim,
                                           a.vdim, self.dt, st), "retention_prep")
        o = self._new(T, nv, dtype=torch.float32)
        with tm("retention"):
            cabi.check(L.pg_lightning_attention(ptr(o), ptr(kv.state.layers[ri]), ptr(rec), ptr(w["decay"]), ptr(inp.segs),
                                                inp.n_segs, a.heads, a.dim, a.vdim, st), "retention")
        g = self._new(T, nv)
        with tm("headnorm_gate"):
            cabi.check(L.pg_headnorm_gate_ex(ptr(g), nv, ptr(o), None, ptr(proj[:, at["g"]:]), proj.stride(0), 1, T, a.heads,
                                             a.vdim, self.cfg.eps, 1.0, self.dt, st), "headnorm_gate")
        with tm("o"):
            return self._linear(g, w["o"])

    def _attention(self, kv, inp: StepInputs, ri: int, a: TiedAttnCfg, w: dict, h) -> torch.Tensor:
        L, st, tm, T, at = cabi.lib(), cabi.stream(), self._tm, inp.T, w["at"]
        with tm("proj"):
            proj = self._linear(h, w["proj"])
        pool, nk = self.k_pools[ri], a.kv_heads * a.dim
        with tm("cache_append"):
            cabi.check(L.pg_cache_append(ptr(pool), nk, ptr(proj), proj.stride(0), at["k"], nk, ptr(kv.page_table), kv.max_pages,
                                         self.page_size, ptr(inp.slot), ptr(inp.pos), T, self.dt, st), "cache_append")
        att = self._new(T, a.heads * a.dim)
        q = proj[:, at["q"]:]                               # read in place: the temperature enters with the score's scale
        with tm("attention"):
            if inp.n_tiles and w["attn_tc"]:
                cabi.check(L.pg_attention_ragged_tc_capped(
                    ptr(att), att.stride(0), ptr(q), q.stride(0), None, 0, 0, ptr(pool), 0, ptr(pool), 0,
                    self.num_pages * self.page_size, ptr(kv.page_table), kv.max_pages, self.page_size, ptr(inp.tiles),
                    inp.n_tiles, T, a.heads, a.kv_heads, a.dim, a.dim, a.scale, 0, 0, 0, None, 0, None, ptr(w["sink"]),
                    a.softcap, a.temp_coef, a.temp_every, None, 0, 1.0, ptr(self.err_flag), self.dt, st),
                    "attention_ragged_tc_capped")
            else:
                cabi.check(L.pg_attention_ragged_capped(
                    ptr(att), att.stride(0), ptr(q), q.stride(0), None, 0, 0, ptr(pool), 0, ptr(pool), 0, ptr(kv.page_table),
                    kv.max_pages, self.page_size, ptr(inp.slot), ptr(inp.pos), T, a.heads, a.kv_heads, a.dim, a.dim, a.scale,
                    0, 0, 0, None, 0, None, ptr(w["sink"]), a.softcap, a.temp_coef, a.temp_every, None, 0, 1.0,
                    ptr(self.attn_ws), self.attn_ws.numel(), self.dt, st), "attention_ragged_capped")
        with tm("o"):
            return self._linear(att, w["o"])

    def _route(self, inp: StepInputs):
        """The grouping of every mixture layer's (token, expert) pairs, from the token ids alone: (offsets, places)."""
        if self.tables is None:
            return None, None
        offsets = self._new(self.route_offs, dtype=torch.int32)
        places = self._new(inp.T * self.route_tops, dtype=torch.int32)
        with self._tm("moe_table_sort"):
            cabi.check(cabi.lib().pg_moe_table_sort(ptr(offsets), ptr(places), ptr(self.tables), ptr(self.route_desc),
                                                    self.route_desc.shape[0], ptr(inp.ids), inp.T, self.cfg.vocab,
                                                    self.max_experts, cabi.stream()), "moe_table_sort")
        return offsets, places

    def _forward_device(self, kv, inp: StepInputs, layer_sink: Optional[list]) -> torch.Tensor:
        c, tm = self.cfg, self._tm
        T, nw, D = inp.T, inp.nw, self.cfg.width
        offsets, places = self._route(inp)
        x = self._new(T, D, dtype=torch.float32)
        y = None                                            # a sublayer's output that the next row kernel sums into x
        for ri, run in enumerate(self.runs):
            lc, w = c.layers[run.layer], self.layers[run.layer]
            emb = cabi.EMB_INIT if ri == 0 else (cabi.EMB_ADD if run.loop_pass else cabi.EMB_NONE)
            vec = None if run.loop_pass is None else self.loop_step[run.loop_pass]
            h = self._new(T, D)
            with tm("norm"):
                self._between(inp, x, y, h, w["norm1"], w["norm1_b"], emb=emb, vec=vec)
            mixer = self._retention if lc.kind == "retention" else self._attention
            y = mixer(kv, inp, ri, lc.mixer, w, h)
            ml = lc.mlp
            if ml is not None and ml.kind == "dense":
                with tm("norm"):
                    self._between(inp, x, y, h, w["norm2"], w["norm2_b"])
                with tm("gate_up"):
                    act = self._linear(h, w["gu"], cabi.EPI_GEGLU)
                with tm("down"):
                    y = self._linear(act, w["down"])
            elif ml is not None:
                tops, offs = w["route"]
                pos, P = places[T * tops:T * (tops + ml.top)], T * ml.top
                hp = self._new(P, D)                        # the norm's rows in expert order, once per chosen expert
                with tm("norm_scatter"):
                    self._between(inp, x, y, hp, w["norm2"], w["norm2_b"], out_route=(pos, ml.top))
                y = (self._moe_ffn(hp, None, offsets[offs:], P, ml.experts, ml.ff, w["up"], w["dn"], cabi.ACT_RELU2), pos, ml.top)
            if layer_sink is not None:
                self._between(inp, x, y, None)
                y = None
                layer_sink.append(x.clone())
        if nw == 0:
            return torch.empty((0, c.vocab), dtype=torch.float32, device=self.device)
        hf = self._new(nw, D)
        with tm("norm"):                                    # only the wanted rows: the last sum, the norm, the output scale
            self._between(inp, x, y, hf, self.final_norm, self.final_bias, rows_idx=inp.want, out_scale=c.logit_scale)
        with tm("head"):
            return self._linear(hf, self.emb, out_f32=True)

    def weight_bytes(self) -> int:
        n = self.emb.numel() + self.final_norm.numel() + self.final_bias.numel()
        if self.loop_step is not None:
            n += self.loop_step.numel()
        for w in self.layers:
            n += sum(t.numel() for t in w.values() if isinstance(t, torch.Tensor) and t.dtype == self.dtype)
        return n * torch.tensor([], dtype=self.dtype).element_size()
