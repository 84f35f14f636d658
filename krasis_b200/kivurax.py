"""Kivurax: a decoder-only design whose sublayers read the residual stream as it is and are normed on their output only,
x <- x + m norm1(mixer(x)), x <- x + m norm2(ff(x)), with plain RMS norms and a fixed factor m; the output norm's result meets the embedding
table again (tied head).

Mixers:
  "mlstm"     matrix memory: exponential gates relative to a running maximum, a key sum as normaliser, unit RMS norm per head, a sigmoid
              gate per element (krasis_b200.mixers.MatrixMemory)
  "delta"     gated delta rule with one decay per head, short convolutions on q / k / v (krasis_b200.mixers.GatedDeltaMixer)
  "parallel"  left_scale times
              left   grouped-query attention under a sliding window whose values are the projected keys, ahead of their norm and rotation;
                     query / key RMS norms per head, interleaved rotary pairs with YaRN frequency blending and amplitude, one added to
                     the softmax denominator (krasis_b200.mixers.MultiMapAttention)
              plus right_scale times
              right  Griffin's recurrent block with a real-gated linear recurrent unit (krasis_b200.mixers.GatedRecurrentUnit)
Feed-forward: dense, down(silu(gate h) * (up h)) with biases on all three (krasis_b200.mixers.GatedMLP); or a mixture of such experts
without biases, chosen and weighted by sigmoid scores, the weight on the expert's input (krasis_b200.mixers.RoutedExperts); or none.

config.json keys: architecture, vocab, width, norm.eps, residual_mult, layers [{type, mixer, mlp}] with
  mlstm: heads, dim, vdim, gate_cap;  delta: heads, kv_heads, dim, vdim, conv;
  parallel: left_scale, right_scale, left {heads, kv_heads, dim, vdim, scale, mask.size, rot {base, dims, scaling {factor, original, fast,
  slow}}}, right {width, blocks, conv};
  mlp: null | {kind: "dense", ff} | {kind: "moe", router {experts, top}, expert.ff}.
Tensor names: embed, final.norm, l<i>.norm1, l<i>.norm2;
  mlstm: l<i>.mix.{q, k, v, g, i, i.b, f, f.b, norm, o};  delta: l<i>.mix.{q, k, v}[.conv], l<i>.mix.{g, a, b, A_log, dt_bias, norm, o};
  left: l<i>.mix.left.{q, k}[.norm], l<i>.mix.left.o;
  right: l<i>.mix.right.{x, y, conv, ra, ri}[.b], l<i>.mix.right.{lam, o};
  l<i>.mlp.{gate, up, down}[.b] | l<i>.mlp.{router, e<j>.{gate, up, down}}.

The model exposes the step interface of `krasis_b200.scheduler`: `make_caches`, `forward_step(tables, want_rows)`.
The residual stream, every norm, attention scores, angles, the router and everything that feeds a recurrence are fp32; `dtype` (bfloat16 or
float32) is the type of weights, GEMM inputs and the key / value cache.
"""
import json
import os
from dataclasses import dataclass, field
from typing import List, Optional

import torch

from . import seqops as ops
from .attention import HeadKVCache, RecurrentStatePool
from .mixers import (GatedDeltaMixer, GatedMLP, GatedRecurrentUnit, MatrixMemory, MultiMapAttention, RoutedExperts, SideBySide, lin,
                     yarn_table)

MIXERS = ("mlstm", "delta", "parallel")


@dataclass
class KivuraxConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    layers: List[dict]
    raw: dict = field(default_factory=dict, repr=False)

    @classmethod
    def from_dict(cls, raw: dict) -> "KivuraxConfig":
        cfg = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), eps=float(raw["norm"]["eps"]), residual_mult=float(raw["residual_mult"]),
                  layers=list(raw["layers"]), raw=raw)
        for i, L in enumerate(cfg.layers):
            m, mlp = L["mixer"], L.get("mlp")
            if L["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
            for a in (m, m.get("left", {})):
                if "kv_heads" in a and a["heads"] % a["kv_heads"]:
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if L["type"] == "parallel":
                if m["left"]["vdim"] != m["left"]["dim"]:
                    raise ValueError(f"layer {i}: the values are the keys, vdim must equal dim")
                if m["right"]["width"] % m["right"]["blocks"]:
                    raise ValueError(f"layer {i}: the blocks must divide the width of the recurrence")
            if mlp and mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        return cfg


def _sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):].replace(".", "_"): v for k, v in weights.items() if k.startswith(prefix)}


def random_weights(cfg: KivuraxConfig, seed: int = 0) -> dict:
    """Random tensors of the design's names and shapes (bf16-representable fp32 on the CPU): tests and benchmarks."""
    g = torch.Generator().manual_seed(seed)
    W = cfg.width
    b = lambda t: t.to(torch.bfloat16).float()
    r = lambda *s, sd=1.0: b(torch.randn(*s, generator=g) * sd)
    p_in = lambda rows: r(rows, W, sd=W ** -0.5)
    nw = lambda n: b(1.0 + 0.1 * torch.randn(n, generator=g))
    w = {"embed": r(cfg.vocab, W), "final.norm": nw(W)}
    for i, L in enumerate(cfg.layers):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        q = p + "mix."
        w[p + "norm1"] = nw(W)
        if L["type"] == "mlstm":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            w.update({q + "q": p_in(H * d), q + "k": p_in(H * d), q + "v": p_in(H * dv), q + "g": p_in(H * dv), q + "i": p_in(H), q + "f": p_in(H),
                      q + "i.b": r(H), q + "f.b": b(torch.randn(H, generator=g) + 4.0), q + "norm": nw(H * dv), q + "o": r(W, H * dv, sd=(H * dv) ** -0.5)})
        elif L["type"] == "delta":
            H, G, d, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for nm, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                w.update({q + nm: p_in(rows), q + nm + ".conv": r(rows, K, sd=0.5)})
            w.update({q + "g": p_in(H * dv), q + "a": p_in(H), q + "b": p_in(H), q + "A_log": b(torch.log(1.0 + 7.0 * torch.rand(H, generator=g))),
                      q + "dt_bias": b(torch.randn(H, generator=g) - 3.0), q + "norm": nw(dv), q + "o": r(W, H * dv, sd=(H * dv) ** -0.5)})
        else:
            a, c, u, v = m["left"], m["right"], q + "left.", q + "right."
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            w.update({u + "q": p_in(H * d), u + "k": p_in(G * d), u + "q.norm": nw(d), u + "k.norm": nw(d), u + "o": r(W, H * d, sd=(H * d) ** -0.5)})
            C, B, K = c["width"], c["blocks"], c["conv"]
            n = C // B
            w.update({v + "x": p_in(C), v + "x.b": r(C, sd=0.1), v + "y": p_in(C), v + "y.b": r(C, sd=0.1), v + "conv": r(C, K, sd=0.5),
                      v + "conv.b": r(C, sd=0.1), v + "ra": r(B, n, n, sd=n ** -0.5), v + "ra.b": r(B, n), v + "ri": r(B, n, n, sd=n ** -0.5),
                      v + "ri.b": r(B, n), v + "lam": b(torch.randn(C, generator=g) - 4.0), v + "o": r(W, C, sd=C ** -0.5)})
        if not mlp:
            continue
        w[p + "norm2"] = nw(W)
        q = p + "mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            w.update({q + "gate": p_in(F), q + "up": p_in(F), q + "down": r(W, F, sd=F ** -0.5), q + "gate.b": r(F, sd=0.3), q + "up.b": r(F, sd=0.3),
                      q + "down.b": r(W, sd=0.3)})
        else:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            w[q + "router"] = r(E, W, sd=W ** -0.5 * 2)
            for e in range(E):
                w.update({f"{q}e{e}.gate": p_in(F), f"{q}e{e}.up": p_in(F), f"{q}e{e}.down": r(W, F, sd=F ** -0.5)})
    return w


class KivuraxModel:
    """Weights on the device plus the step function; caches and state slots are made by `make_caches` for a serving session."""

    architecture = "Kivurax"
    page_size = 64

    def __init__(self, cfg: KivuraxConfig, weights: dict, dtype=torch.bfloat16, device=0):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("dtype: bfloat16 or float32")
        if not torch.cuda.is_available():
            raise RuntimeError("KivuraxModel needs a CUDA device (krasis_b200 has no CPU path)")
        ops.load()
        self.cfg, self.dtype = cfg, dtype
        self.device = torch.device("cuda", device) if isinstance(device, int) else torch.device(device)
        dev, eps = self.device, cfg.eps
        f = lambda t: t.to(device=dev, dtype=torch.float32).contiguous()
        self.embed = weights["embed"].to(device=dev, dtype=dtype).contiguous()              # token table and output head
        self.final_norm = f(weights["final.norm"])
        self.layers = []
        for i, L in enumerate(cfg.layers):
            p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
            lay = {"type": L["type"], "norm1": f(weights[p + "norm1"]), "mlp": None}
            if L["type"] == "mlstm":
                lay["mixer"] = MatrixMemory(_sub(weights, p + "mix."), m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps, dtype, dev)
            elif L["type"] == "delta":
                lay["mixer"] = GatedDeltaMixer(_sub(weights, p + "mix."), m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], eps, dtype, dev)
            else:
                lay["mixer"] = self._parallel(m, _sub(weights, p + "mix.left."), _sub(weights, p + "mix.right."))
            if mlp:
                lay["norm2"] = f(weights[p + "norm2"])
                mw = _sub(weights, p + "mlp.")
                if mlp["kind"] == "dense":
                    lay["mlp"] = GatedMLP(mw, dtype, dev, act="silu")
                else:
                    lay["mlp"] = RoutedExperts(mw, mlp["router"]["experts"], 0, mlp["router"]["top"], dtype, dev, score="sigmoid", act="silu",
                                               weight_input=True)
            self.layers.append(lay)

    def _parallel(self, m: dict, lw: dict, rw: dict) -> SideBySide:
        a, c, eps, dtype, dev = m["left"], m["right"], self.cfg.eps, self.dtype, self.device
        rot = a.get("rot") or {}
        dims = int(rot.get("dims", 0))
        freq, amp = yarn_table(dims, rot["base"], rot.get("scaling")) if dims else (None, 1.0)
        left = MultiMapAttention(lw, a["heads"], a["kv_heads"], 1, a["dim"], a["vdim"], a["scale"], eps, dtype, dev,
                                 window=(a.get("mask") or {}).get("size"), rot_dims=dims, rot_freq=freq, rot_amp=amp, keys_as_values=True,
                                 off_by_one=True)
        return SideBySide(left, GatedRecurrentUnit(rw, c["width"], c["blocks"], c["conv"], dtype, dev), scales=(m["left_scale"], m["right_scale"]))

    # ------------------------------------------------------------------------------------------- construction
    @classmethod
    def from_pretrained(cls, model_dir: str, dtype=torch.bfloat16, device=0, **_):
        from . import loader
        cfg = KivuraxConfig.from_dict(json.load(open(os.path.join(model_dir, "config.json"))))
        return cls(cfg, loader.read_named_tensors(model_dir), dtype=dtype, device=device)

    @classmethod
    def random(cls, cfg: KivuraxConfig, seed: int = 0, dtype=torch.bfloat16, device=0):
        return cls(cfg, random_weights(cfg, seed), dtype=dtype, device=device)

    # ------------------------------------------------------------------------------------------- serving interface
    def make_caches(self, max_tokens: int, max_requests: int):
        """(paged cache, state pool) for a session that holds at most max_tokens tokens (each request rounded up to whole pages) in at
        most max_requests live requests.  Only the "parallel" layers cache keys and values; every layer keeps recurrent state in the slots."""
        pages = (max_tokens + self.page_size - 1) // self.page_size
        pool = RecurrentStatePool(max_requests, self.device)
        dims, self._kv_index, self._state = [], [], []
        for lay in self.layers:
            mixer = lay["mixer"]
            if isinstance(mixer, SideBySide):
                self._kv_index.append(len(dims))
                dims.append(mixer.left.cache_dims())
                self._state.append(mixer.right.register_state(pool))
            else:
                self._kv_index.append(-1)
                self._state.append(mixer.register_state(pool))
        self.kv_cache = HeadKVCache(dims, self.device, max_pages=max(pages, 1), dtype=self.dtype, page_size=self.page_size)
        self.state_pool = pool
        return self.kv_cache, pool

    def _mix(self, i: int, h: torch.Tensor, tb: ops.StepTables):
        """Output of layer i's mixer as the terms of the residual update: (y, y2 or None, their factors)."""
        mixer = self.layers[i]["mixer"]
        if not isinstance(mixer, SideBySide):
            return mixer.forward(h, tb, *self._state[i]), None, (1.0, 1.0)
        y = mixer.left.forward(h, tb, *self.kv_cache.get_layer_caches(self._kv_index[i]), self.kv_cache.page_size)
        return y, mixer.right.forward(h, tb, *self._state[i]), mixer.scales

    def forward_step(self, tb: ops.StepTables, want_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """Run the step's tokens through every layer; returns fp32 logits [len(want_rows), vocab] (None if nothing is wanted)."""
        eps, dt, m = self.cfg.eps, self.dtype, self.cfg.residual_mult
        x = ops.embed(self.embed, tb.tokens, 1.0)
        h = ops.residual_post_rms(x, out_dtype=dt)                       # what a sublayer reads: the stream itself, in the GEMM's type
        for i, lay in enumerate(self.layers):
            mlp = lay["mlp"]
            head = dict(out_norm=self.final_norm, out_dtype=torch.float32) if i + 1 == len(self.layers) else dict(out_dtype=dt)
            y, y2, coefs = self._mix(i, h, tb)
            h = ops.residual_post_rms(x, y, lay["norm1"], m, y2=y2, coefs=coefs, eps=eps, **(dict(out_dtype=dt) if mlp is not None else head))
            if mlp is not None:
                h = ops.residual_post_rms(x, mlp.forward(h), lay["norm2"], m, bias=getattr(mlp, "out_bias", None), eps=eps, **head)
            if self.layer_trace is not None:
                self.layer_trace.append(x.clone())
        if not self.layers:
            h = ops.residual_scale_rms(x, norm=self.final_norm, out_dtype=torch.float32, eps=eps)
        if want_rows is None or want_rows.numel() == 0:
            return None
        return lin(h.index_select(0, want_rows), self.embed, torch.float32)

    layer_trace = None      # tests: set to a list to collect the residual stream after every layer
