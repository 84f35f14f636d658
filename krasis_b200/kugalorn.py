"""Kugalorn: a decoder-only design of pre-normed layers whose residual stream exists in several copies (hyper-connections).  A sublayer
reads a weighted sum of the copies, and its output y goes back to all of them at once: with the copies x_s of before,
x_t <- sum_s mix[s, t] x_s + out[t] y.  All copies start as the embedding output; after the last layer their sum goes to the output
norm and the head, a tensor of its own.  Norms are RMS norms whose weight tensor holds the distance from one.

Mixers:
  "attention"         grouped-query attention under a sliding window; no rotation: queries and keys are divided by their root mean square
                      per head, and slope_h times the distance to the key is taken off the scores, slope_h = 2^(-8 (h + 1) / heads)
                      (krasis_b200.mixers.MultiMapAttention)
  "latent_attention"  causal attention over a cached low-rank latent plus one shared rotated key part, interleaved rotary pairs on the
                      rotated part, a sigmoid output gate per head (krasis_b200.mixers.WindowLatentAttention)
Feed-forward: a mixture of clamped-swish experts (min(g, limit) sigmoid(1.702 g) (clamp(u) + 1)) chosen by the largest biased router
logits and weighted by a softmax over the chosen ones, plus a shared expert with sizes and limit of its own; or none
(krasis_b200.mixers.RoutedExperts).
A span of layers may run several times in a row with the same weights; every run has a cache of its own.

config.json keys: architecture, vocab, width, streams, norm.eps, loop {start, stop, times} (optional), layers [{type, mixer, mlp}] with
  attention: heads, kv_heads, dim, vdim, scale, mask.size;
  latent_attention: heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims};
  mlp: null | {kind: "moe", router {experts, top}, expert {ff, limit}, shared {ff, limit} (optional)}.
Tensor names: embed, head, final.norm, l<i>.norm1, l<i>.norm2, l<i>.hc{1, 2}.{in, out, mix};
  l<i>.mix.{q, k, v, o} | l<i>.mix.{q, dkv, dkv.norm, uk, uv, g, o};  l<i>.mlp.{router, router.b, e<j>.{gate, up, down},
  shared.{gate, up, down}}.

The model exposes the step interface of `krasis_b200.scheduler`: `make_caches`, `forward_step(tables, want_rows)`.
The copies of the residual stream, every norm, attention scores, angles and the router are fp32; `dtype` (bfloat16 or float32) is the type
of weights, GEMM inputs and the caches.
"""
import json
import os
from dataclasses import dataclass, field
from typing import List, Optional

import torch

from . import seqops as ops
from .attention import HeadKVCache, RecurrentStatePool
from .mixers import MultiMapAttention, RoutedExperts, WindowLatentAttention, distance_slopes, layer_runs, lin, rotary_table

SWISH_ALPHA = 1.702      # slope inside the sigmoid of the experts' activation
NORM_SHIFT = 1.0         # a norm's weight tensor holds the offset from one


@dataclass
class KugalornConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    layers: List[dict]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    raw: dict = field(default_factory=dict, repr=False)

    @classmethod
    def from_dict(cls, raw: dict) -> "KugalornConfig":
        loop = raw.get("loop") or {}
        cfg = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), eps=float(raw["norm"]["eps"]), streams=int(raw["streams"]),
                  layers=list(raw["layers"]), loop_start=int(loop.get("start", 0)), loop_stop=int(loop.get("stop", 0)),
                  loop_times=int(loop.get("times", 1)), raw=raw)
        if not 1 <= cfg.streams <= 32:
            raise ValueError("streams: 1 to 32")
        if not 0 <= cfg.loop_start <= cfg.loop_stop <= len(cfg.layers) or cfg.loop_times < 1:
            raise ValueError("loop span outside the layer list, or run less than once")
        for i, L in enumerate(cfg.layers):
            m, mlp = L["mixer"], L.get("mlp")
            if L["type"] not in ("attention", "latent_attention"):
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
            if L["type"] == "attention" and m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if L["type"] == "latent_attention" and m["rot"]["dims"] != m["rot_dim"]:
                raise ValueError(f"layer {i}: the rotated part turns in all of its dimensions")
            if mlp and mlp.get("kind") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        return cfg

    def runs(self):
        """Layer indices in execution order."""
        return [i for i, _ in layer_runs(len(self.layers), self.loop_start, self.loop_stop, self.loop_times)]


def _sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):].replace(".", "_"): v for k, v in weights.items() if k.startswith(prefix)}


def random_weights(cfg: KugalornConfig, seed: int = 0) -> dict:
    """Random tensors of the design's names and shapes (bf16-representable fp32 on the CPU): tests and benchmarks."""
    g = torch.Generator().manual_seed(seed)
    W, n = cfg.width, cfg.streams
    b = lambda t: t.to(torch.bfloat16).float()
    r = lambda *s, sd=1.0: b(torch.randn(*s, generator=g) * sd)
    w = {"embed": r(cfg.vocab, W), "head": r(cfg.vocab, W, sd=W ** -0.5), "final.norm": r(W, sd=0.1)}

    def expert(p, F):
        w.update({p + "gate": r(F, W, sd=W ** -0.5), p + "up": r(F, W, sd=W ** -0.5), p + "down": r(W, F, sd=F ** -0.5)})

    for i, L in enumerate(cfg.layers):
        p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        H, dv = m["heads"], m["vdim"]
        for q in (1, 2) if mlp else (1,):
            w[p + f"norm{q}"] = r(W, sd=0.1)
            w[p + f"hc{q}.in"] = b(torch.full((n,), 1.0 / n) + 0.2 * torch.randn(n, generator=g))
            w[p + f"hc{q}.out"] = b(torch.ones(n) + 0.3 * torch.randn(n, generator=g))
            w[p + f"hc{q}.mix"] = b(0.8 * torch.eye(n) + 0.2 / n + 0.1 * torch.randn(n, n, generator=g))
        if L["type"] == "attention":
            G, d = m["kv_heads"], m["dim"]
            w.update({p + "mix.q": r(H * d, W, sd=W ** -0.5), p + "mix.k": r(G * d, W, sd=W ** -0.5), p + "mix.v": r(G * dv, W, sd=W ** -0.5)})
        else:
            dn, dr, rk = m["dim"], m["rot_dim"], m["kv_rank"]
            w.update({p + "mix.q": r(H * (dn + dr), W, sd=W ** -0.5), p + "mix.dkv": r(rk + dr, W, sd=W ** -0.5),
                      p + "mix.dkv.norm": b(1.0 + 0.1 * torch.randn(rk, generator=g)), p + "mix.uk": r(H * dn, rk, sd=rk ** -0.5),
                      p + "mix.uv": r(H * dv, rk, sd=rk ** -0.5), p + "mix.g": r(H, W, sd=W ** -0.5)})
        w[p + "mix.o"] = r(W, H * dv, sd=(H * dv) ** -0.5)
        if mlp:
            E = mlp["router"]["experts"]
            w.update({p + "mlp.router": r(E, W, sd=W ** -0.5 * 2), p + "mlp.router.b": r(E, sd=0.3)})
            for e in range(E):
                expert(p + f"mlp.e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                expert(p + "mlp.shared.", mlp["shared"]["ff"])
    return w


class KugalornModel:
    """Weights on the device plus the step function; the cache pools are made by `make_caches` for a serving session."""

    architecture = "Kugalorn"
    page_size = 64

    def __init__(self, cfg: KugalornConfig, weights: dict, dtype=torch.bfloat16, device=0):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("dtype: bfloat16 or float32")
        if not torch.cuda.is_available():
            raise RuntimeError("KugalornModel needs a CUDA device (krasis_b200 has no CPU path)")
        ops.load()
        self.cfg, self.dtype = cfg, dtype
        self.device = torch.device("cuda", device) if isinstance(device, int) else torch.device(device)
        dev, eps = self.device, cfg.eps
        d = lambda t: t.to(device=dev, dtype=dtype).contiguous()
        f = lambda t: t.to(device=dev, dtype=torch.float32).contiguous()
        self.embed, self.head, self.final_norm = d(weights["embed"]), d(weights["head"]), f(weights["final.norm"])
        self.layers = []
        for i, L in enumerate(cfg.layers):
            p, m, mlp = f"l{i}.", L["mixer"], L.get("mlp")
            mw = _sub(weights, p + "mix.")
            if L["type"] == "attention":
                mixer = MultiMapAttention(mw, m["heads"], m["kv_heads"], 1, m["dim"], m["vdim"], m["scale"], eps, dtype, dev,
                                          window=m["mask"]["size"], qk_unit=True, slopes=distance_slopes(m["heads"]))
            else:
                dims, base = m["rot"]["dims"], m["rot"]["base"]
                mixer = WindowLatentAttention(mw, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], None, dims, base,
                                              None, eps, dtype, dev, rot_freq=rotary_table(dims, base))
            lay = {"type": L["type"], "mixer": mixer, "mlp": None}
            for q in (1, 2) if mlp else (1,):
                lay[f"norm{q}"] = f(weights[p + f"norm{q}"])
                lay[f"hc{q}"] = {k: f(weights[p + f"hc{q}.{k}"]) for k in ("in", "out", "mix")}
            if mlp:
                sh = mlp.get("shared") or {}
                lay["mlp"] = RoutedExperts(_sub(weights, p + "mlp."), mlp["router"]["experts"], 0, mlp["router"]["top"], dtype, dev,
                                           score="top_softmax", act="clamped_swish", limit=mlp["expert"]["limit"], alpha=SWISH_ALPHA,
                                           shared_limit=sh.get("limit"))
            self.layers.append(lay)
        self.runs = cfg.runs()
        # (run, layer, sublayer 1 | 2) in execution order
        self.sublayers = [(ri, li, q) for ri, li in enumerate(self.runs) for q in ((1, 2) if self.layers[li]["mlp"] is not None else (1,))]

    # ------------------------------------------------------------------------------------------- construction
    @classmethod
    def from_pretrained(cls, model_dir: str, dtype=torch.bfloat16, device=0, **_):
        from . import loader
        cfg = KugalornConfig.from_dict(json.load(open(os.path.join(model_dir, "config.json"))))
        return cls(cfg, loader.read_named_tensors(model_dir), dtype=dtype, device=device)

    @classmethod
    def random(cls, cfg: KugalornConfig, seed: int = 0, dtype=torch.bfloat16, device=0):
        return cls(cfg, random_weights(cfg, seed), dtype=dtype, device=device)

    # ------------------------------------------------------------------------------------------- serving interface
    def make_caches(self, max_tokens: int, max_requests: int):
        """(paged cache, state pool) for a session that holds at most max_tokens tokens (each request rounded up to whole pages) in at
        most max_requests live requests.  Every run of a layer gets pools of its own: keys and values, or latents and the rotated key
        part.  The design has no recurrent state: the state pool only hands out request slots."""
        pages = (max_tokens + self.page_size - 1) // self.page_size
        dims = [self.layers[li]["mixer"].cache_dims() for li in self.runs]
        self.kv_cache = HeadKVCache(dims, self.device, max_pages=max(pages, 1), dtype=self.dtype, page_size=self.page_size)
        self.state_pool = RecurrentStatePool(max_requests, self.device)
        return self.kv_cache, self.state_pool

    def forward_step(self, tb: ops.StepTables, want_rows: Optional[torch.Tensor]) -> Optional[torch.Tensor]:
        """Run the step's tokens through every layer run; returns fp32 logits [len(want_rows), vocab] (None if nothing is wanted)."""
        cfg, eps, dt = self.cfg, self.cfg.eps, self.dtype
        x0 = ops.embed(self.embed, tb.tokens, 1.0)
        xs = torch.empty((x0.shape[0], cfg.streams, cfg.width), dtype=torch.float32, device=x0.device)
        back = {"x0": x0}                       # what the copies take up next: the embedding output, then each sublayer's output
        for k, (ri, li, q) in enumerate(self.sublayers):
            lay = self.layers[li]
            hc = lay[f"hc{q}"]
            # one pass: the copies take up what came before, this sublayer's input is read from them and normed
            h = ops.stream_mix(xs, read=hc["in"], norm=lay[f"norm{q}"], w_shift=NORM_SHIFT, out_dtype=dt, eps=eps, **back)
            if self.layer_trace is not None and q == 1 and k > 0:
                self.layer_trace.append(xs.sum(1))
            if q == 1:
                y = lay["mixer"].forward(h, tb, *self.kv_cache.get_layer_caches(ri), self.kv_cache.page_size)
            else:
                y = lay["mlp"].forward(h)
            back = {"y": y, "mix": hc["mix"], "out": hc["out"]}
        h = ops.stream_mix(xs, norm=self.final_norm, w_shift=NORM_SHIFT, out_dtype=torch.float32, eps=eps, **back)
        if self.layer_trace is not None and self.sublayers:
            self.layer_trace.append(xs.sum(1))
        if want_rows is None or want_rows.numel() == 0:
            return None
        return lin(h.index_select(0, want_rows), self.head, torch.float32)

    layer_trace = None      # tests: set to a list to collect the sum of the copies after every layer run
