"""Kugalorn on the GPU against the plain float64 oracle (tests/oracle_kugalorn.py): each mechanism alone, then the whole model through the
scheduler — prefill against decoding, portions down to two tokens, unequal batches, reuse of pages and slots, far keys, page borders and
window edges with peaked scores, the first tokens of a sequence, long decoding, odd sizes, looped spans, and greedy generation through
the generation entry point.  Small random configurations made here; none of them is a shipped model's."""
import json
import struct

import numpy as np
import pytest
import torch

from tests import oracle_kugalorn as O

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
EPS = 1e-5


@pytest.fixture(scope="module")
def seq():
    from krasis_b200.build import build_seq
    build_seq()
    from krasis_b200 import seqops
    seqops.load()
    return seqops


# ------------------------------------------------------------------------------------------------ configurations
def att(heads=4, kv_heads=2, dim=12, vdim=10, size=9, scale=0.3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}


def latent(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=12, base=300.0, scale=0.25):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}


def moe(experts=6, top=2, ff=20, limit=0.7, shared_ff=13, shared_limit=1.1):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared_ff:
        m["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return m


def AT(m=None, mlp="moe"):
    return {"type": "attention", "mixer": m or att(), "mlp": moe() if mlp == "moe" else mlp}


def LA(m=None, mlp="moe"):
    return {"type": "latent_attention", "mixer": m or latent(), "mlp": moe() if mlp == "moe" else mlp}


def model_cfg(layers, width=40, vocab=50, eps=EPS, streams=3, loop=None):
    raw = {"architecture": "Kugalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers}
    if loop:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return raw


def default_cfg(**kw):
    layers = [LA(), AT(), AT(att(heads=6, kv_heads=6, dim=8, vdim=16, size=30), mlp=None),
              LA(latent(heads=5, dim=4, rot_dim=8, vdim=6, kv_rank=7, base=50.0), moe(experts=5, top=5, ff=17, shared_ff=0)),
              AT(att(heads=3, kv_heads=1, dim=16, vdim=4, size=5), moe(experts=9, top=1, ff=8, limit=2.0, shared_ff=24, shared_limit=0.4))]
    return model_cfg(layers, **dict({"loop": (1, 4, 2)}, **kw))


def build(raw, dtype=torch.float32, seed=0, page_size=None, tweak=None):
    from krasis_b200.kugalorn import KugalornConfig, KugalornModel, random_weights
    cfg = KugalornConfig.from_dict(raw)
    w = random_weights(cfg, seed)
    if tweak:
        tweak(w)
    model = KugalornModel(cfg, w, dtype=dtype)
    if page_size:
        model.page_size = page_size
    return model, f64(w)


def sched(model, max_tokens=512, max_requests=4, **kw):
    from krasis_b200.scheduler import Scheduler
    return Scheduler(model, max_tokens=max_tokens, max_requests=max_requests, **kw)


def toks(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def close(got, want, rel, what=""):
    got = np.asarray(got, dtype=np.float64)
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-9)
    assert err <= rel, f"{what}: relative error {err:.3e} > {rel:.1e}"


def differs(other, want, rel):
    assert np.abs(other - want).max() > rel * np.abs(want).max()


def run_portions(model, tokens, cuts, s=None, rid="a", finish=True):
    """Feed `tokens` in portions of the given sizes (the rest one by one); logits of every position."""
    s = s or sched(model)
    out, at = [], 0
    for n in list(cuts) + [1] * (len(tokens) - sum(cuts)):
        out.append(s.step([(rid, tokens[at:at + n], list(range(n)))]).cpu().numpy())
        at += n
    if finish:
        s.finish(rid)
    return np.concatenate(out, 0)


def rnd(*shape, seed=0, sd=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * sd).to(torch.bfloat16).float()


def f64(d):
    return {k: v.numpy().astype(np.float64) for k, v in d.items()}


def n64(t):
    return t.numpy().astype(np.float64)


def under(d):
    return {k.replace(".", "_"): v for k, v in d.items()}


# ------------------------------------------------------------------------------------------------ mechanisms alone
def att_weights(m, W, seed):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": rnd(H * d, W, seed=seed, sd=W ** -0.5), "k": rnd(G * d, W, seed=seed + 1, sd=W ** -0.5), "v": rnd(G * dv, W, seed=seed + 2, sd=W ** -0.5),
            "o": rnd(W, H * dv, seed=seed + 3, sd=0.2)}


def make_att(m, w, dtype=torch.float32):
    from krasis_b200.mixers import MultiMapAttention, distance_slopes
    return MultiMapAttention(under(w), m["heads"], m["kv_heads"], 1, m["dim"], m["vdim"], m["scale"], EPS, dtype, torch.device(DEV),
                             window=m["mask"]["size"], qk_unit=True, slopes=distance_slopes(m["heads"]))


def latent_weights(m, W, seed):
    H, dn, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    return {"q": rnd(H * (dn + dr), W, seed=seed, sd=W ** -0.5 * 2), "dkv": rnd(r + dr, W, seed=seed + 3, sd=W ** -0.5 * 2),
            "dkv.norm": 1 + rnd(r, seed=seed + 4, sd=0.3), "uk": rnd(H * dn, r, seed=seed + 5, sd=r ** -0.5 * 2),
            "uv": rnd(H * dv, r, seed=seed + 6, sd=r ** -0.5), "g": rnd(H, W, seed=seed + 7, sd=W ** -0.5 * 2), "o": rnd(W, H * dv, seed=seed + 8, sd=0.2)}


def make_latent(m, w, dtype=torch.float32):
    from krasis_b200.mixers import WindowLatentAttention, rotary_table
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    return WindowLatentAttention(under(w), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], None, dims, base, None, EPS,
                                 dtype, torch.device(DEV), rot_freq=rotary_table(dims, base))


def run_mixer(seq, mixer, h, cuts, page_size=4):
    """One sequence through a mixer with a paged cache of its own, in portions (the rest one by one)."""
    from krasis_b200.attention import HeadKVCache, SequenceKVState
    T = h.shape[0]
    kv = HeadKVCache([mixer.cache_dims()], DEV, max_pages=(T + page_size - 1) // page_size + 2, dtype=mixer.dtype, page_size=page_size)
    st, out, at = SequenceKVState(kv), [], 0
    for n in list(cuts) + [1] * (T - sum(cuts)):
        st.ensure_capacity(n)
        tb = seq.StepTables([([0] * n, st.seq_len, 1, st.pages)], torch.device(DEV))
        out.append(mixer.forward(h[at:at + n].to(DEV, mixer.dtype).contiguous(), tb, *kv.get_layer_caches(0), page_size).cpu().numpy())
        st.advance(n)
        at += n
    return np.concatenate(out, 0)


CUTS = ([41], [], [2, 2, 5, 17], [30, 2], [3, 1, 1, 9, 2])


@pytest.mark.parametrize("m", [att(), att(heads=2, kv_heads=2, dim=32, vdim=8, size=5), att(heads=8, kv_heads=1, dim=6, vdim=70, size=12),
                               att(heads=3, kv_heads=3, dim=10, vdim=33, size=100, scale=0.7), att(heads=5, kv_heads=1, dim=16, vdim=16, size=1),
                               att(heads=1, kv_heads=1, dim=4, vdim=2, size=41), att(heads=12, kv_heads=4, dim=64, vdim=64, size=40, scale=0.125)])
def test_windowed_attention_with_unit_queries_and_distance_penalty(seq, m):
    W, T = 48, 41
    w, h = att_weights(m, W, seed=3), rnd(T, W, seed=1)
    want = O.windowed_attention(n64(h), f64(w), m, EPS)
    mixer = make_att(m, w)
    for cuts in CUTS:
        close(run_mixer(seq, mixer, h, cuts), want, 2e-5, f"portions {cuts}")
    if m["mask"]["size"] > 4:                       # the penalty, and which head has which slope, show by far more than the tolerance
        keep = O.head_slopes
        try:
            O.head_slopes = lambda H: [0.0] * H
            differs(O.windowed_attention(n64(h), f64(w), m, EPS), want, 1e-2)
            if m["heads"] > 1:
                O.head_slopes = lambda H: keep(H)[::-1]
                differs(O.windowed_attention(n64(h), f64(w), m, EPS), want, 1e-2)
        finally:
            O.head_slopes = keep


@pytest.mark.parametrize("m", [latent(), latent(heads=2, dim=4, rot_dim=8, vdim=6, kv_rank=5, base=10000.0), latent(heads=9, dim=16, rot_dim=2, vdim=40, kv_rank=24),
                               latent(heads=1, dim=1, rot_dim=4, vdim=8, kv_rank=8), latent(heads=4, dim=8, rot_dim=16, vdim=1, kv_rank=70, scale=0.1),
                               latent(heads=17, dim=6, rot_dim=4, vdim=5, kv_rank=16, base=7.0)])
def test_latent_attention_with_a_gate_per_head(seq, m):
    W, T = 48, 41
    w, h = latent_weights(m, W, seed=7), rnd(T, W, seed=3)
    want = O.latent_attention(n64(h), f64(w), m, EPS)
    mixer = make_latent(m, w)
    for cuts in CUTS:
        close(run_mixer(seq, mixer, h, cuts), want, 3e-5, f"portions {cuts}")
    flat = dict(f64(w), g=np.zeros((m["heads"], W)))                # every gate one half
    differs(O.latent_attention(n64(h), flat, m, EPS), want, 1e-2)
    halves = dict(f64(w))
    halves["q"] = halves["q"][::-1]
    differs(O.latent_attention(n64(h), halves, m, EPS), want, 1e-2)


@pytest.mark.parametrize("T", [1, 3, 8, 9, 70, 200])
@pytest.mark.parametrize("m", [moe(), moe(experts=5, top=5, ff=17, shared_ff=0), moe(experts=9, top=1, ff=8, limit=2.0, shared_ff=24, shared_limit=0.4),
                               moe(experts=1, top=1, ff=3, shared_ff=1), moe(experts=70, top=7, ff=16, limit=0.3, shared_ff=16, shared_limit=5.0)])
def test_routed_experts_with_biased_choice_and_clamped_units(seq, m, T):
    from krasis_b200.mixers import RoutedExperts
    W, E = 48, m["router"]["experts"]
    w = {"router": rnd(E, W, seed=1, sd=W ** -0.5 * 2), "router.b": rnd(E, seed=2, sd=0.8)}
    for i, (p, F) in enumerate([(f"e{e}.", m["expert"]["ff"]) for e in range(E)] + ([("shared.", m["shared"]["ff"])] if "shared" in m else [])):
        w.update({p + "gate": rnd(F, W, seed=10 + 3 * i, sd=W ** -0.5 * 1.5), p + "up": rnd(F, W, seed=11 + 3 * i, sd=W ** -0.5 * 1.5),
                  p + "down": rnd(W, F, seed=12 + 3 * i, sd=F ** -0.5)})
    h = rnd(T, W, seed=5 + T)
    want = O.routed_experts(n64(h), f64(w), m)
    mlp = RoutedExperts(under(w), E, 0, m["router"]["top"], torch.float32, torch.device(DEV), score="top_softmax", act="clamped_swish",
                        limit=m["expert"]["limit"], alpha=1.702, shared_limit=(m.get("shared") or {}).get("limit"))
    close(mlp.forward(h.to(DEV)).cpu().numpy(), want, 1e-5, "experts")
    if T >= 70:                                     # limits and bias matter by far more than the tolerance
        differs(O.routed_experts(n64(h), f64(w), dict(m, expert=dict(m["expert"], limit=50.0))), want, 1e-3)
        if m["router"]["top"] > 1 or E > 1:
            differs(O.routed_experts(n64(h), dict(f64(w), **{"router.b": np.zeros(E)}), m), want, 1e-2)
        if "shared" in m:
            differs(O.routed_experts(n64(h), f64(w), dict(m, shared=dict(m["shared"], limit=m["shared"]["limit"] * 0.5))), want, 1e-4)


@pytest.mark.parametrize("E,top", [(8, 3), (5, 5), (1, 1), (100, 9)])
def test_router_choice_and_weights(seq, E, top):
    T = 37
    z, b = rnd(T, E, seed=1, sd=3.0), rnd(E, seed=2)
    ids, wts = seq.route(z.to(DEV), None, top, score="top_softmax", bias=b.to(DEV))
    for t in range(T):
        want = O.choose(n64(z[t]) + n64(b), top)
        assert ids[t].tolist() == [e for e, _ in want]
        close(wts[t].cpu().numpy(), np.array([p for _, p in want]), 1e-6, f"token {t}")
    # far below the range of exp the weights stay a softmax
    ids, wts = seq.route((z - 500.0).to(DEV), None, top, score="top_softmax", bias=b.to(DEV))
    close(wts.sum(1).cpu().numpy(), np.ones(T), 1e-6, "sums to one")
    # the other scores take the bias as well: softmax and sigmoid of the biased logits
    for score, fn in (("softmax", lambda v: O.softmax(v)), ("sigmoid", O.sigmoid)):
        ids, wts = seq.route(z.to(DEV), None, top, score=score, bias=b.to(DEV))
        for t in range(T):
            s = fn(n64(z[t]) + n64(b))
            close(wts[t].cpu().numpy(), s[ids[t].cpu().numpy()], 1e-5, score)


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 8, 32])
@pytest.mark.parametrize("W", [36, 37, 1, 2052])
def test_mixed_copies_of_the_stream(seq, n, W):
    T = 5
    x0, y = rnd(T, W, seed=1), rnd(T, W, seed=2)
    old, mix, out, read, nw = rnd(T, n, W, seed=3), rnd(n, n, seed=4), rnd(n, seed=5), rnd(n, seed=6), rnd(W, seed=7, sd=0.3)
    dev = lambda t: t.to(DEV).contiguous()
    cols = [n64(old[:, s]) for s in range(n)]
    # in the middle of the model: update, read, norm
    xs = dev(old)
    h = seq.stream_mix(xs, y=dev(y), mix=dev(mix), out=dev(out), read=dev(read), norm=dev(nw), w_shift=1.0, eps=EPS)
    new = O.write_streams(cols, n64(mix), n64(out), n64(y))
    close(xs.cpu().numpy(), np.stack(new, 1), 3e-6, "update")
    u = O.read_streams(new, n64(read))
    # where the read cancels (u far below the copies) the norm blows rounding up: bound the error in units of u's own size
    close(h.cpu().numpy(), O.offset_norm(u, n64(nw), EPS), 1e-4 if W == 1 else 1e-5, "norm of the read")
    # the beginning: every copy is x0; a bfloat16 result
    xs = torch.empty_like(xs)
    h = seq.stream_mix(xs, x0=dev(x0), read=dev(read), norm=dev(nw), w_shift=1.0, out_dtype=torch.bfloat16, eps=EPS)
    assert all(torch.equal(xs[:, s].cpu(), x0) for s in range(n))
    close(h.float().cpu().numpy(), O.offset_norm(O.read_streams([n64(x0)] * n, n64(read)), n64(nw), EPS), 8e-3, "start")
    # the end: the plain sum, and the sum without a norm
    xs = dev(old)
    h = seq.stream_mix(xs, norm=dev(nw), w_shift=1.0, eps=EPS)
    close(h.cpu().numpy(), O.offset_norm(sum(cols), n64(nw), EPS), 1e-4 if W == 1 else 1e-5, "norm of the sum")
    assert torch.equal(xs.cpu(), old)
    close(seq.stream_mix(xs).cpu().numpy(), sum(cols), 3e-6, "sum")


def aligned_inputs(T, W, d, marks, seed):
    """Hidden states for identity-like q / k projections onto the first d dimensions: the last position and the marked ones point in one
    direction there, all others in directions at right angles to it; the other W - d dimensions are random (they make the values)."""
    g = torch.Generator().manual_seed(seed)
    h = torch.randn(T, W, generator=g)
    u = torch.zeros(d)
    u[0] = 1.0
    h[:, 0] = 0.0
    for j in list(marks) + [T - 1]:
        h[j, :d] = 2.0 * u
    return h.to(torch.bfloat16).float()


def peaked_att(m, W, seed):
    H, d = m["heads"], m["dim"]
    w = att_weights(m, W, seed)
    eye = torch.zeros(d, W)
    eye[:, :d] = torch.eye(d)
    w["q"], w["k"] = eye.repeat(H, 1), eye.repeat(m["kv_heads"], 1)
    w["v"] = rnd(m["kv_heads"] * m["vdim"], W, seed=seed + 9, sd=1.0)
    w["v"][:, :d] = 0.0
    return w


@pytest.mark.parametrize("size,page,T", [(9, 4, 61), (16, 4, 50), (8, 8, 33), (5, 8, 30), (33, 8, 80), (1, 4, 20)])
def test_window_edges_with_peaked_scores(seq, size, page, T):
    """The last query scores the first and last position of its window, the one that has just left it, and the next ones on either side
    of a page border far above everything else; a window that is off by one moves the output by much more than the tolerance — in a
    prompt and when the last token is decoded alone."""
    W, d, i = 32, 8, T - 1
    m = att(heads=2, kv_heads=1, dim=d, vdim=6, size=size, scale=1.2)
    marks = {j for j in (i - 1, i - size + 1, i - size, i - size - 1, i // page * page - 1) if 0 <= j < i}
    w, h = peaked_att(m, W, seed=11), aligned_inputs(T, W, d, marks, seed=4)
    want = O.windowed_attention(n64(h), f64(w), m, EPS)
    for wrong in (size + 1, size - 1):
        if wrong > 0:
            off = O.windowed_attention(n64(h), f64(w), dict(m, mask={"size": wrong}), EPS)
            differs(off[i], want[i], 3e-2)
    mixer = make_att(m, w)
    for cuts in ([T], [T - 1], [T - 3, 2], [5, 2, 2, 9]):
        close(run_mixer(seq, mixer, h, cuts, page_size=page)[i], want[i], 3e-5, f"portions {cuts}")


@pytest.mark.parametrize("far", [0, 1, 3, 4, 63, 64, 297])
def test_far_latent_keys_with_peaked_scores(seq, far):
    """One key hundreds of positions back (the first tokens, either side of page borders) takes most of the weight of the last query; the
    unrotated part makes the peak, so it does not fade with the distance."""
    W, T = 40, 301
    m = latent(heads=2, dim=8, rot_dim=4, vdim=6, kv_rank=W - 4, scale=0.9)
    H, dn, dr, r = 2, 8, 4, W - 4
    w = latent_weights(m, W, seed=7)
    w["dkv"] = torch.zeros(r + dr, W)
    w["dkv"][:r, :r] = torch.eye(r)                       # the latent is the normed input itself
    w["dkv"][r:] = 0.02 * rnd(dr, W, seed=2)
    w["dkv.norm"] = torch.ones(r)
    w["uk"] = torch.zeros(H * dn, r)
    w["q"] = torch.zeros(H * (dn + dr), W)
    for a in range(H):
        w["uk"][a * dn:(a + 1) * dn, :dn] = torch.eye(dn)
        w["q"][a * (dn + dr), dn] = 1.0                   # the query asks along key dimension 0 with what stands in column dn of h
        w["q"][a * (dn + dr) + dn:(a + 1) * (dn + dr)] = 0.02 * rnd(dr, W, seed=3 + a)
    w["dkv"] = w["dkv"].to(torch.bfloat16).float()
    w["uv"][:, :dn] = 0.0
    h = rnd(T, W, seed=5)
    h[:, 0], h[:, dn] = 0.0, 0.0
    h[far, 0], h[T - 1, dn] = 6.0, 4.0
    want = O.latent_attention(n64(h), f64(w), m, EPS)
    lost = h.clone()
    lost[far, 0] = 0.0
    differs(O.latent_attention(n64(lost), f64(w), m, EPS)[T - 1], want[T - 1], 0.2)
    mixer = make_latent(m, w)
    for cuts, page in (([T], 4), ([T - 1], 64), ([100, 2, 150, 40], 4), ([T - 3], 8)):
        close(run_mixer(seq, mixer, h, cuts, page_size=page)[T - 1], want[T - 1], 3e-5, f"portions {cuts}")


# ------------------------------------------------------------------------------------------------ the model through the scheduler
def test_prefill_against_the_oracle_layer_by_layer(seq):
    raw = default_cfg()
    model, w = build(raw, seed=1, page_size=4)
    tk = toks(75, raw["vocab"], 3)
    trace = []
    want = O.forward(raw, w, tk, trace)
    model.layer_trace = []
    got = run_portions(model, tk, [75])
    assert len(model.layer_trace) == len(trace) == 8
    for i, (a, b) in enumerate(zip(model.layer_trace, trace)):
        close(a.cpu().numpy(), b, 3e-5, f"sum of the copies after layer run {i}")
    model.layer_trace = None
    close(got, want, 5e-5, "logits")


def test_decoding_and_portions_equal_prefill(seq):
    raw = default_cfg()
    model, w = build(raw, seed=2, page_size=4)
    tk = toks(70, raw["vocab"], 4)
    want = O.forward(raw, w, tk)
    for cuts in ([], [2] * 35, [2, 3, 4, 5, 6, 7, 8, 9], [33, 2, 2, 31], [69]):
        close(run_portions(model, tk, cuts), want, 5e-5, f"portions {cuts}")


@pytest.mark.parametrize("streams", [1, 2, 4, 7])
def test_numbers_of_stream_copies(seq, streams):
    raw = default_cfg(streams=streams)
    model, w = build(raw, seed=12, page_size=4)
    tk = toks(40, raw["vocab"], 5)
    want = O.forward(raw, w, tk)
    for cuts in ([40], [20, 2]):
        close(run_portions(model, tk, cuts), want, 5e-5, f"portions {cuts}")


@pytest.mark.parametrize("loop", [None, (0, 1, 3), (0, 5, 2), (4, 5, 4), (2, 2, 5), (1, 3, 1)])
def test_looped_spans(seq, loop):
    """No span, the first layer, all layers, the last layer, an empty span, a span that runs once; every run has a cache of its own."""
    raw = default_cfg(loop=loop)
    model, w = build(raw, seed=13, page_size=4)
    tk = toks(30, raw["vocab"], 6)
    want = O.forward(raw, w, tk)
    model.layer_trace = []
    for cuts in ([30], [11, 2, 2]):
        close(run_portions(model, tk, cuts), want, 5e-5, f"portions {cuts}")
    assert model.kv_cache.num_layers == len(O.layer_order(5, raw.get("loop")))


def test_first_tokens_of_a_sequence(seq):
    raw = default_cfg()
    model, w = build(raw, seed=3, page_size=4)
    for n in (1, 2, 3):
        tk = toks(n, raw["vocab"], 20 + n)
        want = O.forward(raw, w, tk)
        close(run_portions(model, tk, [n]), want, 5e-5, f"{n} tokens at once")
        close(run_portions(model, tk, []), want, 5e-5, f"{n} tokens one by one")


def test_unequal_requests_in_one_batch_equal_each_alone(seq):
    raw = default_cfg()
    model, w = build(raw, seed=4, page_size=4)
    a, b, c = toks(50, 50, 5), toks(23, 50, 6), toks(9, 50, 7)
    want = {k: O.forward(raw, w, v) for k, v in (("a", a), ("b", b), ("c", c))}
    s = sched(model, max_tokens=256)
    got = {"a": [], "b": [], "c": []}

    def step(*parts):
        out = s.step([(rid, t, list(range(len(t)))) for rid, t in parts]).cpu().numpy()
        at = 0
        for rid, t in parts:
            got[rid].append(out[at:at + len(t)])
            at += len(t)
    step(("a", a[:30]), ("b", b[:2]))
    step(("b", b[2:4]), ("a", a[30:31]), ("c", c[:7]))
    step(("c", c[7:8]), ("a", a[31:32]), ("b", b[4:21]))
    step(("a", a[32:]), ("c", c[8:]))
    step(("b", b[21:]),)
    for k in got:
        close(np.concatenate(got[k], 0), want[k], 5e-5, f"request {k}")


def test_pages_and_slots_are_reused(seq):
    """A pool of a few pages and two slots serves five requests one after another and two at a time; what a finished request left in its
    pages must not reach the next one."""
    raw = default_cfg()
    model, w = build(raw, seed=5, page_size=4)
    s = sched(model, max_tokens=64, max_requests=2)
    reqs = [toks(n, 50, 30 + n) for n in (29, 31, 14, 30, 7)]
    for i, tk in enumerate(reqs):
        close(run_portions(model, tk, [len(tk) // 2, 2], s=s, rid=i), O.forward(raw, w, tk), 5e-5, f"request {i}")
        assert s.kv_cache.free_page_count == 16 and s.state_pool.free_slot_count == 2
    x, y = reqs[2], reqs[4]
    out = s.step([("x", x, [len(x) - 1]), ("y", y, [len(y) - 1])]).cpu().numpy()
    close(out[0], O.forward(raw, w, x)[-1], 5e-5, "two at a time, first")
    close(out[1], O.forward(raw, w, y)[-1], 5e-5, "two at a time, second")


def test_long_decoding(seq):
    raw = model_cfg([AT(att(size=20)), LA(mlp=None)], loop=(0, 2, 2))
    model, w = build(raw, seed=6)
    tk = toks(330, raw["vocab"], 8)
    want = O.forward(raw, w, tk)
    got = run_portions(model, tk, [10])                     # 320 tokens decoded one by one, across five pages of 64
    close(got, want, 1e-4, "330 tokens")
    close(got[-1], want[-1], 1e-4, "the last token")


def test_bfloat16_serving_stays_near_the_oracle(seq):
    """Every position bounded where each token uses every expert; the median where rounding can turn a close choice of experts."""
    every = [LA(mlp=moe(experts=4, top=4)), AT(mlp=moe(experts=3, top=3, shared_ff=0)), AT(mlp=None)]
    for raw, quantile in ((model_cfg(every, loop=(0, 2, 2)), 0.9), (default_cfg(), 0.5)):
        model, w = build(raw, dtype=torch.bfloat16, seed=7, page_size=8)
        tk = toks(90, raw["vocab"], 9)
        want = O.forward(raw, w, tk)
        for got, what in ((run_portions(model, tk, [90]), "prefill"), (run_portions(model, tk, [40, 2, 17]), "portions and decoding")):
            err = np.abs(got.astype(np.float64) - want).max(-1) / np.abs(want).max()
            assert np.quantile(err, quantile) <= 4e-2, f"{what}: {np.quantile(err, quantile):.3e}"


def test_other_sizes_than_any_shipped_model(seq):
    """Every size that tends to coincide in shipped configurations is made different here, or 1: one head, a latent larger than the width,
    a window of one, one expert, a shared expert of one unit, no feed-forward at all, odd widths."""
    layers = [LA(latent(heads=1, dim=2, rot_dim=2, vdim=3, kv_rank=30), mlp=None), AT(att(heads=1, kv_heads=1, dim=2, vdim=5, size=1), mlp=None),
              AT(att(heads=5, kv_heads=5, dim=7, vdim=9, size=2), moe(experts=1, top=1, ff=1, limit=0.2, shared_ff=1, shared_limit=9.0)),
              LA(latent(heads=6, dim=5, rot_dim=10, vdim=1, kv_rank=3, base=1.5), moe(experts=7, top=6, ff=31, shared_ff=0)),
              AT(att(heads=6, kv_heads=2, dim=4, vdim=8, size=300), moe(experts=2, top=1, ff=5, shared_ff=64))]
    raw = model_cfg(layers, width=23, vocab=13, streams=5, loop=(3, 5, 3), eps=3e-4)
    model, w = build(raw, seed=8, page_size=4)
    tk = toks(45, 13, 10)
    want = O.forward(raw, w, tk)
    for cuts in ([45], [], [7, 2, 2]):
        close(run_portions(model, tk, cuts), want, 5e-5, f"portions {cuts}")


def test_greedy_generation_through_the_entry_point(seq):
    """Scheduler.generate (admission, portions under a token budget, decode beside prefill, slot and page reuse) against greedy
    decoding with the oracle.  Steps whose two best logits are closer than the comparison tolerance end the comparison of a prompt."""
    raw = default_cfg()
    model, w = build(raw, seed=9, page_size=4)
    prompts = [toks(n, 50, 50 + n) for n in (19, 3, 33, 8, 1, 12)]
    s = sched(model, max_tokens=160, max_requests=3)
    outs = s.generate(prompts, max_new_tokens=12, step_tokens=16)
    assert s.kv_cache.free_page_count == 40 and s.state_pool.free_slot_count == 3 and not s.live
    checked = 0
    for p, out in zip(prompts, outs):
        assert len(out) == 12
        seqn = list(p)
        for tok in out:
            lg = O.forward(raw, w, seqn)[-1]
            top = np.sort(lg)[-2:]
            if top[1] - top[0] < 1e-3 * np.abs(lg).max():
                break
            assert tok == int(np.argmax(lg))
            seqn.append(tok)
            checked += 1
    assert checked >= 40


def test_decode_steps_replayed_from_cuda_graphs_equal_eager_steps(seq):
    raw = default_cfg()
    model, w = build(raw, seed=17, page_size=4)
    a, b = toks(70, 50, 1), toks(60, 50, 2)
    outs = []
    for graphs in (False, True):
        s = sched(model, max_tokens=512, max_requests=3, cuda_graphs=graphs)
        got = [s.step([("a", a[:20], [19]), ("b", b[:5], [4])])]
        for i in range(40):
            got.append(s.step([("a", [a[20 + i]], [0]), ("b", [b[5 + i]], [0])]))
        s.finish("b")
        for i in range(8):
            got.append(s.step([("a", [a[60 + i]], [0])]))
        outs.append([g.clone() for g in got])
        if graphs:
            assert sum(1 for v in s._graphs.values() if v) >= 2
    for x, y in zip(*outs):
        close(y.cpu().numpy(), n64(x.cpu()), 1e-5, "graph against eager")
    close(outs[1][-1][0].cpu().numpy(), O.forward(raw, w, a[:68])[67], 5e-5, "last decoded token of request a")


def test_registry_loads_a_checkpoint_directory_and_the_trace_runner_replays_it(seq, tmp_path, monkeypatch, capsys):
    import io
    import sys
    from krasis_b200 import trace_runner
    from krasis_b200.kugalorn import KugalornConfig, random_weights
    from krasis_b200.registry import architecture_of, load_model
    raw = default_cfg()
    w = random_weights(KugalornConfig.from_dict(raw), 10)
    header, blobs, off = {}, [], 0
    for k, v in w.items():
        b = v.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        header[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    hj = json.dumps(header).encode()
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    assert architecture_of(str(tmp_path)) == "Kugalorn"
    tk = toks(25, 50, 14)
    want = O.forward(raw, f64(w), tk)
    close(run_portions(load_model(str(tmp_path), dtype=torch.float32), tk, [25]), want, 5e-5, "loaded checkpoint")
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tk[:10], "want": [0, 9]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tk[10:12], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": tk[12:], "want": [12]}, {"id": "y", "tokens": tk[:3], "want": [2]}], "end": ["x", "y"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    out = tmp_path / "out"
    assert trace_runner.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"]) == 0
    assert [ln for ln in capsys.readouterr().out.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "1.f32").exists()
    close(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1), want[[0, 9]], 5e-5, "step 0")
    close(np.fromfile(out / "2.f32", dtype="<f4").reshape(2, -1), want[[24, 2]], 5e-5, "step 2")


# ------------------------------------------------------------------------------------------------ long bfloat16 portions on the tensor cores
def test_tensor_core_attention_with_distance_penalty(seq):
    """128 query / key dims and 128 or 256 value dims: portions of 128 tokens or more run the tcgen05 attention core with the penalty inside
    it.  Peaked scores on the window's edges; against the oracle and against the plain kernels on the same bf16 cache."""
    from krasis_b200.build import build as build_core
    build_core()
    W, d, T = 192, 128, 400
    i = T - 1
    for heads, kv_heads, vdim, size in ((2, 1, 128, 100), (4, 2, 256, 64), (16, 4, 128, 37)):
        m = att(heads=heads, kv_heads=kv_heads, dim=d, vdim=vdim, size=size, scale=0.06)
        w = peaked_att(m, W, seed=21)
        h = aligned_inputs(T, W, d, {i - 1, i - size + 1, i - size, i - size - 1, 200}, seed=6)
        want = O.windowed_attention(n64(h), f64(w), m, EPS)
        for wrong in (size - 1, size + 1):
            differs(O.windowed_attention(n64(h), f64(w), dict(m, mask={"size": wrong}), EPS)[i], want[i], 0.1)
        keep = O.head_slopes
        try:
            O.head_slopes = lambda H: [0.0] * H
            differs(O.windowed_attention(n64(h), f64(w), m, EPS), want, 0.1)
        finally:
            O.head_slopes = keep
        mixer = make_att(m, w, torch.bfloat16)
        assert mixer.tc_shape
        fast = run_mixer(seq, mixer, h, [T], page_size=8)
        parts = run_mixer(seq, mixer, h, [130, 2, T - 132], page_size=8)
        mixer.tc_min_portion = 1 << 30
        plain = run_mixer(seq, mixer, h, [T], page_size=8)
        for got, what in ((plain, "plain kernels"), (fast, "tensor-core prefill"), (parts, "tensor-core portions")):
            err = np.abs(got.astype(np.float64) - want).max(-1) / np.abs(want).max()
            assert err.max() <= 2e-2, f"{heads} heads, {what}: {err.max():.3e} at {err.argmax()}"
        close(fast, plain.astype(np.float64), 1e-2, "tensor core against plain kernels")


def test_tensor_core_latent_attention_with_a_gate_per_head(seq):
    from krasis_b200.build import build as build_core
    build_core()
    W, T = 128, 330
    for heads in (2, 5):
        m = latent(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=64, base=10000.0, scale=0.07)
        w, h = latent_weights(m, W, seed=9), rnd(T, W, seed=4)
        want = O.latent_attention(n64(h), f64(w), m, EPS)
        differs(O.latent_attention(n64(h), dict(f64(w), g=np.zeros((heads, W))), m, EPS), want, 0.1)
        mixer = make_latent(m, w, torch.bfloat16)
        assert mixer.tc_shape
        fast, parts = run_mixer(seq, mixer, h, [T]), run_mixer(seq, mixer, h, [130, 2, T - 132])
        mixer.tc_min_portion = 1 << 30
        plain = run_mixer(seq, mixer, h, [T])
        for got, what in ((plain, "plain kernels"), (fast, "tensor-core prefill"), (parts, "tensor-core portions")):
            err = np.abs(got.astype(np.float64) - want).max(-1) / np.abs(want).max()
            assert np.quantile(err, 0.95) <= 3e-2, f"{what}: {np.quantile(err, 0.95):.3e}"


def test_tensor_core_prefill_of_the_whole_model(seq):
    from krasis_b200.build import build as build_core
    build_core()
    every = lambda **kw: moe(experts=4, top=4, ff=64, shared_ff=128, **kw)      # every expert runs: no close choice turns by rounding
    layers = [AT(att(heads=4, kv_heads=2, dim=128, vdim=128, size=200, scale=0.08), every()),
              LA(latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=64, base=10000.0, scale=0.07), every(limit=1.5)),
              AT(att(heads=2, kv_heads=1, dim=128, vdim=256, size=70, scale=0.08), None)]
    raw = model_cfg(layers, width=128, streams=4, loop=(0, 2, 2))
    model, w = build(raw, dtype=torch.bfloat16, seed=31)
    assert all(lay["mixer"].tc_shape for lay in model.layers)
    tk = toks(520, raw["vocab"], 16)
    want = O.forward(raw, w, tk)

    def most(got, ref, rel, what):
        err = np.abs(got.astype(np.float64) - ref).max(-1) / np.abs(ref).max()
        assert np.quantile(err, 0.9) <= rel, f"{what}: {np.quantile(err, 0.9):.3e}"
    whole = run_portions(model, tk, [520], s=sched(model, 1024))
    parts = run_portions(model, tk, [130, 257, 128], s=sched(model, 1024))
    for lay in model.layers:
        lay["mixer"].tc_min_portion = 1 << 30
    plain = run_portions(model, tk, [520], s=sched(model, 1024))
    most(plain, want, 4e-2, "plain kernels against the oracle")
    most(whole, want, 4e-2, "tensor-core prefill against the oracle")
    most(whole, plain.astype(np.float64), 3e-2, "tensor-core prefill against the plain kernels")
    most(parts, plain.astype(np.float64), 3e-2, "tensor-core portions against the plain kernels")
