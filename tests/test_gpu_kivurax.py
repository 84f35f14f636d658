"""Kivurax on the GPU against the plain float64 oracle (tests/oracle_kivurax.py): each mechanism alone, then the whole model through the
scheduler — prefill against decoding, portions down to two tokens, unequal batches, reuse of pages and slots, far tokens kept by the
recurrent states, page borders and window edges with peaked scores, the first tokens of a sequence, long decoding, odd sizes, and greedy
generation through the generation entry point.  Small random configurations made here; none of them is a shipped model's."""
import json
import struct

import numpy as np
import pytest
import torch

from tests import oracle_kivurax as O

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
def mem(heads=3, dim=12, vdim=10, gate_cap=6.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def dlt(heads=4, kv_heads=2, dim=12, vdim=10, conv=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


YARN = {"factor": 8.0, "original": 64, "fast": 4.0, "slow": 1.0}


def att(heads=4, kv_heads=2, dim=12, size=9, scale=0.3, dims=8, base=100.0, scaling=YARN):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": size},
            "rot": {"base": base, "dims": dims, "scaling": scaling}}


def rec(width=24, blocks=3, conv=4):
    return {"width": width, "blocks": blocks, "conv": conv}


def par(left=None, right=None, left_scale=0.6, right_scale=1.3):
    return {"left": left or att(), "right": right or rec(), "left_scale": left_scale, "right_scale": right_scale}


def dense(ff=28):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=20):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def ME(m=None, mlp=None):
    return {"type": "mlstm", "mixer": m or mem(), "mlp": mlp}


def DE(m=None, mlp=None):
    return {"type": "delta", "mixer": m or dlt(), "mlp": mlp}


def PA(m=None, mlp=None):
    return {"type": "parallel", "mixer": m or par(), "mlp": mlp}


def model_cfg(layers, width=40, vocab=50, eps=EPS, m=0.7):
    return {"architecture": "Kivurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": m, "layers": layers}


def default_cfg(**kw):
    return model_cfg([PA(mlp=moe()), ME(mlp=dense()), DE(mlp=moe(experts=5, top=1, ff=17)), ME(mem(heads=2, dim=32, vdim=64, gate_cap=3.0)),
                      PA(par(att(heads=6, kv_heads=6, dim=8, size=30, dims=4, scaling=None), rec(width=33, blocks=1, conv=2), 1.1, 0.4), dense(9)),
                      DE(dlt(heads=3, kv_heads=3, dim=32, vdim=32, conv=4), moe(experts=4, top=4, ff=8))], **kw)


def build(raw, dtype=torch.float32, seed=0, page_size=None, tweak=None):
    from krasis_b200.kivurax import KivuraxConfig, KivuraxModel, random_weights
    cfg = KivuraxConfig.from_dict(raw)
    w = random_weights(cfg, seed)
    if tweak:
        tweak(w)
    model = KivuraxModel(cfg, w, dtype=dtype)
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


def rows_within(got, want, rel, what, quantile=1.0):
    err = np.abs(got.astype(np.float64) - want).max(-1) / np.abs(want).max()
    assert np.quantile(err, quantile) <= rel, f"{what}: {np.quantile(err, quantile):.3e} at {err.argmax()}"


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


def bf(t):
    return t.to(torch.bfloat16).float()


def f64(d):
    return {k: v.numpy().astype(np.float64) for k, v in d.items()}


def n64(t):
    return t.numpy().astype(np.float64)


def under(d):
    return {k.replace(".", "_"): v for k, v in d.items()}


# ------------------------------------------------------------------------------------------------ mixers alone: weights and runs
def mem_weights(m, W, seed, forget=2.0):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    n = lambda rows, k: rnd(rows, W, seed=seed + k, sd=W ** -0.5)
    return {"q": n(H * d, 0), "k": n(H * d, 1), "v": n(H * dv, 2), "g": n(H * dv, 3), "i": 2 * n(H, 4), "f": 2 * n(H, 5), "i.b": rnd(H, seed=seed + 6),
            "f.b": bf(rnd(H, seed=seed + 7) + forget), "norm": bf(1 + rnd(H * dv, seed=seed + 8, sd=0.2)), "o": rnd(W, H * dv, seed=seed + 9, sd=0.2)}


def make_mem(m, w, dtype=torch.float32):
    from krasis_b200.mixers import MatrixMemory
    return MatrixMemory(under(w), m["heads"], m["dim"], m["vdim"], m["gate_cap"], EPS, dtype, torch.device(DEV))


def dlt_weights(m, W, seed, dt=-1.0):
    H, G, d, dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    w = {}
    for i, (nm, rows) in enumerate((("q", G * d), ("k", G * d), ("v", H * dv))):
        w[nm], w[nm + ".conv"] = rnd(rows, W, seed=seed + i, sd=W ** -0.5), rnd(rows, K, seed=seed + 3 + i, sd=0.6)
    w.update({"g": rnd(H * dv, W, seed=seed + 6, sd=W ** -0.5), "a": rnd(H, W, seed=seed + 7, sd=W ** -0.5), "b": rnd(H, W, seed=seed + 8, sd=W ** -0.5),
              "A_log": rnd(H, seed=seed + 9, sd=0.5), "dt_bias": bf(rnd(H, seed=seed + 10) + dt), "norm": bf(1 + rnd(dv, seed=seed + 11, sd=0.2)),
              "o": rnd(W, H * dv, seed=seed + 12, sd=0.2)})
    return w


def make_dlt(m, w, dtype=torch.float32):
    from krasis_b200.mixers import GatedDeltaMixer
    return GatedDeltaMixer(under(w), m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], EPS, dtype, torch.device(DEV))


def att_weights(m, W, seed):
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    return {"q": rnd(H * d, W, seed=seed, sd=W ** -0.5), "k": rnd(G * d, W, seed=seed + 1, sd=W ** -0.5), "q.norm": bf(1 + rnd(d, seed=seed + 2, sd=0.3)),
            "k.norm": bf(1 + rnd(d, seed=seed + 3, sd=0.3)), "o": rnd(W, H * d, seed=seed + 4, sd=0.2)}


def make_att(m, w, dtype=torch.float32):
    from krasis_b200.mixers import MultiMapAttention, yarn_table
    freq, amp = yarn_table(m["rot"]["dims"], m["rot"]["base"], m["rot"]["scaling"])
    return MultiMapAttention(under(w), m["heads"], m["kv_heads"], 1, m["dim"], m["vdim"], m["scale"], EPS, dtype, torch.device(DEV),
                             window=m["mask"]["size"], rot_dims=m["rot"]["dims"], rot_freq=freq, rot_amp=amp, keys_as_values=True, off_by_one=True)


def rec_weights(m, W, seed, lam=-1.0):
    C, B, K = m["width"], m["blocks"], m["conv"]
    n = C // B
    return {"x": rnd(C, W, seed=seed, sd=W ** -0.5), "x.b": rnd(C, seed=seed + 1, sd=0.5), "y": rnd(C, W, seed=seed + 2, sd=W ** -0.5), "y.b": rnd(C, seed=seed + 3, sd=0.5),
            "conv": rnd(C, K, seed=seed + 4, sd=0.6), "conv.b": rnd(C, seed=seed + 5, sd=0.5), "ra": rnd(B, n, n, seed=seed + 6, sd=n ** -0.5),
            "ra.b": rnd(B, n, seed=seed + 7), "ri": rnd(B, n, n, seed=seed + 8, sd=n ** -0.5), "ri.b": rnd(B, n, seed=seed + 9),
            "lam": bf(rnd(C, seed=seed + 10) + lam), "o": rnd(W, C, seed=seed + 11, sd=0.2)}


def make_rec(m, w, dtype=torch.float32):
    from krasis_b200.mixers import GatedRecurrentUnit
    return GatedRecurrentUnit(under(w), m["width"], m["blocks"], m["conv"], dtype, torch.device(DEV))


def run_attention(seq, mixer, h, cuts, page_size=4):
    """One sequence through an attention mixer with a paged cache of its own, in portions (the rest one by one)."""
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


def run_recurrent(seq, mixer, h, cuts):
    """One sequence through a mixer with state slots: slot 1 of 3, the neighbours filled with numbers that must neither be read nor change."""
    from krasis_b200.attention import RecurrentStatePool
    pool = RecurrentStatePool(3, DEV)
    states = mixer.register_state(pool)
    for t in states:
        t[0], t[2] = 7.0, -3.0
    out, at, T = [], 0, h.shape[0]
    for n in list(cuts) + [1] * (T - sum(cuts)):
        tb = seq.StepTables([([0] * n, at, 1, [0])], torch.device(DEV))
        out.append(mixer.forward(h[at:at + n].to(DEV, mixer.dtype).contiguous(), tb, *states).cpu().numpy())
        at += n
    assert all(bool((t[0] == 7.0).all()) and bool((t[2] == -3.0).all()) for t in states)
    return np.concatenate(out, 0)


CUTS = ([41], [], [2, 2, 5, 17], [30, 2], [3, 1, 1, 9, 2])


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("m", [mem(), mem(heads=2, dim=32, vdim=32, gate_cap=2.0), mem(heads=1, dim=64, vdim=96), mem(heads=2, dim=128, vdim=64, gate_cap=15.0),
                               mem(heads=1, dim=256, vdim=32), mem(heads=5, dim=1, vdim=1), mem(heads=2, dim=70, vdim=130), mem(heads=2, dim=32, vdim=33),
                               mem(heads=3, dim=8, vdim=300, gate_cap=0.5), mem(heads=1, dim=520, vdim=7)])
def test_matrix_memory(seq, m, monkeypatch):
    W, T = 48, 41
    w, h = mem_weights(m, W, seed=3), rnd(T, W, seed=1)
    want = O.matrix_memory(n64(h), f64(w), m, EPS)
    mixer = make_mem(m, w)
    for cuts in CUTS:
        close(run_recurrent(seq, mixer, h, cuts), want, 3e-5, f"portions {cuts}")
    # the cap, the floor of the divisor and the forget gate show by far more than the tolerance
    differs(O.matrix_memory(n64(h), f64(w), dict(m, gate_cap=m["gate_cap"] * 3), EPS), want, 1e-3)
    differs(O.matrix_memory(n64(h), dict(f64(w), **{"f.b": np.full(m["heads"], 40.0)}), m, EPS), want, 1e-3)
    if m["vdim"] == 1:
        return
    # (a factor of a head's read-out is lost in its unit norm up to eps: the floor shows where read-outs are small)
    small = dict(w, v=0.002 * w["v"])
    want = O.matrix_memory(n64(h), f64(small), m, EPS)
    close(run_recurrent(seq, make_mem(m, small), h, [20, 2, 9]), want, 3e-5, "small read-outs")
    monkeypatch.setattr(O, "memory_read", lambda S, n, q, mm: S.T @ q / (abs(n @ q) + 1e-6))
    differs(O.matrix_memory(n64(h), f64(small), m, EPS), want, 1e-2)


def test_matrix_memory_gates_over_a_long_portion(seq):
    """More tokens than the gate kernel's block has threads; the maximum falls over hundreds of tokens and jumps back."""
    m, W, T = mem(heads=2, dim=8, vdim=6, gate_cap=20.0), 16, 2300
    w, h = mem_weights(m, W, seed=5, forget=-1.0), rnd(T, W, seed=2)
    w["i"] = 4 * w["i"]
    want = O.matrix_memory(n64(h), f64(w), m, EPS)
    mixer = make_mem(m, w)
    for cuts in ([T], [1024, 2, 1025, 249], [1000, 1300]):
        got = run_recurrent(seq, mixer, h, cuts)
        close(got, want, 1e-3, f"portions {cuts}")            # a read-out that cancels shows the fp32 state's own rounding
        rows_within(got, want, 1e-5, f"portions {cuts}", 0.999)


@pytest.mark.parametrize("m", [dlt(), dlt(heads=6, kv_heads=2, dim=32, vdim=64, conv=4), dlt(heads=2, kv_heads=2, dim=7, vdim=9, conv=1),
                               dlt(heads=4, kv_heads=1, dim=64, vdim=32, conv=2), dlt(heads=1, kv_heads=1, dim=16, vdim=40, conv=6)])
def test_gated_delta_rule(seq, m):
    W, T = 48, 41
    w, h = dlt_weights(m, W, seed=3), rnd(T, W, seed=1)
    want = O.delta_rule(n64(h), f64(w), m, EPS)
    mixer = make_dlt(m, w)
    for cuts in CUTS:
        close(run_recurrent(seq, mixer, h, cuts), want, 3e-5, f"portions {cuts}")
    differs(O.delta_rule(n64(h), dict(f64(w), dt_bias=n64(w["dt_bias"]) - 3), m, EPS), want, 1e-2)


@pytest.mark.parametrize("m", [att(), att(heads=2, kv_heads=2, dim=32, size=5, dims=32), att(heads=8, kv_heads=1, dim=6, size=12, dims=2, base=10000.0),
                               att(heads=3, kv_heads=3, dim=10, size=100, scale=0.7, scaling=None), att(heads=5, kv_heads=1, dim=16, size=1, dims=12),
                               att(heads=1, kv_heads=1, dim=4, size=41, dims=4, scaling={"factor": 32.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                               att(heads=12, kv_heads=4, dim=64, size=40, scale=0.1, dims=48, base=50.0)])
def test_attention_whose_values_are_the_projected_keys(seq, m, monkeypatch):
    W, T = 48, 41
    w, h = att_weights(m, W, seed=3), rnd(T, W, seed=1)
    want = O.key_value_attention(n64(h), f64(w), m, EPS)
    mixer = make_att(m, w)
    for cuts in CUTS:
        close(run_attention(seq, mixer, h, cuts), want, 3e-5, f"portions {cuts}")
    if m["rot"]["scaling"]:                         # frequencies and amplitude of the scaled rotation
        if m["mask"]["size"] > 1:
            differs(O.key_value_attention(n64(h), f64(w), dict(m, rot=dict(m["rot"], scaling=None)), EPS), want, 1e-3)
        keep = O.pair_frequencies
        monkeypatch.setattr(O, "pair_frequencies", lambda rot: (keep(rot)[0], 1.0))
        differs(O.key_value_attention(n64(h), f64(w), m, EPS), want, 1e-3)
    monkeypatch.undo()
    monkeypatch.setattr(O, "softmax_plus_one", lambda s: np.exp(s - s.max()) / np.exp(s - s.max()).sum())
    differs(O.key_value_attention(n64(h), f64(w), m, EPS), want, 1e-2)


@pytest.mark.parametrize("m", [rec(), rec(width=33, blocks=1, conv=1), rec(width=64, blocks=2, conv=2), rec(width=70, blocks=70, conv=4), rec(width=1, blocks=1, conv=3),
                               rec(width=96, blocks=4, conv=9), rec(width=160, blocks=5, conv=3)])
def test_recurrent_block(seq, m):
    W, T = 48, 150
    w, h = rec_weights(m, W, seed=3), rnd(T, W, seed=1)
    want = O.recurrent_block(n64(h), f64(w), m)
    mixer = make_rec(m, w)
    for cuts in ([T], [], [2, 2, 5, 65], [64, 2], [63, 1, 66, 2]):
        close(run_recurrent(seq, mixer, h, cuts), want, 2e-5, f"portions {cuts}")
    for name in ("x.b", "y.b", "conv.b", "ra.b", "ri.b"):
        differs(O.recurrent_block(n64(h), dict(f64(w), **{name: 0.0 * n64(w[name])}), m), want, 1e-3)


@pytest.mark.parametrize("T", [1, 3, 8, 9, 70, 200])
@pytest.mark.parametrize("m", [moe(), moe(experts=5, top=5, ff=17), moe(experts=9, top=1, ff=8), moe(experts=1, top=1, ff=3), moe(experts=70, top=7, ff=16)])
def test_routed_experts_with_weights_on_their_inputs(seq, m, T):
    from krasis_b200.mixers import RoutedExperts
    W, E, F = 48, m["router"]["experts"], m["expert"]["ff"]
    w = {"router": rnd(E, W, seed=1, sd=W ** -0.5 * 2)}
    for e in range(E):
        w.update({f"e{e}.gate": rnd(F, W, seed=10 + 3 * e, sd=W ** -0.5 * 1.5), f"e{e}.up": rnd(F, W, seed=11 + 3 * e, sd=W ** -0.5 * 1.5),
                  f"e{e}.down": rnd(W, F, seed=12 + 3 * e, sd=F ** -0.5)})
    h = rnd(T, W, seed=5 + T)
    want = O.routed_experts(n64(h), f64(w), m)
    mlp = RoutedExperts(under(w), E, 0, m["router"]["top"], torch.float32, torch.device(DEV), score="sigmoid", act="silu", weight_input=True)
    close(mlp.forward(h.to(DEV)).cpu().numpy(), want, 1e-5, "experts")
    # the same weights on the outputs are something else
    outputs = np.zeros_like(want)
    for t in range(T):
        for e, p in O.choose(n64(h[t]) @ n64(w["router"]).T, m["router"]["top"]):
            outputs[t] += p * O.expert(n64(h[t]), O.sub(f64(w), f"e{e}."))
    differs(outputs, want, 1e-3)
    other = RoutedExperts(under(w), E, 0, m["router"]["top"], torch.float32, torch.device(DEV), score="sigmoid", act="silu")
    close(other.forward(h.to(DEV)).cpu().numpy(), outputs, 1e-5, "weights on the outputs")


@pytest.mark.parametrize("T", [1, 7, 40])
@pytest.mark.parametrize("ff", [1, 28, 33])
def test_dense_unit_with_biases(seq, T, ff):
    from krasis_b200.mixers import GatedMLP
    W = 40
    w = {"gate": rnd(ff, W, seed=1, sd=W ** -0.5), "up": rnd(ff, W, seed=2, sd=W ** -0.5), "down": rnd(W, ff, seed=3, sd=ff ** -0.5), "gate.b": rnd(ff, seed=4),
         "up.b": rnd(ff, seed=5), "down.b": rnd(W, seed=6)}
    h, want = rnd(T, W, seed=7), None
    want = O.dense(n64(h), f64(w))
    mlp = GatedMLP(under(w), torch.float32, torch.device(DEV), act="silu")
    close((mlp.forward(h.to(DEV)) + mlp.out_bias).cpu().numpy(), want, 1e-5, "dense")
    for name in ("gate.b", "up.b", "down.b"):
        differs(O.dense(n64(h), dict(f64(w), **{name: 0.0 * n64(w[name])})), want, 1e-3)
    half = GatedMLP(under(w), torch.bfloat16, torch.device(DEV), act="silu")             # bf16 in and out: vector and scalar forms of the pass
    close((half.forward(h.to(DEV, torch.bfloat16)) + half.out_bias).cpu().numpy(), want, 2e-2, "bf16")


@pytest.mark.parametrize("W", [36, 37, 1, 2052])
def test_norm_on_the_output_only(seq, W):
    T, m, c = 5, 0.3, (0.8, -1.1)
    x, y, z, b, nw, fw = rnd(T, W, seed=1), rnd(T, W, seed=2), rnd(T, W, seed=3), rnd(W, seed=4), rnd(W, seed=5), rnd(W, seed=6)
    dev = lambda t: t.to(DEV).contiguous()
    both = c[0] * n64(y) + c[1] * n64(z) + n64(b)
    new = n64(x) + m * O.norm(both, n64(nw), EPS)
    xs = dev(x)
    h = seq.residual_post_rms(xs, dev(y), dev(nw), m, y2=dev(z), coefs=c, bias=dev(b), out_dtype=torch.bfloat16, eps=EPS)
    close(xs.cpu().numpy(), new, 3e-6, "two terms and a bias")
    assert torch.equal(h.cpu(), xs.cpu().to(torch.bfloat16))
    xs = dev(x)
    h = seq.residual_post_rms(xs, dev(y), dev(nw), m, out_norm=dev(fw), out_dtype=torch.float32, eps=EPS)
    new = n64(x) + m * O.norm(n64(y), n64(nw), EPS)
    close(xs.cpu().numpy(), new, 3e-6, "one term")
    close(h.cpu().numpy(), O.norm(new, n64(fw), EPS), 1e-4 if W == 1 else 1e-5, "norm of the new stream")
    # nothing to add: the stream rounded, or itself
    h = seq.residual_post_rms(xs, out_dtype=torch.bfloat16)
    assert torch.equal(h, xs.to(torch.bfloat16)) and seq.residual_post_rms(xs, out_dtype=torch.float32) is xs
    with pytest.raises(ValueError):
        seq.residual_post_rms(xs, dev(y), dev(nw)[:-1] if W > 1 else dev(rnd(2)), m)


# ------------------------------------------------------------------------------------------------ far tokens and edges that show
def marked_inputs(T, W, d, marks, seed):
    """Hidden states for identity-like q / k projections onto the first d dimensions: the last position and the marked ones point along
    dimension d - 1 (which does not turn), each with a size of its own — the key norm drops the size, the values keep it —, all others at
    right angles to it."""
    h = rnd(T, W, seed=seed)
    h[:, d - 1] = 0.0
    for n, j in enumerate(sorted(marks) + [T - 1]):
        h[j, :d] = 0.0
        h[j, d - 1] = [8.0, 0.5, 6.0, 0.25, 10.0, 0.125][n % 6] if j != T - 1 else 1.0
    return h


@pytest.mark.parametrize("size,page,T", [(9, 4, 61), (16, 4, 50), (8, 8, 33), (5, 8, 30), (33, 8, 80), (1, 4, 20)])
def test_window_edges_with_peaked_scores(seq, size, page, T):
    """The last query scores the first and last position of its window, the one that has just left it, and the next ones on either side
    of a page border far above everything else; a window that is off by one moves the output by much more than the tolerance — in a
    prompt and when the last token is decoded alone."""
    W, d, i = 32, 8, T - 1
    m = att(heads=2, kv_heads=1, dim=d, size=size, scale=0.8, dims=4)
    marks = {j for j in (i - 1, i - size + 1, i - size, i - size - 1, i // page * page - 1) if 0 <= j < i}
    w, h = att_weights(m, W, seed=11), marked_inputs(T, W, d, marks, seed=4)
    eye = torch.zeros(d, W)
    eye[:, :d] = torch.eye(d)
    w["q"], w["k"] = eye.repeat(2, 1), eye.clone()
    w["q.norm"][d - 1] = w["k.norm"][d - 1] = 1.0
    want = O.key_value_attention(n64(h), f64(w), m, EPS)
    for wrong in (size + 1, size - 1):
        if wrong > 0:
            differs(O.key_value_attention(n64(h), f64(w), dict(m, mask={"size": wrong}), EPS)[i], want[i], 3e-2)
    mixer = make_att(m, w)
    for cuts in ([T], [T - 1], [T - 3, 2], [5, 2, 2, 9]):
        close(run_attention(seq, mixer, h, cuts, page_size=page)[i], want[i], 3e-5, f"portions {cuts}")


def test_softmax_with_one_added_when_all_scores_are_low(seq):
    """Scores far below zero: nearly all of the weight goes to the added one, and the outputs are small but exact."""
    m = att(heads=2, kv_heads=1, dim=8, size=30, scale=1.2, dims=4, scaling=None)
    W, T = 24, 40
    w, h = att_weights(m, W, seed=2), rnd(T, W, seed=3).abs() + 0.5
    h = bf(h)
    eye = torch.zeros(8, W)
    eye[4:, 4:8] = torch.eye(4)                      # the part that does not turn
    w["q"], w["k"] = eye.repeat(2, 1), -eye
    w["q.norm"], w["k.norm"] = torch.ones(8), torch.ones(8)
    want = O.key_value_attention(n64(h), f64(w), m, EPS)
    assert np.abs(want).max() < 0.1 * np.abs(n64(w["o"])).max() * np.abs(n64(h)).max()
    mixer = make_att(m, w)
    for cuts in ([T], [], [17, 2]):
        close(run_attention(seq, mixer, h, cuts), want, 3e-5, f"portions {cuts}")


@pytest.mark.parametrize("far", [0, 1, 3, 250])
@pytest.mark.parametrize("kind", ["mlstm", "mlstm_registers", "delta", "recurrent"])
def test_far_tokens_kept_by_the_state(seq, kind, far):
    """Slow forgetting: one token hundreds of positions back carries a large share of the last output."""
    W, T = 24, 301
    h = 0.3 * rnd(T, W, seed=5)
    h[far] = (40.0 if kind == "recurrent" else 6.0) * rnd(W, seed=6)
    h = bf(h)
    if kind.startswith("mlstm"):
        m = mem(heads=2, dim=8, vdim=6) if kind == "mlstm" else mem(heads=2, dim=64, vdim=32)
        w = mem_weights(m, W, seed=7, forget=12.0)
        m = dict(m, gate_cap=20.0)
        w["f"], w["i.b"] = 0.0 * w["f"], torch.zeros(2)
        w["i"] = w["k"][:2] * 0.0
        mixer, oracle = make_mem(m, w), lambda x: O.matrix_memory(x, f64(w), m, EPS)
    elif kind == "delta":
        m = dlt(heads=2, kv_heads=1, dim=8, vdim=6)
        w = dlt_weights(m, W, seed=7, dt=-12.0)
        w["a"], w["b"], w["A_log"] = 0.0 * w["a"], 0.0 * w["b"], torch.zeros(2)
        w["b"] = bf(0.02 * rnd(2, W, seed=3))
        h[far + 1:, :] = bf(0.05 * h[far + 1:, :])
        w["b"][:, 0] = 1.0                            # later tokens write little: their write strength is closed by column 0
        h[:, 0] = -6.0
        h[far, 0] = 6.0
        mixer, oracle = make_dlt(m, w), lambda x: O.delta_rule(x, f64(w), m, EPS)
    else:
        m = rec(width=24, blocks=3, conv=3)
        w = rec_weights(m, W, seed=7, lam=-9.0)
        mixer, oracle = make_rec(m, w), lambda x: O.recurrent_block(x, f64(w), m)
    want = oracle(n64(h))
    lost = n64(h)
    lost[far, 1:] = 0.0
    differs(oracle(lost)[T - 1], want[T - 1], 0.05)
    for cuts in ([T], [T - 1], [100, 2, 150, 40]):
        close(run_recurrent(seq, mixer, h, cuts)[T - 1], want[T - 1], 5e-5, f"portions {cuts}")


# ------------------------------------------------------------------------------------------------ the model through the scheduler
def test_prefill_against_the_oracle_layer_by_layer(seq):
    raw = default_cfg()
    model, w = build(raw, seed=1, page_size=4)
    tk = toks(75, raw["vocab"], 3)
    trace = []
    want = O.forward(raw, w, tk, trace)
    model.layer_trace = []
    got = run_portions(model, tk, [75])
    assert len(model.layer_trace) == len(trace) == 6
    for i, (a, b) in enumerate(zip(model.layer_trace, trace)):
        close(a.cpu().numpy(), b, 3e-5, f"residual stream after layer {i}")
    model.layer_trace = None
    close(got, want, 5e-5, "logits")


def test_decoding_and_portions_equal_prefill(seq):
    raw = default_cfg()
    model, w = build(raw, seed=2, page_size=4)
    tk = toks(70, raw["vocab"], 4)
    want = O.forward(raw, w, tk)
    for cuts in ([], [2] * 35, [2, 3, 4, 5, 6, 7, 8, 9], [33, 2, 2, 31], [69]):
        close(run_portions(model, tk, cuts), want, 5e-5, f"portions {cuts}")


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
    pages and slots must not reach the next one."""
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
    raw = model_cfg([PA(par(att(size=20))), ME(mlp=dense()), DE(), ME(mem(heads=1, dim=32, vdim=32))])
    model, w = build(raw, seed=6)
    tk = toks(330, raw["vocab"], 8)
    want = O.forward(raw, w, tk)
    got = run_portions(model, tk, [10])                     # 320 tokens decoded one by one, across five pages of 64
    close(got, want, 1e-4, "330 tokens")
    close(got[-1], want[-1], 1e-4, "the last token")


def test_bfloat16_serving_stays_near_the_oracle(seq):
    """Every position bounded where each token uses every expert; the median where rounding can turn a close choice of experts."""
    every = [PA(mlp=moe(experts=4, top=4)), ME(mlp=dense()), DE(mlp=moe(experts=3, top=3))]
    for raw, quantile in ((model_cfg(every), 0.9), (default_cfg(), 0.5)):
        model, w = build(raw, dtype=torch.bfloat16, seed=7, page_size=8)
        tk = toks(90, raw["vocab"], 9)
        want = O.forward(raw, w, tk)
        for got, what in ((run_portions(model, tk, [90]), "prefill"), (run_portions(model, tk, [40, 2, 17]), "portions and decoding")):
            err = np.abs(got.astype(np.float64) - want).max(-1) / np.abs(want).max()
            assert np.quantile(err, quantile) <= 4e-2, f"{what}: {np.quantile(err, quantile):.3e}"


def test_other_sizes_than_any_shipped_model(seq):
    """Every size that tends to coincide in shipped configurations is made different here, or 1: one head, a window of one, one expert, one
    tap, blocks of one channel, rotated parts of the head, no feed-forward at all, odd widths."""
    layers = [ME(mem(heads=1, dim=3, vdim=17, gate_cap=1.5)),
              PA(par(att(heads=1, kv_heads=1, dim=2, size=1, dims=2, base=7.0), rec(width=5, blocks=5, conv=1), 1.0, 1.0), moe(experts=1, top=1, ff=1)),
              DE(dlt(heads=5, kv_heads=5, dim=9, vdim=1, conv=1), dense(1)),
              PA(par(att(heads=6, kv_heads=2, dim=14, size=300, dims=6, base=1000.0, scaling={"factor": 2.0, "original": 16, "fast": 1.5, "slow": 0.5}),
                     rec(width=57, blocks=3, conv=7), -0.5, 2.0), dense(70)),
              DE(dlt(heads=6, kv_heads=3, dim=1, vdim=5, conv=5), moe(experts=7, top=6, ff=31))]
    raw = model_cfg(layers, width=23, vocab=13, eps=3e-4, m=1.7)
    model, w = build(raw, seed=8, page_size=4)
    tk = toks(45, 13, 10)
    want = O.forward(raw, w, tk)
    for cuts in ([45], [], [7, 2, 2]):                          # (a head of one value is little more than a sign after its norm: it amplifies rounding)
        close(run_portions(model, tk, cuts), want, 1e-4, f"portions {cuts}")


@pytest.mark.parametrize("layers", [[ME()], [DE(mlp=dense())], [PA()], [ME(mlp=moe()), ME(mlp=dense(5))], []])
def test_layer_lists_of_every_kind(seq, layers):
    """One mixer alone (also a model that caches no keys at all), and no layer at all."""
    raw = model_cfg(layers, width=16)
    model, w = build(raw, seed=14, page_size=4)
    tk = toks(21, 50, 11)
    want = O.forward(raw, w, tk)
    for cuts in ([21], [4, 2, 9]):
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
    from krasis_b200.kivurax import KivuraxConfig, random_weights
    from krasis_b200.registry import architecture_of, load_model
    raw = default_cfg()
    w = random_weights(KivuraxConfig.from_dict(raw), 10)
    header, blobs, off = {}, [], 0
    for k, v in w.items():
        b = v.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        header[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    hj = json.dumps(header).encode()
    (tmp_path / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    assert architecture_of(str(tmp_path)) == "Kivurax"
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
def test_tensor_core_attention_with_one_added(seq):
    """128 dims: portions of 128 tokens or more run the tcgen05 attention core.  Peaked scores on the window's edges; against the oracle and
    against the plain kernels on the same bf16 cache."""
    from krasis_b200.build import build as build_core
    build_core()
    W, d, T = 192, 128, 400
    i = T - 1
    for heads, kv_heads, size in ((2, 1, 100), (4, 4, 64), (16, 4, 37)):
        m = att(heads=heads, kv_heads=kv_heads, dim=d, size=size, scale=0.05, dims=64, base=10000.0)
        w = att_weights(m, W, seed=21)
        h = marked_inputs(T, W, d, {i - 1, i - size + 1, i - size, i - size - 1, 200}, seed=6)
        eye = torch.zeros(d, W)
        eye[:, :d] = torch.eye(d)
        w["q"], w["k"] = eye.repeat(heads, 1), eye.repeat(kv_heads, 1)
        w["q.norm"][d - 1] = w["k.norm"][d - 1] = 1.0
        want = O.key_value_attention(n64(h), f64(w), m, EPS)
        for wrong in (size - 1, size + 1):
            off = O.key_value_attention(n64(h), f64(w), dict(m, mask={"size": wrong}), EPS)
            differs(off[i], want[i], 0.1)
        mixer = make_att(m, w, torch.bfloat16)
        assert mixer.tc_shape
        fast = run_attention(seq, mixer, h, [T], page_size=8)
        parts = run_attention(seq, mixer, h, [130, 2, T - 132], page_size=8)
        mixer.tc_min_portion = 1 << 30
        plain = run_attention(seq, mixer, h, [T], page_size=8)
        for got, what in ((plain, "plain kernels"), (fast, "tensor-core prefill"), (parts, "tensor-core portions")):
            rows_within(got, want, 2e-2, f"{heads} heads, {what}")
            close(got[i], want[i], 2e-2, f"{heads} heads, the marked row, {what}")
        close(fast, plain.astype(np.float64), 1e-2, "tensor core against plain kernels")


@pytest.mark.parametrize("m", [rec(width=256, blocks=4, conv=4), rec(width=96, blocks=3, conv=2), rec(width=128, blocks=1, conv=3)])
def test_tensor_core_gates_of_the_recurrent_block(seq, m):
    """The gate products of long bfloat16 steps: inputs as a high and a low part, so that the products keep 16 bits of their inputs."""
    from krasis_b200.build import build as build_core
    build_core()
    W, T = 64, 300
    w, h = rec_weights(m, W, seed=3), rnd(T, W, seed=1)
    mixer = make_rec(m, w, torch.bfloat16)
    u = rnd(T, m["width"], seed=4) * 3.0 + 0.01 * torch.randn(T, m["width"], generator=torch.Generator().manual_seed(5))
    z, ldz, zb = mixer._gate_products(u.to(DEV))
    n, B = m["width"] // m["blocks"], m["blocks"]
    z = torch.as_strided(z, (T, B, 2 * n), (ldz, zb, 1)).cpu().numpy()
    assert zb > 2 * n                                                     # the grouped layout: the tensor cores ran
    for k, name in enumerate(("ra", "ri")):
        close(z[:, :, k * n:(k + 1) * n].reshape(T, -1), O.block_product(n64(u), n64(w[name])), 3e-5, name)
    want = O.recurrent_block(n64(h), f64(w), m)
    fast, parts = run_recurrent(seq, mixer, h, [T]), run_recurrent(seq, mixer, h, [257, 2, 40])
    mixer.tc_min_tokens = 1 << 30
    plain = run_recurrent(seq, mixer, h, [T])
    for got, what in ((plain, "plain kernels"), (fast, "tensor-core gates"), (parts, "portions")):
        rows_within(got, want, 2e-2, what)
    close(fast, plain.astype(np.float64), 1e-2, "tensor cores against plain kernels")


def test_tensor_core_experts_with_weights_on_their_inputs(seq):
    from krasis_b200.build import build as build_core
    from krasis_b200.mixers import RoutedExperts
    build_core()
    m, W, T = moe(experts=4, top=4, ff=64), 128, 300
    E, F = 4, 64
    w = {"router": rnd(E, W, seed=1, sd=W ** -0.5 * 2)}
    for e in range(E):
        w.update({f"e{e}.gate": rnd(F, W, seed=10 + 3 * e, sd=W ** -0.5 * 1.5), f"e{e}.up": rnd(F, W, seed=11 + 3 * e, sd=W ** -0.5 * 1.5),
                  f"e{e}.down": rnd(W, F, seed=12 + 3 * e, sd=F ** -0.5)})
    h = rnd(T, W, seed=5)
    want = O.routed_experts(n64(h), f64(w), m)
    mlp = RoutedExperts(under(w), E, 0, 4, torch.bfloat16, torch.device(DEV), score="sigmoid", act="silu", weight_input=True)
    hb = h.to(DEV, torch.bfloat16)
    assert mlp._tensor_core_ok(hb, T * 4)
    fast = mlp.forward(hb).cpu().numpy()
    mlp.tc_min_rows_per_expert = 1 << 30
    rows_within(fast, want, 1.5e-2, "tensor cores")
    rows_within(mlp.forward(hb).cpu().numpy(), want, 1.5e-2, "plain kernels")


def test_tensor_core_prefill_of_the_whole_model(seq):
    from krasis_b200.build import build as build_core
    build_core()
    every = moe(experts=4, top=4, ff=64)                                  # every expert runs: no close choice turns by rounding
    layers = [PA(par(att(heads=4, kv_heads=2, dim=128, size=200, scale=0.05, dims=64, base=10000.0), rec(width=128, blocks=2)), every),
              ME(mem(heads=2, dim=64, vdim=64), dense(128)), DE(dlt(heads=4, kv_heads=2, dim=64, vdim=64, conv=4), every),
              ME(mem(heads=1, dim=128, vdim=128, gate_cap=15.0))]
    raw = model_cfg(layers, width=128)
    model, w = build(raw, dtype=torch.bfloat16, seed=31)
    assert model.layers[0]["mixer"].left.tc_shape
    tk = toks(520, raw["vocab"], 16)
    want = O.forward(raw, w, tk)
    whole = run_portions(model, tk, [520], s=sched(model, 1024))
    parts = run_portions(model, tk, [130, 257, 128], s=sched(model, 1024))
    model.layers[0]["mixer"].left.tc_min_portion = model.layers[0]["mixer"].right.tc_min_tokens = 1 << 30
    plain = run_portions(model, tk, [520], s=sched(model, 1024))
    rows_within(plain, want, 4e-2, "plain kernels against the oracle", 0.9)
    rows_within(whole, want, 4e-2, "tensor-core prefill against the oracle", 0.9)
    rows_within(whole, plain.astype(np.float64), 3e-2, "tensor-core prefill against the plain kernels", 0.9)
    rows_within(parts, plain.astype(np.float64), 3e-2, "tensor-core portions against the plain kernels", 0.9)
