"""Ribovik against the plain implementation (tests/plain/ribovik_plain.py): every mechanism alone through the part bench (whole
prompts, portions beside decoded tokens, pages that are freed and used again, positions far out), whole models through the trace
runner in every way of cutting with the stream compared after every layer, and greedy generation through the engine's own entry
point and the command line.  Weights are made here so that a fault shows: loud keys just inside and just outside a chunk's edge,
scores around the sink's, biases as large as the products, gates beyond their clip, corrections that decide the choice of
experts, identity experts among the chosen."""
import json
import math
import os

import numpy as np
import pytest
import torch

from imp_b200.parts.bench import PartBench
from imp_b200.parts.plan import PartSpec
from imp_b200.parts.registry import mixer_cache_spec
from plain import ribovik_plain as R
from replay_helpers import collect, mixed, portions, round64, run_trace, tail_decode, whole
from safetensors_io import save_safetensors

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
NAME = {torch.float32: "float32", torch.bfloat16: "bfloat16"}
EPS = 2e-4


def rnd(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(*shape, generator=g) * scale


def close(got, want, dtype, what="", loose=1.0):
    got, want = got.float().cpu(), want.float().cpu()
    scale = max(float(want.abs().max()), 1e-3)
    atol, rtol = (3e-5 * scale, 3e-5) if dtype == torch.float32 else (0.025 * scale * loose, 0.025 * loose)
    err = (got - want).abs()
    assert (err <= atol + rtol * want.abs()).all(), f"{what}: max error {err.max().item():.3g} (scale {scale:.3g})"


def run_part(bench, part, x, ctx, cache=None):
    torch.cuda.synchronize()
    out = part.forward(x.to(DEV), ctx, cache)
    bench.sync()
    return out.clone()


def in_pieces(bench, part, x, sizes, rid="a"):
    """One request's rows in steps of `sizes` tokens."""
    outs, done = [], 0
    for n in sizes:
        ctx = bench.prepare([(rid, [1] * n, [])])
        outs.append(run_part(bench, part, x[done:done + n], ctx, bench.cache_view(0)))
        bench.commit()
        done += n
    assert done == x.shape[0]
    return torch.cat(outs)


# ------------------------------------------------------------------ weights by checkpoint suffix
def attention_weights(d, c, seed):
    H, G, D, Dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    s = 1.0 / math.sqrt(d)
    return {"q": rnd(H * D, d, seed=seed, scale=s), "q.b": rnd(H * D, seed=seed + 1), "k": rnd(G * D, d, seed=seed + 2, scale=s),
            "k.b": rnd(G * D, seed=seed + 3), "v": rnd(G * Dv, d, seed=seed + 4, scale=s), "v.b": rnd(G * Dv, seed=seed + 5),
            "o": rnd(d, H * Dv, seed=seed + 6, scale=1.0 / math.sqrt(H * Dv))}


def dense_weights(d, ff, seed):
    s = 1.0 / math.sqrt(d)
    return {"gate": rnd(ff, d, seed=seed, scale=s), "gate.b": rnd(ff, seed=seed + 1), "up": rnd(ff, d, seed=seed + 2, scale=s),
            "up.b": rnd(ff, seed=seed + 3), "down": rnd(d, ff, seed=seed + 4, scale=1.0 / math.sqrt(ff)), "down.b": rnd(d, seed=seed + 5)}


def moe_weights(d, c, seed):
    E, N, F = c["router"]["experts"], c["router"]["experts"] + c["router"].get("identity", 0), c["expert"]["ff"]
    s = 1.0 / math.sqrt(d)
    w = {"router": rnd(N, d, seed=seed, scale=2 * s), "correction": rnd(N, seed=seed + 1, scale=0.1)}

    def one(name, ff, sd):
        w[name + ".gate"] = rnd(ff, d, seed=sd, scale=2 * s)
        w[name + ".up"] = rnd(ff, d, seed=sd + 1, scale=2 * s)
        w[name + ".down"] = rnd(d, ff, seed=sd + 2, scale=1.0 / math.sqrt(ff))

    for e in range(E):
        one(f"e{e}", F, seed + 10 * e + 3)
    if c.get("shared"):
        one("shared", c["shared"]["ff"], seed + 9003)
    return w


ATTENTION_NAMES = {"q": "q_proj", "q.b": "q_bias", "k": "k_proj", "k.b": "k_bias", "v": "v_proj", "v.b": "v_bias", "o": "o_proj"}
DENSE_NAMES = {"gate": "gate_proj", "gate.b": "gate_bias", "up": "up_proj", "up.b": "up_bias", "down": "down_proj", "down.b": "down_bias"}


def moe_names(c):
    n = {"router": "router", "correction": "choice_bias"}
    for e in list(range(c["router"]["experts"])) + (["shared"] if c.get("shared") else []):
        for m in ("gate", "up", "down"):
            n[f"shared.{m}" if e == "shared" else f"e{e}.{m}"] = f"shared_{m}" if e == "shared" else f"{m}_{e}"
    return n


def moe_params(d, c):
    p = {"hidden_size": d, "num_experts": c["router"]["experts"], "num_identity": c["router"].get("identity", 0), "top_k": c["router"]["top"],
         "expert_size": c["expert"]["ff"], "expert": "clipped", "expert_limit": c["expert"]["limit"], "router_bias": False, "scores": "softmax_all",
         "choice_bias": True, "renormalise": True}
    if c.get("shared"):
        p.update(shared_size=c["shared"]["ff"], shared_limit=c["shared"]["limit"], shared_gate=False)
    return p


# ------------------------------------------------------------------------------------ attention alone
YARN = {"factor": 4.0, "original": 60, "fast": 3.0, "slow": 0.6}
ATTENTION_CASES = [
    dict(d=72, heads=6, kv_heads=2, dim=24, vdim=40, chunk=10, rot=8, base=100.0, scaling=YARN, page=4),       # values longer than keys; part of a head rotated
    dict(d=64, heads=4, kv_heads=4, dim=64, vdim=64, chunk=33, rot=64, base=10000.0, scaling=dict(YARN, factor=40.0), page=16),   # a key head per head
    dict(d=40, heads=2, kv_heads=1, dim=12, vdim=20, chunk=0, rot=0, base=1.0, scaling=None, page=8),          # neither chunks nor rotation
    dict(d=48, heads=3, kv_heads=1, dim=128, vdim=96, chunk=64, rot=32, base=500.0, scaling=YARN, page=16),    # chunks of whole pages; values shorter than keys
    dict(d=32, heads=1, kv_heads=1, dim=16, vdim=16, chunk=1, rot=2, base=7.0, scaling=None, page=16),         # a token sees itself and the sink
    dict(d=48, heads=20, kv_heads=1, dim=8, vdim=8, chunk=7, rot=8, base=50.0, scaling=YARN, page=16),         # twenty heads on one key head
    dict(d=50, heads=2, kv_heads=2, dim=10, vdim=6, chunk=21, rot=6, base=90.0, scaling=YARN, page=4),         # sizes that are multiples of nothing
    dict(d=64, heads=2, kv_heads=1, dim=200, vdim=64, chunk=50, rot=100, base=1e6, scaling=YARN, page=16),     # a large head
]


def attention_config(case, scale=None):
    c = {k: case[k] for k in ("heads", "kv_heads", "dim", "vdim")}
    c["scale"] = scale or 1.3 / math.sqrt(c["dim"])
    if case["chunk"]:
        c["mask"] = {"size": case["chunk"]}
    if case["rot"]:
        c["rot"] = {"base": case["base"], "dims": case["rot"]}
        if case["scaling"]:
            c["rot"]["scaling"] = case["scaling"]
    return c


def attention_setup(dtype, case, w=None, scale=None, pages=None):
    c = attention_config(case, scale)
    params = {"hidden_size": case["d"], "num_heads": c["heads"], "num_kv_heads": c["kv_heads"], "head_dim": c["dim"], "value_dim": c["vdim"],
              "scale": c["scale"], "norm_eps": EPS, "chunk": case["chunk"], "rot_dims": case["rot"], "rot_base": case["base"], "rot_pairing": "neighbours",
              "qkv_bias": True, "qk_norm": True, "qk_norm_weight": False, "qk_norm_position": "after_rotation", "sink": True}
    if case["scaling"] and case["rot"]:
        params["rot_scaling"] = dict(case["scaling"], kind="yarn")
    bench = PartBench(NAME[dtype], [mixer_cache_spec("gated_head_attention", params)], page_size=case["page"],
                      num_pages=pages or 2048 // case["page"], max_tokens=1024, max_seq_len=1 << 17)
    w = {k: v.to(dtype) for k, v in (w or attention_weights(case["d"], c, seed=100)).items()}
    part = bench.build("mixer", PartSpec("gated_head_attention", params), {ATTENTION_NAMES[k]: v.to(DEV) for k, v in w.items()})
    return bench, part, c, {"m." + k: v.double() for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ATTENTION_CASES)
def test_attention_whole_portions_decoding_and_reused_pages(dtype, case):
    bench, part, c, W = attention_setup(dtype, case)
    lengths = [93, 11]
    xs = [rnd(n, case["d"], seed=20 + i).to(dtype) for i, n in enumerate(lengths)]
    want = [R.attention(x.double(), W, "m.", c, EPS) for x in xs]
    ctx = bench.prepare([(f"w{i}", [1] * n, []) for i, n in enumerate(lengths)])
    out = run_part(bench, part, torch.cat(xs), ctx, bench.cache_view(0))
    bench.commit()
    close(out[:93], want[0], dtype, "whole", loose=2.0)
    close(out[93:], want[1], dtype, "whole, second sequence", loose=2.0)
    bench.end("w0")
    bench.end("w1")                       # their pages come out first for the next requests
    done, outs, other = 0, [], 0
    for n in (10, 2, 20, 1, 4, 2, 33, 1, 1, 1, 2, 16):       # the first sequence in portions, the second decoding beside it
        es, parts = [("p0", [1] * n, [])], [xs[0][done:done + n]]
        if other < 11:
            es.append(("p1", [1], []))
            parts.append(xs[1][other:other + 1])
        ctx = bench.prepare(es)
        o = run_part(bench, part, torch.cat(parts), ctx, bench.cache_view(0))
        bench.commit()
        outs.append(o[:n])
        if other < 11:
            close(o[n:], want[1][other:other + 1], dtype, f"decoded token {other}", loose=2.0)
            other += 1
        done += n
    pieces = torch.cat(outs)
    close(pieces, want[0], dtype, "portions", loose=2.0)
    if dtype == torch.float32:
        assert torch.equal(pieces, out[:93]), "the cut changes no bit"


def test_what_attention_rests_on_shows_in_the_plain_results():
    case = dict(ATTENTION_CASES[0], rot=16, chunk=25)
    c = attention_config(case, scale=0.5)
    W = {"m." + k: v.double() for k, v in attention_weights(case["d"], c, seed=100).items()}
    x = rnd(60, case["d"], seed=20).double()
    run = lambda W=W, c=c, **kw: R.attention(x, W, "m.", c, EPS, **kw)
    want = run()
    far = lambda other: float((other - want).abs().max()) > 0.02 * float(want.abs().max())
    assert far(run(c=dict(c, mask={"size": 26}))), "one more key in the chunk"
    assert far(run(c=dict(c, scale=c["scale"] * 1.2))), "the scale"
    assert far(run(c=dict(c, rot=dict(c["rot"], base=90.0)))), "the rotation's base"
    assert far(run(c=dict(c, rot={"base": 100.0, "dims": 16}))), "the slowed pairs and the stretch"
    assert far(run(c=dict(c, rot=dict(c["rot"], scaling=dict(YARN, factor=16.0))))), "the factor"
    assert far(run(positions=torch.arange(60) * 2)), "positions"
    for b in ("q.b", "k.b", "v.b"):
        other = dict(W)
        other["m." + b] = torch.zeros_like(W["m." + b])
        assert far(run(W=other)), b


def test_sink_and_unit_norms_decide():
    """Queries and keys of very different lengths give the same scores up to their direction, and with scores around zero a chunk's
    first tokens give most of their weight to the sink."""
    case = ATTENTION_CASES[1]
    dtype = torch.float32
    c = attention_config(case)
    w = attention_weights(case["d"], c, seed=100)
    w["q"], w["q.b"] = 30 * w["q"], 30 * w["q.b"]
    w["k"], w["k.b"] = 0.2 * w["k"], 0.2 * w["k.b"]
    bench, part, c, W = attention_setup(dtype, case, w=w)
    x = rnd(70, case["d"], seed=21)
    want = R.attention(x.double(), W, "m.", c, EPS)
    close(in_pieces(bench, part, x, (40, 1, 2, 27)), want, dtype, "lengths that differ")
    H, D, Dv, O = c["heads"], c["dim"], c["vdim"], W["m.o"]
    v = (x.double() @ W["m.v"].T + W["m.v.b"])[33]           # the first token of a chunk sees itself alone: exp(s) / (1 + exp(s)) of its value
    q = (x.double() @ W["m.q"].T + W["m.q.b"])[33].view(H, D)
    k = (x.double() @ W["m.k"].T + W["m.k.b"])[33].view(H, D)
    assert c["rot"]["dims"] == D, "the rotation turns q and k of one position alike: their product stays"
    s = (R.unit_rms(q, EPS) * R.unit_rms(k, EPS)).sum(-1) * c["scale"]
    p = torch.sigmoid(s)
    assert float((p - 1).abs().max()) > 0.2
    assert torch.allclose((p[:, None] * v.view(H, Dv)).reshape(-1) @ O.T, want[33], rtol=1e-3, atol=1e-3 * float(want.abs().max()))


def loud_key_weights(case, c, seed):
    """Random weights in which every query looks along one unrotated entry of its head, and a token with much of input 0 is a key
    along it; q and k are divided by their root mean square, so the other entries are kept small."""
    d, D = case["d"], case["dim"]
    w = attention_weights(d, c, seed)
    at = D - 1
    assert at >= case["rot"], "beyond the rotated front"
    for n, heads in (("q", c["heads"]), ("k", c["kv_heads"])):
        w[n], w[n + ".b"] = 0.3 * w[n], 0.3 * w[n + ".b"]
        for h in range(heads):
            w[n][h * D + at] = 0.0
            w[n][h * D + at, 0 if n == "k" else 1] = 2.0
            w[n + ".b"][h * D + at] = 0.0
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
def test_a_loud_key_just_inside_and_just_outside_a_chunk_and_far_away(dtype, decoded):
    """The token at `at` is the key every later token looks for.  The last query of its chunk still sees it, the next one does not;
    without chunks a query 600 tokens later finds it among all the others.  In a prompt, and with the edge passed while decoding."""
    for case, T, at in ((dict(d=48, heads=3, kv_heads=1, dim=32, vdim=24, chunk=37, rot=8, base=100.0, scaling=YARN, page=16), 120, 40),
                        (dict(d=48, heads=2, kv_heads=2, dim=16, vdim=16, chunk=64, rot=0, base=1.0, scaling=None, page=16), 150, 70),
                        (dict(d=40, heads=2, kv_heads=1, dim=16, vdim=32, chunk=0, rot=4, base=100.0, scaling=None, page=16), 640, 3)):
        c = attention_config(case, scale=1.0)
        bench, part, c, W = attention_setup(dtype, case, w=loud_key_weights(case, c, seed=300), scale=1.0)
        x = rnd(T, case["d"], seed=301, scale=0.5)
        x[:, 0] = 0.0
        x[:, 1] = 1.5
        x[at, 0] = 6.0
        x = x.to(dtype)
        want = R.attention(x.double(), W, "m.", c, EPS)
        quiet = x.clone()
        quiet[at, 0] = 0.0
        moved = (want - R.attention(quiet.double(), W, "m.", c, EPS)).abs().amax(dim=-1) / want.abs().max()
        size = case["chunk"]
        if size:
            edge = (at // size + 1) * size
            assert moved[edge - 1] > 0.1 and moved[edge] < 1e-9 and edge < T, "the plain result hangs on the key exactly inside the chunk"
        else:
            assert moved[T - 1] > 0.1, "the plain result hangs on the far key"
        n_tail = 60 if decoded else 0
        if decoded and size:
            assert T - n_tail <= edge - 1, "the edge is passed while decoding"
        out = in_pieces(bench, part, x, (T - n_tail,) + (1,) * n_tail)
        close(out, want, dtype, f"chunk {size}", loose=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [64, 128, 96])
def test_long_portions_with_chunk_edges_inside_the_kernels_tiles(dtype, dim):
    """Portions of hundreds of tokens take the tiled kernels (tcgen05 at head sizes 64 and 128, mma.sync at 96); chunk edges fall
    inside their tiles."""
    case = dict(d=64, heads=4, kv_heads=2, dim=dim, vdim=dim, chunk=150, rot=dim, base=1000.0, scaling=YARN, page=16)
    bench, part, c, W = attention_setup(dtype, case)
    x = rnd(700, 64, seed=21).to(dtype)
    want = R.attention(x.double(), W, "m.", c, EPS)
    close(in_pieces(bench, part, x, (300, 257, 2, 141)), want, dtype, "long portions", loose=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_positions_in_few_pages(dtype):
    """12,000 tokens through a pool of 1,200: earlier chunks give their pages back, and the angles are right far out (a last chunk's
    result depends on its own tokens and positions alone)."""
    size, T, n = 48, 12000, 1000
    case = dict(d=32, heads=2, kv_heads=1, dim=16, vdim=16, chunk=size, rot=16, base=10.0, scaling=dict(YARN, original=10), page=16)
    bench, part, c, W = attention_setup(dtype, case, pages=75, scale=1.5)
    x = rnd(T, 32, seed=22).to(dtype)
    at = T // size * size - size
    tail = x[at:].double()
    want = R.attention(tail, W, "m.", c, EPS, positions=torch.arange(at, T))
    shifted = R.attention(tail, W, "m.", c, EPS, positions=torch.arange(at + 0.004, T).to(torch.float64))
    assert torch.allclose(want, shifted, atol=1e-9), "only differences of positions matter"
    outs, done = [], 0
    for m in [n] * (T // n - 1) + [n - 30] + [1] * 30:
        ctx = bench.prepare([("a", [1] * m, [])])
        o = run_part(bench, part, x[done:done + m], ctx, bench.cache_view(0))
        bench.commit()
        done += m
        if done > at:
            outs.append(o)
    got = torch.cat(outs)
    close(got[-(T - at):], want, dtype, "the last chunks", loose=2.0)
    assert sum(p >= 0 for t in bench.cache_info()["paged"][0]["tables"].values() for p in t) <= 2 * size // 16 + 1


# ------------------------------------------------------------------------------------- feed-forwards alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, ff", [(72, 100), (64, 256), (40, 37), (256, 1024)])
def test_dense_feed_forward_with_biases(dtype, d, ff):
    bench = PartBench(NAME[dtype], [], max_tokens=512, max_seq_len=512)
    w = {k: v.to(dtype) for k, v in dense_weights(d, ff, seed=600).items()}
    part = bench.build("feed_forward", PartSpec("gated_mlp", {"hidden_size": d, "intermediate_size": ff, "activation": "silu", "bias": True}),
                       {DENSE_NAMES[k]: v.to(DEV) for k, v in w.items()})
    W = {"f." + k: v.double() for k, v in w.items()}
    x = rnd(300, d, seed=601).to(dtype)
    want = R.dense_ff(x.double(), W, "f.")
    for b in ("gate.b", "up.b", "down.b"):
        other = dict(W)
        other["f." + b] = torch.zeros_like(W["f." + b])
        assert (R.dense_ff(x.double(), other, "f.") - want).abs().max() > 0.05 * want.abs().max(), b
    out = run_part(bench, part, x, bench.prepare([("a", [1] * 300, [])]))
    close(out, want, dtype, "whole", loose=2.0)
    for lo, hi in ((5, 7), (9, 10), (20, 60)):
        few = run_part(bench, part, x[lo:hi], bench.prepare([(f"b{lo}", [1] * (hi - lo), [])]))
        close(few, want[lo:hi], dtype, f"{hi - lo} tokens", loose=2.0)
        if dtype == torch.float32:
            assert torch.equal(few, out[lo:hi]), "a token's result does not depend on its neighbours"


def moe_config(experts, identity, top, ff, limit, shared=None):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top},
            "shared": None if shared is None else {"ff": shared[0], "limit": shared[1]}}


MOE_CASES = [
    (72, moe_config(12, 3, 5, 20, 1.5, (28, 0.5))),
    (64, moe_config(6, 1, 1, 32, 0.7, (64, 3.0))),          # one choice a token: its weight is one
    (40, moe_config(15, 0, 3, 24, 2.5, None)),              # no identity, no shared expert
    (48, moe_config(4, 9, 6, 16, 1.0, (40, 1.0))),          # more identities than experts
    (50, moe_config(70, 5, 6, 9, 1.2, (11, 0.9))),          # sizes that are multiples of nothing
    (48, moe_config(5, 3, 8, 16, 2.0, None)),               # every output chosen
    (32, moe_config(1, 1, 1, 8, 1.0, None)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, c", MOE_CASES)
def test_routed_clipped_experts_with_identities_and_a_shared_one(dtype, d, c):
    w = {k: v.to(dtype) for k, v in moe_weights(d, c, seed=500).items()}
    bench = PartBench(NAME[dtype], [], max_tokens=256)
    names = moe_names(c)
    part = bench.build("feed_forward", PartSpec("routed_experts", moe_params(d, c)), {names[k]: v.to(DEV) for k, v in w.items()})
    W = {"f." + k: v.double() for k, v in w.items()}
    x = rnd(150, d, seed=501).to(dtype)
    want = R.moe(x.double(), W, "f.", c)
    sure = R.route_margin(x.double(), W, "f.", c) > 1e-3           # rows whose choice hangs on less than rounding are not judged
    assert sure.sum() > 110
    idx = R.route(x.double(), W, "f.", c)[0]
    E, N = c["router"]["experts"], c["router"]["experts"] + c["router"]["identity"]
    if c["router"]["identity"]:
        assert (idx >= E).any() and (idx < E).any(), "identities and experts are both chosen"
    out = run_part(bench, part, x, bench.prepare([("a", [1] * 150, [])]))
    close(out[sure], want[sure], dtype, "whole", loose=2.0)
    outs, done = [], 0
    for n in (3, 1, 2, 64, 70, 10):
        outs.append(run_part(bench, part, x[done:done + n], bench.prepare([("b", [1] * n, [])])))
        done += n
    pieces = torch.cat(outs)
    if dtype == torch.float32:
        assert torch.equal(pieces, out), "a token's result does not depend on its neighbours"
    else:
        close(pieces[sure], want[sure], dtype, "pieces", loose=2.0)
    far = lambda other: (other - want).abs().max() > 0.03 * want.abs().max()
    assert far(R.moe(x.double(), W, "f.", dict(c, expert=dict(c["expert"], limit=c["expert"]["limit"] * 1.3)))), "the experts' clip"
    if c["shared"]:
        assert far(R.moe(x.double(), W, "f.", dict(c, shared=dict(c["shared"], limit=c["shared"]["limit"] * 1.3)))), "the shared expert's own clip"
    if c["router"]["top"] < N:
        free = dict(W)
        free["f.correction"] = torch.zeros(N, dtype=torch.float64)
        assert far(R.moe(x.double(), free, "f.", c)), "the correction decides"


def test_experts_of_long_portions_take_the_dense_products():
    """Enough work an expert that its rows go to the tensor-memory products with the clipped gate in their epilogue."""
    d, c = 512, moe_config(2, 1, 2, 1024, 1.1, None)
    w = {k: v.to(torch.bfloat16) for k, v in moe_weights(d, c, seed=510).items()}
    bench = PartBench("bfloat16", [], max_tokens=9216, max_seq_len=9216)
    names = moe_names(c)
    part = bench.build("feed_forward", PartSpec("routed_experts", moe_params(d, c)), {names[k]: v.to(DEV) for k, v in w.items()})
    x = rnd(9000, d, seed=511).to(torch.bfloat16)
    run_part(bench, part, x[:7000], bench.prepare([("c", [1] * 7000, [])]))         # leaves the workspace full of other numbers
    out = run_part(bench, part, x, bench.prepare([("a", [1] * 9000, [])]))
    few = run_part(bench, part, x[:200], bench.prepare([("b", [1] * 200, [])]))     # the grouped products
    close(out[:200], few, torch.bfloat16, "dense against grouped products")
    W = {"f." + k: v.float() for k, v in w.items()}
    at = torch.arange(0, 9000, 450)
    sure = R.route_margin(x[at].float(), W, "f.", c) > 5e-3
    close(out[at.to(DEV)].cpu()[sure], R.moe(x[at].float(), W, "f.", c)[sure], torch.bfloat16, "rows of the long portion", loose=2.0)


# ------------------------------------------------------------------------------------------ the block alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["dense", "moe", None])
def test_block_adds_the_norm_of_what_a_sublayer_gives(dtype, kind):
    d, case = 64, dict(d=64, heads=4, kv_heads=2, dim=16, vdim=16, chunk=9, rot=16, base=100.0, scaling=YARN, page=16)
    bench, mixer, c, W = attention_setup(dtype, case)
    n1, n2 = (1 + 0.5 * rnd(d, seed=1)).to(dtype), (1 + 0.5 * rnd(d, seed=2)).to(dtype)
    norm = lambda w: bench.build("norm", PartSpec("rmsnorm", {"size": d, "eps": EPS}), {"weight": w.to(DEV)})
    parts = {"mixer": mixer, "mixer_post_norm": norm(n1)}
    x = rnd(20, d, seed=5)
    h16 = x.to(dtype).double()
    stream = x.double() + R.rms_norm(R.attention(h16, W, "m.", c, EPS), n1.double(), EPS)
    if kind == "dense":
        f = {k: v.to(dtype) for k, v in dense_weights(d, 40, 3).items()}
        parts["feed_forward"] = bench.build("feed_forward", PartSpec("gated_mlp", {"hidden_size": d, "intermediate_size": 40, "activation": "silu", "bias": True}),
                                            {DENSE_NAMES[k]: v.to(DEV) for k, v in f.items()})
        y = R.dense_ff(stream, {"f." + k: v.double() for k, v in f.items()}, "f.")
    elif kind == "moe":
        mc = moe_config(5, 2, 3, 16, 1.0, (24, 0.8))
        f = {k: v.to(dtype) for k, v in moe_weights(d, mc, 9).items()}
        parts["feed_forward"] = bench.build("feed_forward", PartSpec("routed_experts", moe_params(d, mc)), {moe_names(mc)[k]: v.to(DEV) for k, v in f.items()})
        Wf = {"f." + k: v.double() for k, v in f.items()}
        y = R.moe(stream, Wf, "f.", mc)
    if kind:
        parts["ffn_post_norm"] = norm(n2)
        want = stream + R.rms_norm(y, n2.double(), EPS)
    else:
        want = stream
    sure = torch.ones(20, dtype=torch.bool) if kind != "moe" or dtype == torch.float32 else R.route_margin(stream, Wf, "f.", mc) > 5e-3
    block = bench.build_block("output_norm", parts, {"has_ffn": kind is not None})
    ctx = bench.prepare([("a", [1] * 20, [])])
    h = x.clone().to(DEV)
    torch.cuda.synchronize()
    block.block_forward(h, None, ctx, bench.cache_view(0))
    bench.sync()
    close(h.cpu()[sure], want[sure], dtype, f"the stream behind feed-forward {kind}", loose=2.0)


# --------------------------------------------------------------- whole models
def att(heads, kv_heads, dim, vdim, chunk, rot, base, scaling, scale=None):
    case = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, chunk=chunk, rot=rot, base=base, scaling=scaling)
    return {"type": "attention", "mixer": attention_config(case, scale)}


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


DENSE = lambda ff: {"kind": "dense", "ff": ff}
# M1: every kind of layer, chunks that differ from layer to layer (several cache groups), keys and values of unequal sizes.
# M2: one geometry throughout, chunks of whole pages, no scaling.  M3: no chunks in one layer, no rotation in another, a layer
# without feed-forward last, pages of 4.  M4: sizes that are multiples of nothing.
MODELS = {
    "M1": ({"architecture": "Ribovik", "vocab": 97, "width": 64, "norm": {"eps": 3e-5},
            "layers": [layer(att(6, 2, 24, 40, 19, 16, 100.0, YARN), DENSE(72)),
                       layer(att(4, 1, 32, 16, 40, 32, 1000.0, dict(YARN, fast=9.0, original=300)), moe_config(9, 2, 4, 24, 1.5, (32, 0.7))),
                       layer(att(3, 3, 16, 16, 19, 4, 50.0, None), None),
                       layer(att(6, 2, 24, 40, 19, 16, 100.0, YARN), moe_config(5, 3, 2, 16, 3.0, None))]}, 16),
    "M2": ({"architecture": "Ribovik", "vocab": 151, "width": 112, "norm": {"eps": 1e-6},
            "layers": [layer(att(5, 1, 64, 64, 48, 64, 10000.0, None, scale=0.2), moe_config(6, 1, 1, 32, 0.9, (48, 2.0))),
                       layer(att(5, 1, 64, 64, 48, 64, 10000.0, None, scale=0.2), DENSE(128)),
                       layer(att(5, 1, 64, 64, 48, 64, 10000.0, None, scale=0.2), moe_config(6, 1, 3, 32, 0.9, (48, 2.0)))]}, 16),
    "M3": ({"architecture": "Ribovik", "vocab": 130, "width": 96, "norm": {"eps": 1e-5},
            "layers": [layer(att(2, 2, 128, 128, 0, 64, 1e5, dict(YARN, original=1000, fast=30.0, slow=2.0)), DENSE(64)),
                       layer(att(8, 4, 16, 16, 100, 0, 1.0, None), moe_config(16, 4, 6, 24, 2.0, (24, 2.0))),
                       layer(att(2, 1, 48, 32, 1, 48, 30.0, YARN), None)]}, 4),
    "M4": ({"architecture": "Ribovik", "vocab": 83, "width": 70, "norm": {"eps": 1e-3},
            "layers": [layer(att(3, 1, 10, 6, 11, 6, 20.0, YARN), moe_config(3, 1, 2, 13, 1.1, (7, 1.9))),
                       layer(att(1, 1, 18, 22, 25, 18, 300.0, YARN), DENSE(37))]}, 8),
}
LENGTHS = {"M1": (1, 23, 75, 40, 130, 64), "M2": (150, 2, 33, 201, 64, 97), "M3": (70, 5, 140, 31, 64, 2), "M4": (45, 3, 70, 20, 64, 9)}


def make_weights(cfg, seed):
    d = cfg["width"]
    W = {"embed": rnd(cfg["vocab"], d, seed=seed), "embed.norm": 1 + 0.2 * rnd(d, seed=seed + 1), "final.norm": (1 + 0.2 * rnd(d, seed=seed + 2)) / math.sqrt(d)}
    for i, lay in enumerate(cfg["layers"]):
        p, s = f"l{i}.", seed + 100000 * (i + 1)
        W[p + "norm1"] = 0.6 + 0.2 * rnd(d, seed=s)
        for k, v in attention_weights(d, lay["mixer"], s + 30).items():
            W[p + "mix." + k] = v
        if lay["mlp"]:
            W[p + "norm2"] = 0.6 + 0.2 * rnd(d, seed=s + 2)
            for k, v in (dense_weights(d, lay["mlp"]["ff"], s + 80) if lay["mlp"]["kind"] == "dense" else moe_weights(d, lay["mlp"], s + 80)).items():
                W[p + "mlp." + k] = v
    return {k: v.to(torch.bfloat16) for k, v in W.items()}


@pytest.fixture(scope="module")
def ribovik_folders(tmp_path_factory):
    out = {}
    for n, (name, (cfg, page)) in enumerate(MODELS.items()):
        folder = str(tmp_path_factory.mktemp(f"ribovik_{name}"))
        W = make_weights(cfg, seed=70 + n)
        with open(os.path.join(folder, "config.json"), "w") as f:
            json.dump(cfg, f)
        save_safetensors(os.path.join(folder, "model.safetensors"), W)
        g = torch.Generator().manual_seed(n)
        reqs = {f"r{i}": torch.randint(0, cfg["vocab"], (m,), generator=g).tolist() for i, m in enumerate(LENGTHS[name])}
        Wd = {k: v.double() for k, v in W.items()}
        ref, unsure = {}, set()
        for rid, ids in reqs.items():
            margins = []
            ref[rid] = R.forward(ids, Wd, cfg, margins=margins).float().numpy()
            if margins:
                # tokens whose choice of experts hangs on less than 16-bit rounding moves a router's scores
                close_call = torch.stack(margins).min(dim=0).values < 0.004
                unsure.update((rid, int(p)) for p in torch.nonzero(close_call)[:, 0])
        out[name] = (folder, cfg, page, Wd, reqs, ref, unsure)
    return out


def check_rows(rows, reqs, ref, dtype, label="", unsure=()):
    """float32: every logit to 1e-4 of the largest.  bfloat16: a row's root-mean-square error against the root mean square of all
    logits is at most 4 % for 95 of 100 rows and 25 % for every row; rows in `unsure` (a router's choice for that token hangs on
    less than the rounding of its 16-bit input moves a score) are not judged."""
    scale = max(float(np.abs(r).max()) for r in ref.values())
    rms_all = float(np.sqrt(np.mean(np.concatenate([r.ravel() for r in ref.values()]) ** 2)))
    rel, n = [], 0
    for rid, ids in reqs.items():
        for p in range(len(ids)):
            got, want = rows[(rid, p)], ref[rid][p]
            err = np.abs(got - want)
            if dtype == "float32":
                assert not (err > 1e-4 * max(scale, 1.0) + 1e-4 * np.abs(want)).any(), \
                    f"{label}: request {rid} position {p}: max error {err.max():.3g} (largest logit {scale:.3g}) in {dtype}"
            elif (rid, p) not in unsure:
                rel.append(float(np.sqrt(np.mean(err ** 2))) / rms_all)
                assert rel[-1] <= 0.25, f"{label}: request {rid} position {p}: rms error {rel[-1]:.3g} of the logits' rms in {dtype}"
            n += 1
    assert n == sum(len(v) for v in reqs.values())
    if rel:
        assert float(np.quantile(rel, 0.95)) <= 0.04, f"{label}: 95th percentile of the rows' rms error {np.quantile(rel, 0.95):.3g} in {dtype}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2", "M3", "M4"])
def test_replay_all_ways_of_cutting(name, dtype, ribovik_folders, tmp_path):
    folder, cfg, page, W, reqs, ref, unsure = ribovik_folders[name]
    assert len(unsure) < sum(len(v) for v in reqs.values()) // 2
    V = cfg["vocab"]
    longest = round64(max(len(v) for v in reqs.values()))
    results = {}
    cuts = [("whole", whole(reqs), longest), ("tail", tail_decode(reqs), longest), ("portions", portions(reqs), longest),
            ("wide_portions", portions(reqs, sizes=(70, 2, 33, 64, 1, 100)), longest)]
    for label, steps, pool in cuts:
        rows = collect(steps, run_trace(folder, dtype, steps, pool, str(tmp_path / label), V, page_size=page))
        check_rows(rows, reqs, ref, dtype, label, unsure)
        results[label] = rows
    steps, peak = mixed(reqs)
    assert max(len(s["entries"]) for s in steps) == 4
    assert peak < sum(round64(len(v)) for v in reqs.values()), "the pool must be too small to avoid reuse"
    rows = collect(steps, run_trace(folder, dtype, steps, peak, str(tmp_path / "mixed"), V, page_size=page))
    check_rows(rows, reqs, ref, dtype, "mixed", unsure)
    results["mixed"] = rows
    if dtype == "float32":
        # every reduction of the float32 path has an order that depends on the row alone
        for label in [c[0] for c in cuts[1:]] + ["mixed"]:
            for key, row in results["whole"].items():
                assert np.array_equal(row, results[label][key]), f"{label}: {key} differs from the whole run"


@pytest.mark.parametrize("name", ["M1", "M2", "M3", "M4"])
def test_the_stream_after_every_layer(name, ribovik_folders, tmp_path, monkeypatch):
    """The first layer that differs names the mechanism: the stream after every layer of one prompt, in float32."""
    folder, cfg, page, W, reqs, ref, unsure = ribovik_folders[name]
    ids = reqs["r2"]
    streams = []
    R.forward(ids, W, cfg, streams=streams)
    dump = tmp_path / "streams"
    dump.mkdir()
    monkeypatch.setenv("IMP_B200_DUMP_STREAM", str(dump))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids, "want": [len(ids) - 1]}], "end": ["a"]}]
    run_trace(folder, "float32", steps, round64(len(ids)), str(tmp_path / "out"), cfg["vocab"], page_size=page)
    assert len(streams) == len(cfg["layers"])
    for j, want in enumerate(streams):
        got = torch.from_numpy(np.fromfile(dump / f"step0_run{j}.f32", dtype="<f4").reshape(len(ids), cfg["width"]).copy())
        close(got, want, torch.float32, f"{name}: stream after layer {j}")


def test_embedding_norm_and_table_shared_with_the_head(ribovik_folders):
    """The logits of a first token when nothing but the embedding's norm, one layer and the last norm stand before them, against a
    table whose rows have very different lengths: the embedding is normalised, the head is not."""
    from imp_b200 import Engine, EngineConfig, StepEntry
    folder, cfg, page, W, reqs, ref, unsure = ribovik_folders["M4"]
    cfg = dict(cfg, layers=cfg["layers"][1:2])
    W = {k.replace("l1.", "l0."): v for k, v in W.items() if not k.startswith("l0.")}
    W["embed"] = (W["embed"] * torch.logspace(-2, 1, cfg["vocab"], dtype=torch.float64)[:, None]).to(torch.bfloat16).double()
    import tempfile
    with tempfile.TemporaryDirectory() as t:
        with open(os.path.join(t, "config.json"), "w") as f:
            json.dump(cfg, f)
        save_safetensors(os.path.join(t, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in W.items()})
        eng = Engine.from_folder(t, EngineConfig(compute_dtype="float32", kv_block_size=16, kv_cache_tokens=64, max_batch_size=2, max_seq_len=64, max_batch_tokens=64))
        ids = [0, 82, 40, 3, 0]
        got = torch.from_numpy(np.asarray(eng.step_tokens([StepEntry("a", ids, list(range(5)))])))
    close(got, R.forward(ids, W, cfg), torch.float32, "logits")


def test_greedy_generation_through_the_engine(ribovik_folders):
    """Prompts of unequal length through submit / schedule / step / sample with short prefill portions; the tokens are
    those of the plain model's argmax, and pages and slots all come back."""
    from imp_b200 import Engine, EngineConfig, GenerateParams
    folder, cfg, page, W, reqs, ref, unsure = ribovik_folders["M1"]
    g = torch.Generator().manual_seed(11)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (1, 7, 30, 12, 3)]

    def plain_generate(ids, n):
        ids, out = list(ids), []
        for _ in range(n):
            tok = int(torch.argmax(R.forward(ids, W, cfg)[-1]))
            out.append(tok)
            ids.append(tok)
        return out

    want = [plain_generate(p, 8) for p in prompts]
    for lookahead in (True, False):
        eng = Engine.from_folder(folder, EngineConfig(compute_dtype="float32", kv_block_size=page, max_batch_size=3, max_seq_len=256,
                                                      kv_cache_tokens=1024, max_batch_tokens=32, prefill_chunk_size=8, lookahead=lookahead))
        assert eng.generate(prompts, GenerateParams(max_tokens=8, temperature=0.0)) == want
        assert eng.free_pages() == eng.num_pages and not eng.has_work()
        info = eng.info()
        assert info["cache"]["free_slots"] == info["cache"]["slots"]
        assert info["model"]["graph_safe"]
    # the same with CUDA graphs for the decode steps in bfloat16: first tokens from well separated logits agree
    eng16 = Engine.from_folder(folder, EngineConfig(compute_dtype="bfloat16", kv_block_size=page, max_batch_size=4, max_seq_len=256,
                                                    kv_cache_tokens=1024, max_batch_tokens=64))
    got16 = eng16.generate(prompts, GenerateParams(max_tokens=8, temperature=0.0))
    for p, g16, w in zip(prompts, got16, want):
        lg = R.forward(p, W, cfg)[-1]
        top2 = torch.topk(lg, 2).values
        if float(top2[0] - top2[1]) > 0.1 * float(lg.abs().max()):
            assert g16[0] == w[0]


def test_unsummed_products_reach_the_norm(tmp_path):
    """Wide enough that a decode step's output products are cut over the contraction: the mixer's, the dense feed-forward's (its bias
    beside them) and the shared expert's (the routed rows beside them) are added by the norm behind them.  Decode graphs replay it."""
    from imp_b200 import Engine, EngineConfig, StepEntry
    cfg = {"architecture": "Ribovik", "vocab": 64, "width": 512, "norm": {"eps": 1e-5},
           "layers": [layer(att(16, 4, 64, 64, 16, 64, 1e4, YARN), DENSE(2048)),
                      layer(att(8, 2, 128, 128, 25, 128, 1e4, YARN), moe_config(4, 1, 2, 256, 2.0, (2048, 1.5)))]}
    W = make_weights(cfg, 5)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    Wd = {k: v.double() for k, v in W.items()}
    g = torch.Generator().manual_seed(1)
    seqs = {r: torch.randint(0, 64, (30,), generator=g).tolist() for r in "abc"}
    margins = {r: [] for r in seqs}
    want = {r: R.forward(ids, Wd, cfg, margins=margins[r]) for r, ids in seqs.items()}
    sure = {r: torch.stack(m).min(dim=0).values > 0.004 for r, m in margins.items()}
    for graphs in (False, True):
        eng = Engine.from_folder(str(tmp_path), EngineConfig(compute_dtype="bfloat16", kv_block_size=16, kv_cache_tokens=256, max_batch_size=4, max_seq_len=64,
                                                             max_batch_tokens=128, enable_cuda_graphs=graphs))
        eng.step_tokens([StepEntry(r, ids[:20], []) for r, ids in seqs.items()])
        rel = []
        for t in range(20, 30):
            got = eng.step_tokens([StepEntry(r, [ids[t]], [0]) for r, ids in seqs.items()])
            for i, r in enumerate(seqs):
                if sure[r][t]:
                    err = torch.from_numpy(np.asarray(got[i])).double() - want[r][t]
                    rel.append(float(err.pow(2).mean().sqrt() / want[r].pow(2).mean().sqrt()))
        assert len(rel) > 15 and max(rel) < 0.05, rel
        assert eng.info()["split_norm_calls"] > 0


def test_preemption_recomputes_and_chunks_need_few_pages(ribovik_folders):
    """Too few pages for every request at once: the newest is preempted and recomputed, and no token changes.  And where every layer
    is chunked, a request far longer than the pool runs in it."""
    from imp_b200 import Engine, EngineConfig, GenerateParams
    folder, cfg, page, W, reqs, ref, unsure = ribovik_folders["M3"]
    prompts = [reqs["r2"][:20], reqs["r4"][:25], reqs["r0"][:18]]
    outs = []
    for tokens in (1024, 72):
        eng = Engine.from_folder(folder, EngineConfig(compute_dtype="float32", kv_block_size=page, max_batch_size=3, max_seq_len=64,
                                                      kv_cache_tokens=tokens, max_batch_tokens=32))
        outs.append(eng.generate(prompts, GenerateParams(max_tokens=20, temperature=0.0)))
    assert outs[0] == outs[1]
    folder, cfg, page, W, reqs, ref, unsure = ribovik_folders["M4"]
    outs = []
    for tokens in (1024, 64):
        eng = Engine.from_folder(folder, EngineConfig(compute_dtype="float32", kv_block_size=page, max_batch_size=1, max_seq_len=512,
                                                      kv_cache_tokens=tokens, max_batch_tokens=16, prefill_chunk_size=16))
        outs.append(eng.generate([reqs["r0"]], GenerateParams(max_tokens=150, temperature=0.0)))
    assert len(outs[0][0]) == 150 and outs[0] == outs[1]


def test_command_line_with_a_checkpoint_and_with_random_weights(ribovik_folders, tmp_path):
    import subprocess
    import sys
    cli = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "imp-cli")
    folder, cfg, page, W, reqs, ref, unsure = ribovik_folders["M3"]
    ids, want = [5, 17, 3], []
    for _ in range(6):
        want.append(int(torch.argmax(R.forward(ids + want, W, cfg)[-1])))
    p = subprocess.run([sys.executable, cli, "--model", folder, "--prompt", "5,17,3", "--max-tokens", "6", "--temperature", "0",
                        "--dtype", "fp32", "--page-size", str(page), "--kv-pages", "64", "--max-seq-len", "128"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [int(x) for x in p.stdout.split()] == want
    only_config = tmp_path / "cfg"
    only_config.mkdir()
    (only_config / "config.json").write_text(json.dumps(MODELS["M1"][0]))
    b = subprocess.run([sys.executable, cli, "--model", str(only_config), "--random-weights", "--weights-seed", "3", "--kv-pages", "64",
                        "--max-seq-len", "256", "--bench", "--bench-pp", "48", "--max-tokens", "8", "--bench-reps", "2", "--bench-batch", "2"],
                       capture_output=True, text=True, timeout=600)
    assert b.returncode == 0, b.stderr[-2000:]
    assert "pp    96 tokens" in b.stderr and "tg    16 tokens" in b.stderr
