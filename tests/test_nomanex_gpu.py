"""Nomanex against the plain implementation (tests/plain/nomanex_plain.py): every mechanism alone through the part bench
(whole prompts, portions beside decoded tokens, slots and pages that are freed and used again, long decoding), whole models
through the trace runner in every way of cutting with the stream compared after every layer, and greedy generation
through the engine's own entry point and the command line.  Weights are made here so that a fault shows: decays spread over
(0, 1) and close to 1 with one loud key far back, a loud key just inside and just outside the attention's window, gates beyond
their clip, groups of experts that decide, and token pairs whose order matters."""
import json
import math
import os

import numpy as np
import pytest
import torch

from imp_b200.parts.bench import PartBench
from imp_b200.parts.plan import PartSpec
from imp_b200.parts.registry import mixer_cache_spec
from plain import nomanex_plain as N
from replay_helpers import collect, mixed, portions, round64, run_trace, tail_decode, whole
from safetensors_io import save_safetensors

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
NAME = {torch.float32: "float32", torch.bfloat16: "bfloat16"}
EPS = 2e-5


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


def pieces_beside_a_decoding_sequence(bench, part, xs, want, dtype, sizes, loose=1.0):
    """The first sequence in portions of `sizes`, the second one token at a time beside it."""
    done, outs, other = 0, [], 0
    for n in sizes:
        es, parts = [("p0", [1] * n, [])], [xs[0][done:done + n]]
        if other < xs[1].shape[0]:
            es.append(("p1", [1], []))
            parts.append(xs[1][other:other + 1])
        ctx = bench.prepare(es)
        o = run_part(bench, part, torch.cat(parts), ctx, bench.cache_view(0))
        bench.commit()
        outs.append(o[:n])
        if other < xs[1].shape[0]:
            close(o[n:], want[1][other:other + 1], dtype, f"decoded token {other}", loose=loose)
            other += 1
        done += n
    assert done == xs[0].shape[0]
    close(torch.cat(outs), want[0], dtype, "portions", loose=loose)


# ------------------------------------------------------------------ weights by checkpoint suffix
def gla_weights(d, c, seed):
    H, D, Dv, r = c["heads"], c["dim"], c["vdim"], c["rank"]
    s = 1.0 / math.sqrt(d)
    return {"q": rnd(H * D, d, seed=seed, scale=2 * s), "k": rnd(H * D, d, seed=seed + 1, scale=s), "v": rnd(H * Dv, d, seed=seed + 2, scale=s),
            "g": rnd(H * Dv, d, seed=seed + 3, scale=2 * s), "o": rnd(d, H * Dv, seed=seed + 4, scale=1.0 / math.sqrt(H * Dv)),
            "norm": 1 + 0.3 * rnd(Dv, seed=seed + 5), "a1": rnd(r, d, seed=seed + 6, scale=2 * s),
            "a2": rnd(H * D, r, seed=seed + 7, scale=2.0 / math.sqrt(r)), "a2.b": 1 + rnd(H * D, seed=seed + 8)}


def latent_weights(d, c, seed):
    H, D, R, Dv, C = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    s = 1.0 / math.sqrt(d)
    return {"q": rnd(H * (D + R), d, seed=seed, scale=2 * s), "dkv": rnd(C + R, d, seed=seed + 1, scale=2 * s),
            "dkv.norm": 1 + 0.3 * rnd(C, seed=seed + 2), "uk": rnd(H * D, C, seed=seed + 3, scale=1.0 / math.sqrt(C)),
            "uv": rnd(H * Dv, C, seed=seed + 4, scale=1.0 / math.sqrt(C)), "g": rnd(H * Dv, d, seed=seed + 5, scale=2 * s),
            "o": rnd(d, H * Dv, seed=seed + 6, scale=1.0 / math.sqrt(H * Dv))}


def dense_weights(d, ff, seed):
    s = 1.0 / math.sqrt(d)
    return {"gate": rnd(ff, d, seed=seed, scale=2 * s), "up": rnd(ff, d, seed=seed + 1, scale=2 * s), "down": rnd(d, ff, seed=seed + 2, scale=1.0 / math.sqrt(ff))}


def moe_weights(d, c, seed):
    E, F = c["router"]["experts"], c["expert"]["ff"]
    s = 1.0 / math.sqrt(d)
    w = {"router": rnd(E, d, seed=seed, scale=2 * s)}
    for e in range(E):
        w[f"e{e}.up"] = rnd(F, d, seed=seed + 10 * e + 1, scale=2 * s)
        w[f"e{e}.down"] = rnd(d, F, seed=seed + 10 * e + 2, scale=1.0 / math.sqrt(F))
    return w


GLA_NAMES = {"q": "q_proj", "k": "k_proj", "v": "v_proj", "g": "gate_proj", "o": "o_proj", "norm": "out_norm", "a1": "decay_down", "a2": "decay_up",
             "a2.b": "decay_bias"}
LATENT_NAMES = {"q": "q_proj", "dkv": "kv_down", "dkv.norm": "kv_norm", "uk": "k_up", "uv": "v_up", "g": "gate_proj", "o": "o_proj"}


def moe_names(c):
    names = {"router": "router"}
    for e in range(c["router"]["experts"]):
        names.update({f"e{e}.up": f"up_{e}", f"e{e}.down": f"down_{e}"})
    return names


def moe_params(d, c):
    r = c["router"]
    g = r.get("groups") or {}
    return {"hidden_size": d, "num_experts": r["experts"], "top_k": r["top"], "expert_size": c["expert"]["ff"], "expert": "relu2",
            "router_bias": False, "scores": "softmax_all", "num_groups": g.get("count", 0), "keep_groups": g.get("keep", 0), "group_score": "max"}


# ------------------------------------------------------------------------------ the norm without statistics
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [72, 70, 5, 4096])
def test_dynamic_tanh_with_a_branch_and_a_row_list(dtype, d):
    bench = PartBench(NAME[dtype], [], max_tokens=64)
    w, b = (1 + 0.3 * rnd(d, seed=1)).to(dtype), (0.4 * rnd(d, seed=2)).to(dtype)
    alpha = torch.tensor(0.7).to(dtype)
    part = bench.build("norm", PartSpec("dynamic_tanh", {"size": d}), {"weight": w.to(DEV), "bias": b.to(DEV), "alpha": alpha.to(DEV)})
    n = 37
    h, br = rnd(n, d, seed=3, scale=2.0), rnd(n, d, seed=4).to(dtype)
    total = h.double() + br.double()
    plain = lambda x: N.dynamic_tanh(x, alpha.double(), w.double(), b.double())
    ctx = bench.prepare([("a", [1] * n, [])])
    hd, brd = h.to(DEV), br.to(DEV)
    torch.cuda.synchronize()
    rows = torch.tensor([5, 0, 33], dtype=torch.int32, device=DEV)
    some = part.add_norm(hd, brd, rows=rows, ctx=ctx)
    bench.sync()
    some = some.clone()
    assert torch.equal(hd.cpu(), h), "a row list leaves the stream as it is"
    out = part.add_norm(hd, brd, ctx=ctx)
    bench.sync()
    close(hd, total, torch.float32, "stream")
    close(out, plain(total), dtype, "normalised")
    assert torch.equal(some, out[rows.long()])
    again = part.add_norm(hd, None, ctx=ctx)
    bench.sync()
    close(again, plain(total), dtype, "without a branch")


# ---------------------------------------------------------------- the embedding with a table of token pairs
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, buckets, mul_prev, mul_cur", [(72, 41, 7, 3), (70, 1, 5, 9), (64, 1000, 123457, 98765431), (8, 11, -4, 1)])
def test_bigram_embedding_over_portions_batches_and_reused_slots(dtype, d, buckets, mul_prev, mul_cur):
    V = 50
    c = {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}
    params = dict(c["bigram"], vocab_size=V, hidden_size=d)
    state = {"kind": "state", "tensors": [{"name": "last_token", "shape": [1], "dtype": "int32"}]}
    bench = PartBench(NAME[dtype], [state], slots=2)
    table, pairs = rnd(V, d, seed=1).to(dtype), rnd(buckets + 1, d, seed=2).to(dtype)
    part = bench.build("embedding", PartSpec("bigram_embedding", params), {"weight": table.to(DEV), "bigram": pairs.to(DEV)})
    W = {"embed": table.double(), "bigram": pairs.double()}
    g = torch.Generator().manual_seed(3)
    seqs = {r: torch.randint(0, V, (n,), generator=g).tolist() for r, n in (("a", 30), ("b", 9), ("c", 6))}
    want = {r: N.embed(ids, W, {"embedding": c}) for r, ids in seqs.items()}

    def step(entries):
        ctx = bench.prepare([(r, seqs[r][lo:hi], []) for r, lo, hi in entries])
        torch.cuda.synchronize()
        out = part.embed(ctx, bench.cache_view(0))
        bench.sync()
        out = out.cpu()
        bench.commit()
        at = 0
        for r, lo, hi in entries:
            close(out[at:at + hi - lo], want[r][lo:hi], torch.float32, f"{r} {lo}:{hi}")
            at += hi - lo

    step([("a", 0, 7), ("b", 0, 1)])
    step([("b", 1, 2), ("a", 7, 9)])
    step([("a", 9, 10)])                       # b sits out
    step([("b", 2, 9), ("a", 10, 29)])
    bench.end("b")
    step([("c", 0, 1), ("a", 29, 30)])         # b's slot again: its last token is not c's predecessor
    step([("c", 1, 6)])
    if buckets > 1:
        ids = seqs["a"]
        swapped = N.embed(ids, W, {"embedding": {"bigram": dict(c["bigram"], mul_prev=mul_cur, mul_cur=mul_prev)}})
        assert (swapped - want["a"]).abs().max() > 0.1, "the order of the pair matters"


# --------------------------------------------------------------------------- gated linear attention alone
GLA_CASES = [
    dict(d=72, heads=3, dim=8, vdim=24, rank=6, tau=4.0),
    dict(d=40, heads=1, dim=70, vdim=20, rank=1, tau=16.0),              # one head; a key size that is no multiple of the lanes' rows; an inner size of 1
    dict(d=64, heads=2, dim=128, vdim=40, rank=24, tau=9.0),             # value columns beyond one block of 32
    dict(d=48, heads=5, dim=12, vdim=12, rank=7, tau=1.0),
    dict(d=64, heads=2, dim=33, vdim=96, rank=16, tau=30.0),             # an odd key size
    dict(d=56, heads=1, dim=200, vdim=9, rank=5, tau=2.0),
]


def gla_setup(dtype, case, slots=4, seed=200, w=None):
    c = {k: case[k] for k in ("heads", "dim", "vdim", "rank", "tau")}
    d = case["d"]
    params = {"hidden_size": d, "num_heads": c["heads"], "key_dim": c["dim"], "value_dim": c["vdim"], "tau": c["tau"], "norm_eps": EPS}
    bench = PartBench(NAME[dtype], [mixer_cache_spec("gated_linear_attention", params)], slots=slots, max_tokens=1024, max_seq_len=1024)
    w = {k: v.to(dtype) for k, v in (w or gla_weights(d, c, seed)).items()}
    part = bench.build("mixer", PartSpec("gated_linear_attention", params), {GLA_NAMES[k]: v.to(DEV) for k, v in w.items()})
    W = {"m." + k: v.double() for k, v in w.items()}
    return bench, part, (lambda x: N.gla(x.double(), W, "m.", c, EPS)), W, c


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", GLA_CASES)
def test_gla_whole_portions_decoding_and_reused_slots(dtype, case):
    bench, part, plain, _, _ = gla_setup(dtype, case, slots=2)
    d = case["d"]
    lengths = [75, 9]
    xs = [rnd(n, d, seed=40 + i).to(dtype) for i, n in enumerate(lengths)]
    want = [plain(x) for x in xs]
    ctx = bench.prepare([(f"w{i}", [1] * n, []) for i, n in enumerate(lengths)])
    out = run_part(bench, part, torch.cat(xs), ctx, bench.cache_view(0))
    bench.commit()
    # a single head's first read-out is sign(q . k) v / rms(v): position 0 is judged in float32 only
    skip = 1 if dtype == torch.bfloat16 else 0
    close(out[skip:75], want[0][skip:], dtype, "whole", loose=3.0)
    close(out[75 + skip:], want[1][skip:], dtype, "whole, second sequence", loose=3.0)
    bench.end("w0")
    bench.end("w1")                       # both slots go back; the next requests start from a state of zeros
    if dtype == torch.float32:
        pieces_beside_a_decoding_sequence(bench, part, xs, want, dtype, (10, 2, 1, 1, 20, 1, 4, 2, 2, 1, 17, 3, 1, 1, 1, 1, 1, 1, 2, 3))
    else:
        p = in_pieces(bench, part, xs[0], (10, 2, 1, 1, 20, 1, 4, 2, 2, 1, 17, 3, 1, 1, 1, 1, 1, 1, 2, 3))
        close(p, out[:75], dtype, "portions against the whole prompt")


def test_gla_pieces_change_no_bit_and_what_it_rests_on_shows():
    bench, part, plain, W, c = gla_setup(torch.float32, GLA_CASES[0])
    x = rnd(50, 72, seed=77)
    whole_out = in_pieces(bench, part, x, (50,))
    want = plain(x)
    close(whole_out, want, torch.float32, "whole")
    assert torch.equal(in_pieces(bench, part, x, (3, 2, 1, 30, 1, 13), "b"), whole_out), "prompt kernels and the decode kernel agree to the bit"
    assert torch.equal(in_pieces(bench, part, x, (1,) * 50, "c"), whole_out)
    far = lambda other: float((other - want).abs().max()) > 0.02 * float(want.abs().max())
    assert far(N.gla(x.double(), W, "m.", dict(c, tau=3.0), EPS)), "tau"
    for k in ("a2.b", "norm"):
        other = dict(W)
        other["m." + k] = torch.zeros_like(W["m." + k]) if k == "a2.b" else torch.ones_like(W["m." + k])
        assert far(N.gla(x.double(), other, "m.", c, EPS)), k


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
def test_gla_finds_one_loud_key_far_back(dtype, decoded):
    """Decays close to 1, quiet keys, one loud one 500 tokens before the end: it carries the read-out, so a lost or cut state shows."""
    case = dict(d=48, heads=2, dim=16, vdim=24, rank=4, tau=16.0)
    c = {k: case[k] for k in ("heads", "dim", "vdim", "rank", "tau")}
    w = gla_weights(48, c, 300)
    w["a2.b"] = torch.full_like(w["a2.b"], 5.0)          # alpha about 0.9996
    w["k"] = w["k"] * 0.1
    w["q"] = w["q"] * 0.1
    w["k"][::16, 0] += 3.0                               # channel 0 of every head follows input 0
    w["q"][::16, 1] += 3.0
    bench, part, plain, W, _ = gla_setup(dtype, case, w=w)
    T, at = 560, 47
    x = rnd(T, 48, seed=301, scale=0.5)
    x[:, 0] = 0.0
    x[:, 1] = 1.0
    x[at, 0] = 8.0
    x = x.to(dtype)
    want = plain(x)
    quiet = x.clone()
    quiet[at, 0] = 0.0
    assert (plain(quiet)[-1] - want[-1]).abs().max() > 0.5 * want[-1].abs().max(), "the last token hangs on the loud one"
    out = in_pieces(bench, part, x, (T - 40,) + (1,) * 40 if decoded else (300, 2, T - 302))
    close(out[at:], want[at:], dtype, "after the loud key", loose=2.0)


def test_gla_long_decoding_carries_the_state():
    bench, part, plain, _, _ = gla_setup(torch.float32, GLA_CASES[2])
    x = rnd(300, 64, seed=78)
    close(in_pieces(bench, part, x, (1,) * 300), plain(x), torch.float32, "300 tokens one by one", loose=1.0)


# ----------------------------------------------------------------------------------- latent attention alone
LATENT_CASES = [
    dict(d=72, heads=5, dim=24, rot_dim=8, vdim=40, kv_rank=56, window=10, base=100.0, page=4),      # cached vectors of 64
    dict(d=64, heads=4, dim=32, rot_dim=32, vdim=32, kv_rank=96, window=50, base=10000.0, page=16),  # of 128
    dict(d=40, heads=2, dim=12, rot_dim=4, vdim=20, kv_rank=30, window=0, base=7.0, page=8),         # of 34, padded to 48; no window
    dict(d=48, heads=3, dim=64, rot_dim=16, vdim=96, kv_rank=160, window=33, base=500.0, page=16),   # of 176; a window that is no multiple of a page
    dict(d=32, heads=1, dim=16, rot_dim=2, vdim=16, kv_rank=14, window=1, base=7.0, page=16),        # one head, one rotated pair, a token sees itself
    dict(d=48, heads=20, dim=20, rot_dim=6, vdim=8, kv_rank=255, window=64, base=50.0, page=16),     # of 261, beyond the tensor-core kernels; a window of whole pages
]


def latent_setup(dtype, case, w=None, scale=None, seed=100):
    c = {k: case[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
    c["scale"] = scale or 1.0 / math.sqrt(c["dim"] + c["rot_dim"])
    c["rot"] = {"base": case["base"], "dims": case["rot_dim"]}
    if case["window"]:
        c["mask"] = {"size": case["window"]}
    params = {"hidden_size": case["d"], "num_heads": c["heads"], "head_dim": c["dim"], "rot_dim": c["rot_dim"], "rot_dims": c["rot_dim"],
              "value_dim": c["vdim"], "kv_rank": c["kv_rank"], "q_rank": 0, "scale": c["scale"], "norm_eps": EPS, "rot_base": case["base"],
              "rot_pairing": "neighbours", "window": case["window"], "out_gate": True, "pad_cache": True, "max_positions": 2048}
    bench = PartBench(NAME[dtype], [mixer_cache_spec("latent_attention", params)], page_size=case["page"], num_pages=2048 // case["page"],
                      max_tokens=1024, max_seq_len=1024)
    w = {k: v.to(dtype) for k, v in (w or latent_weights(case["d"], c, seed)).items()}
    part = bench.build("mixer", PartSpec("latent_attention", params), {LATENT_NAMES[k]: v.to(DEV) for k, v in w.items()})
    return bench, part, c, {"m." + k: v.double() for k, v in w.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", LATENT_CASES)
def test_latent_attention_whole_portions_decoding_and_reused_pages(dtype, case):
    bench, part, c, W = latent_setup(dtype, case)
    lengths = [93, 11]
    xs = [rnd(n, case["d"], seed=20 + i).to(dtype) for i, n in enumerate(lengths)]
    want = [N.latent_attention(x.double(), W, "m.", c, EPS) for x in xs]
    ctx = bench.prepare([(f"w{i}", [1] * n, []) for i, n in enumerate(lengths)])
    out = run_part(bench, part, torch.cat(xs), ctx, bench.cache_view(0))
    bench.commit()
    close(out[:93], want[0], dtype, "whole", loose=2.0)
    close(out[93:], want[1], dtype, "whole, second sequence", loose=2.0)
    bench.end("w0")
    bench.end("w1")                       # their pages come out first for the next requests
    pieces_beside_a_decoding_sequence(bench, part, xs, want, dtype, (10, 2, 20, 1, 4, 2, 33, 1, 1, 1, 2, 16), loose=2.0)


def test_what_latent_attention_rests_on_shows_in_the_plain_results():
    case = LATENT_CASES[0]
    c = {k: case[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
    c.update(scale=0.4, rot={"base": 100.0, "dims": 8}, mask={"size": 10})
    W = {"m." + k: v.double() for k, v in latent_weights(case["d"], c, seed=100).items()}
    x = rnd(60, case["d"], seed=20).double()
    run = lambda W=W, c=c, **kw: N.latent_attention(x, W, "m.", c, EPS, **kw)
    want = run()
    far = lambda other: float((other - want).abs().max()) > 0.02 * float(want.abs().max())
    assert far(run(c=dict(c, mask={"size": 11}))), "one more key in the window"
    assert far(run(c=dict(c, scale=0.3))), "the scale"
    assert far(run(c=dict(c, rot={"base": 90.0, "dims": 8}))), "the rotation's base"
    assert far(run(positions=torch.arange(60) * 2)), "positions"
    for k in ("dkv.norm", "g"):
        other = dict(W)
        other["m." + k] = torch.ones_like(W["m." + k]) if k == "dkv.norm" else torch.zeros_like(W["m." + k])
        assert far(run(W=other)), k


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
def test_a_loud_key_just_inside_and_just_outside_the_window_and_far_away(dtype, decoded):
    """The token at `at` is the key every later token looks for.  The query at at + window - 1 still sees it, the one at
    at + window does not; without a window a query 600 tokens later finds it among all the others.  In a prompt, and with
    the last tokens decoded one by one."""
    for window, T, at in ((37, 120, 50), (64, 150, 63), (0, 640, 3)):
        case = dict(d=48, heads=3, dim=16, rot_dim=4, vdim=24, kv_rank=44, window=window, base=1e6, page=16)
        c = {k: case[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
        w = latent_weights(48, c, 300)
        w["q"] = w["q"] * 0.2
        for h in range(3):
            w["q"][h * 20, 1] += 4.0                      # entry 0 of every head's plain query follows input 1, which is 1 everywhere
            w["uk"][h * 16] = 0.0
            w["uk"][h * 16, 0] = 1.5                      # and meets entry 0 of the latent, which follows input 0
        w["dkv"][0] = 0.0
        w["dkv"][0, 0] = 3.0
        bench, part, c, W = latent_setup(dtype, case, w=w, scale=1.0)
        x = rnd(T, 48, seed=301, scale=0.5)
        x[:, 0] = 0.0
        x[:, 1] = 1.0
        x[at, 0] = 6.0
        x = x.to(dtype)
        want = N.latent_attention(x.double(), W, "m.", c, EPS)
        quiet = x.clone()
        quiet[at, 0] = 0.0
        moved = (want - N.latent_attention(quiet.double(), W, "m.", c, EPS)).abs().amax(dim=-1) / want.abs().max()
        if window:
            assert moved[at + window - 1] > 0.2 and moved[at + window] < 1e-9, "the plain result hangs on the key exactly inside the window"
        else:
            assert moved[T - 1] > 0.2, "the plain result hangs on the far key"
        n_tail = 40 if decoded else 0
        if decoded and window:
            assert T - n_tail <= at + window - 1, "the edge is passed while decoding"
        out = in_pieces(bench, part, x, (T - n_tail,) + (1,) * n_tail)
        close(out, want, dtype, f"window {window}", loose=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kv_rank", [56, 120, 232])
def test_long_portions_with_window_edges_inside_the_kernels_tiles(dtype, kv_rank):
    """Portions of hundreds of tokens take the tiled kernels (cached vectors of 64, 128 and 240); the window's edge falls inside their tiles."""
    case = dict(d=64, heads=2, dim=64, rot_dim=8, vdim=64, kv_rank=kv_rank, window=150, base=1000.0, page=16)
    bench, part, c, W = latent_setup(dtype, case)
    x = rnd(700, 64, seed=21).to(dtype)
    want = N.latent_attention(x.double(), W, "m.", c, EPS)
    close(in_pieces(bench, part, x, (300, 257, 2, 141)), want, dtype, "long portions", loose=2.0)


# ------------------------------------------------------------------------------------- feed-forwards alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d, ff, limit", [(72, 100, 1.5), (64, 256, 0.6), (40, 37, 7.0)])
def test_clipped_gate_feed_forward(dtype, d, ff, limit):
    bench = PartBench(NAME[dtype], [], max_tokens=256)
    w = {k: v.to(dtype) for k, v in dense_weights(d, ff, seed=600).items()}
    part = bench.build("feed_forward", PartSpec("gated_mlp", {"hidden_size": d, "intermediate_size": ff, "activation": "clipped", "limit": limit}),
                       {"gate_proj": w["gate"].to(DEV), "up_proj": w["up"].to(DEV), "down_proj": w["down"].to(DEV)})
    W = {"f." + k: v.double() for k, v in w.items()}
    x = rnd(150, d, seed=601).to(dtype)
    want = N.dense_ff(x.double(), W, "f.", {"limit": limit})
    if limit < 5:
        assert (N.dense_ff(x.double(), W, "f.", {"limit": limit * 1.2}) - want).abs().max() > 0.02 * want.abs().max(), "the clip decides"
    out = run_part(bench, part, x, bench.prepare([("a", [1] * 150, [])]))
    close(out, want, dtype, "whole", loose=2.0)
    two = run_part(bench, part, x[5:7], bench.prepare([("b", [1] * 2, [])]))
    close(two, want[5:7], dtype, "two tokens", loose=2.0)
    if dtype == torch.float32:
        assert torch.equal(two, out[5:7]), "a token's result does not depend on its neighbours"


MOE_CASES = [
    dict(d=72, experts=12, top=3, ff=20, groups=(4, 2)),
    dict(d=64, experts=6, top=1, ff=32, groups=None),              # one expert a token, no groups
    dict(d=40, experts=15, top=3, ff=24, groups=(15, 5)),          # groups of one expert
    dict(d=48, experts=8, top=4, ff=16, groups=(2, 2)),            # every group kept
    dict(d=50, experts=70, top=6, ff=9, groups=(7, 3)),            # sizes that are multiples of nothing
    dict(d=48, experts=8, top=8, ff=16, groups=(1, 1)),            # every expert chosen: the weights sum to one
    dict(d=32, experts=1, top=1, ff=8, groups=None),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", MOE_CASES)
def test_routed_experts_with_softmax_scores_and_groups(dtype, case):
    c = {"router": {"experts": case["experts"], "top": case["top"]}, "expert": {"ff": case["ff"]}}
    if case["groups"]:
        c["router"]["groups"] = {"count": case["groups"][0], "keep": case["groups"][1]}
    d = case["d"]
    w = {k: v.to(dtype) for k, v in moe_weights(d, c, seed=500).items()}
    bench = PartBench(NAME[dtype], [], max_tokens=256)
    names = moe_names(c)
    part = bench.build("feed_forward", PartSpec("routed_experts", moe_params(d, c)), {names[k]: v.to(DEV) for k, v in w.items()})
    W = {"f." + k: v.double() for k, v in w.items()}
    x = rnd(150, d, seed=501).to(dtype)
    want = N.moe(x.double(), W, "f.", c)
    sure = N.route_margin(x.double(), W, "f.", c) > 1e-3           # rows whose choice hangs on less than rounding are not judged
    assert sure.sum() > 120
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
    if case["groups"] and case["groups"][1] < case["groups"][0] and case["experts"] > case["groups"][0]:
        free = dict(c, router=dict(c["router"], groups=None))
        assert (N.moe(x.double(), W, "f.", free) - want).abs().max() > 0.05 * want.abs().max(), "the groups decide"


def test_experts_of_long_portions_take_the_dense_products():
    """Enough work an expert that its rows go to the tensor-memory products with the squared relu in their epilogue."""
    d, c = 512, {"router": {"experts": 2, "top": 1}, "expert": {"ff": 1024}}
    w = {k: v.to(torch.bfloat16) for k, v in moe_weights(d, c, seed=510).items()}
    bench = PartBench("bfloat16", [], max_tokens=9216, max_seq_len=9216)
    names = moe_names(c)
    part = bench.build("feed_forward", PartSpec("routed_experts", moe_params(d, c)), {names[k]: v.to(DEV) for k, v in w.items()})
    x = rnd(9000, d, seed=511).to(torch.bfloat16)
    out = run_part(bench, part, x, bench.prepare([("a", [1] * 9000, [])]))
    few = run_part(bench, part, x[:200], bench.prepare([("b", [1] * 200, [])]))     # the grouped products
    close(out[:200], few, torch.bfloat16, "dense against grouped products")
    W = {"f." + k: v.float() for k, v in w.items()}
    at = torch.arange(0, 9000, 450)
    sure = N.route_margin(x[at].float(), W, "f.", c) > 1e-2
    close(out[at.to(DEV)].cpu()[sure], N.moe(x[at].float(), W, "f.", c)[sure], torch.bfloat16, "rows of the long portion", loose=2.0)


# --------------------------------------------------------------- whole models
def gla(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}


def lat(heads, dim, rot_dim, vdim, kv_rank, window, base=10000.0, scale=None):
    c = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale or 1.0 / math.sqrt(dim + rot_dim),
         "rot": {"base": base, "dims": rot_dim}}
    if window:
        c["mask"] = {"size": window}
    return c


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe_cfg(experts, top, ff, groups=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def like(layers, j):
    return dict(layers[j], weights_of=j)


def with_shared(layers, order):
    """Layers by number; a number that came before stands for a layer that uses that one's weights."""
    out, first = [], {}
    for i in order:
        if i in first:
            out.append(like(out, first[i]))
        else:
            first[i] = len(out)
            out.append(dict(layers[i]))
    return out


# M1: both mixers, shared weights of both kinds (an attention layer with two caches), windows of 24 (one and a half pages) and 9,
# grouped experts.  M2: nothing shared, m = 1, no window, no groups, an attention layer without feed-forward first,
# pages of 4.  M3: attention only (no recurrent layer), a layer used four times, one bucket.  M4: gated linear attention only, no
# token pairs, sizes that are multiples of nothing.
L1 = [{"type": "gla", "mixer": gla(3, 16, 24, 5.0, 6), "mlp": dense(72, 1.5)},
      {"type": "latent_attention", "mixer": lat(5, 16, 8, 20, 40, 24, base=100.0), "mlp": moe_cfg(12, 3, 24, (4, 2))},
      {"type": "gla", "mixer": gla(2, 40, 16, 16.0, 9), "mlp": None},
      {"type": "latent_attention", "mixer": lat(2, 24, 4, 32, 60, 9), "mlp": dense(40, 3.0)}]
MODELS = {
    "M1": ({"architecture": "Nomanex", "vocab": 97, "width": 64, "norm": {"eps": 3e-5}, "residual_mult": 0.5,
            "embedding": {"bigram": {"buckets": 211, "mul_prev": 37, "mul_cur": 11}}, "layers": with_shared(L1, [0, 1, 0, 2, 3, 1, 0])}, 16),
    "M2": ({"architecture": "Nomanex", "vocab": 151, "width": 112, "norm": {"eps": 1e-6}, "residual_mult": 1.0,
            "embedding": {"bigram": {"buckets": 75, "mul_prev": 13, "mul_cur": 29}},
            "layers": [{"type": "latent_attention", "mixer": lat(3, 32, 16, 40, 112, 0), "mlp": None},
                       {"type": "gla", "mixer": gla(4, 24, 24, 8.0, 16), "mlp": moe_cfg(6, 1, 32)},
                       {"type": "latent_attention", "mixer": lat(4, 20, 12, 28, 50, 100, base=300.0), "mlp": moe_cfg(16, 4, 24, (16, 5))}]}, 4),
    "M3": ({"architecture": "Nomanex", "vocab": 130, "width": 96, "norm": {"eps": 1e-5}, "residual_mult": 0.4,
            "embedding": {"bigram": {"buckets": 1, "mul_prev": 5, "mul_cur": 7}},
            "layers": with_shared([{"type": "latent_attention", "mixer": lat(6, 16, 16, 16, 48, 40), "mlp": moe_cfg(8, 2, 32, (2, 1))},
                                   {"type": "latent_attention", "mixer": lat(2, 48, 8, 32, 248, 64, base=50.0), "mlp": dense(128, 2.5)}], [0, 1, 0, 0, 0])}, 16),
    "M4": ({"architecture": "Nomanex", "vocab": 83, "width": 70, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
            "layers": [{"type": "gla", "mixer": gla(2, 9, 11, 3.0, 5), "mlp": dense(50, 1.2)},
                       {"type": "gla", "mixer": gla(1, 70, 37, 12.0, 3), "mlp": moe_cfg(3, 2, 12)}]}, 8),
}
LENGTHS = {"M1": (1, 23, 75, 40, 130, 64), "M2": (150, 2, 33, 201, 64, 97), "M3": (70, 5, 140, 31, 64, 2), "M4": (45, 3, 70, 20, 64, 9)}


def make_weights(cfg, seed):
    d = cfg["width"]
    W = {"embed": rnd(cfg["vocab"], d, seed=seed), "head": rnd(cfg["vocab"], d, seed=seed + 3, scale=1.0 / math.sqrt(d))}
    if cfg.get("embedding"):
        W["bigram"] = rnd(cfg["embedding"]["bigram"]["buckets"] + 1, d, seed=seed + 4, scale=0.7)

    def norm(name, s):
        W[name], W[name + ".b"], W[name + ".alpha"] = 1 + 0.2 * rnd(d, seed=s), 0.3 * rnd(d, seed=s + 1), torch.tensor(0.5 + 0.2 * (s % 3))

    norm("final.norm", seed + 1)
    for i, lay in enumerate(cfg["layers"]):
        if lay.get("weights_of") is not None:
            continue
        p, s = f"l{i}.", seed + 1000 * (i + 1)
        norm(p + "norm1", s)
        m = lay["mixer"]
        for k, v in (latent_weights if lay["type"] == "latent_attention" else gla_weights)(d, m, s + 30).items():
            W[p + "mix." + k] = v
        if lay["mlp"]:
            for k, v in (dense_weights(d, lay["mlp"]["ff"], s + 80) if lay["mlp"]["kind"] == "dense" else moe_weights(d, lay["mlp"], s + 80)).items():
                W[p + "mlp." + k] = v
    return {k: v.to(torch.bfloat16) for k, v in W.items()}


def file_config(cfg):
    """The configuration as a checkpoint has it: the inner size of a decay is no key."""
    return dict(cfg, layers=[dict(l, mixer={k: v for k, v in l["mixer"].items() if k != "rank"}) for l in cfg["layers"]])


@pytest.fixture(scope="module")
def nomanex_folders(tmp_path_factory):
    out = {}
    for n, (name, (cfg, page)) in enumerate(MODELS.items()):
        folder = str(tmp_path_factory.mktemp(f"nomanex_{name}"))
        W = make_weights(cfg, seed=70 + n)
        with open(os.path.join(folder, "config.json"), "w") as f:
            json.dump(file_config(cfg), f)
        save_safetensors(os.path.join(folder, "model.safetensors"), W)
        g = torch.Generator().manual_seed(n)
        reqs = {f"r{i}": torch.randint(0, cfg["vocab"], (m,), generator=g).tolist() for i, m in enumerate(LENGTHS[name])}
        Wd = {k: v.double() for k, v in W.items()}
        ref, unsure = {}, set()
        for rid, ids in reqs.items():
            margins = []
            ref[rid] = N.forward(ids, Wd, cfg, margins=margins).float().numpy()
            if margins:
                # tokens whose choice of experts hangs on less than 16-bit rounding moves a router's logits
                close_call = torch.stack(margins).min(dim=0).values < 0.03
                unsure.update((rid, int(p)) for p in torch.nonzero(close_call)[:, 0])
        out[name] = (folder, cfg, page, Wd, reqs, ref, unsure)
    return out


def check_rows(rows, reqs, ref, dtype, label="", unsure=()):
    """float32: every logit to 1e-4 of the largest.  bfloat16: a row's root-mean-square error against the root mean square
    of all logits is at most 5 % for 95 of 100 rows and 30 % for every row; rows in `unsure` (a router's choice for that
    token hangs on less than the rounding of its 16-bit input moves a logit) and first tokens (a head's first read-out is
    sign(q . k) v / rms(v): its sign may hang on rounding) are not judged."""
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
            elif (rid, p) not in unsure and p > 0:
                rel.append(float(np.sqrt(np.mean(err ** 2))) / rms_all)
                assert rel[-1] <= 0.30, f"{label}: request {rid} position {p}: rms error {rel[-1]:.3g} of the logits' rms in {dtype}"
            n += 1
    assert n == sum(len(v) for v in reqs.values())
    if rel:
        assert float(np.quantile(rel, 0.95)) <= 0.05, f"{label}: 95th percentile of the rows' rms error {np.quantile(rel, 0.95):.3g} in {dtype}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["M1", "M2", "M3", "M4"])
def test_replay_all_ways_of_cutting(name, dtype, nomanex_folders, tmp_path):
    folder, cfg, page, W, reqs, ref, unsure = nomanex_folders[name]
    assert len(unsure) < sum(len(v) for v in reqs.values()) // 3
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
def test_the_stream_after_every_layer(name, nomanex_folders, tmp_path, monkeypatch):
    """The first layer that differs names the mechanism: the stream after every layer of one prompt, in float32."""
    folder, cfg, page, W, reqs, ref, unsure = nomanex_folders[name]
    ids = reqs["r2"]
    streams = []
    N.forward(ids, W, cfg, streams=streams)
    dump = tmp_path / "streams"
    dump.mkdir()
    monkeypatch.setenv("IMP_B200_DUMP_STREAM", str(dump))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids, "want": [len(ids) - 1]}], "end": ["a"]}]
    run_trace(folder, "float32", steps, round64(len(ids)), str(tmp_path / "out"), cfg["vocab"], page_size=page)
    assert len(streams) == len(cfg["layers"])
    for j, want in enumerate(streams):
        got = torch.from_numpy(np.fromfile(dump / f"step0_run{j}.f32", dtype="<f4").reshape(len(ids), cfg["width"]).copy())
        close(got, want, torch.float32, f"{name}: stream after layer {j} ({cfg['layers'][j]['type']})")


def test_greedy_generation_through_the_engine(nomanex_folders):
    """Prompts of unequal length through submit / schedule / step / sample with short prefill portions; the tokens are
    those of the plain model's argmax, and pages and slots all come back."""
    from imp_b200 import Engine, EngineConfig, GenerateParams
    folder, cfg, page, W, reqs, ref, unsure = nomanex_folders["M1"]
    g = torch.Generator().manual_seed(11)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (1, 7, 30, 12, 3)]

    def plain_generate(ids, n):
        ids, out = list(ids), []
        for _ in range(n):
            tok = int(torch.argmax(N.forward(ids, W, cfg)[-1]))
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
        lg = N.forward(p, W, cfg)[-1]
        top2 = torch.topk(lg, 2).values
        if float(top2[0] - top2[1]) > 0.1 * float(lg.abs().max()):
            assert g16[0] == w[0]


def test_blocks_sum_worked_out_for_a_norm_that_takes_plain_branches(nomanex_folders):
    """The block alone hands on one tensor: m times the sum of its two sublayers."""
    dtype, d, m = torch.float32, 64, 0.7
    bench = PartBench(NAME[dtype], [], max_tokens=64)
    w, b, alpha = 1 + 0.3 * rnd(d, seed=1), 0.4 * rnd(d, seed=2), torch.tensor(0.7)
    f, c = dense_weights(d, 40, 3), {"router": {"experts": 5, "top": 2}, "expert": {"ff": 16}}
    e = moe_weights(d, c, 9)
    spec = mixer_cache_spec("gated_linear_attention", {"hidden_size": d, "num_heads": 2, "key_dim": 8, "value_dim": 8, "tau": 4.0})
    x = rnd(20, d, seed=5)
    h = N.dynamic_tanh(x.double(), 0.7 * torch.ones((), dtype=torch.float64), w.double(), b.double())
    g = gla_weights(d, gla(2, 8, 8, 4.0, 3), 30)
    G = {"m." + k: v.double() for k, v in g.items()}
    mix = N.gla(h, G, "m.", gla(2, 8, 8, 4.0, 3), EPS)
    for kind in ("dense", "moe", None):
        bench = PartBench(NAME[dtype], [spec], max_tokens=64)
        norm = bench.build("norm", PartSpec("dynamic_tanh", {"size": d}), {"weight": w.to(DEV), "bias": b.to(DEV), "alpha": alpha.to(DEV)})
        mixer = bench.build("mixer", PartSpec("gated_linear_attention", {"hidden_size": d, "num_heads": 2, "key_dim": 8, "value_dim": 8, "tau": 4.0, "norm_eps": EPS}),
                            {GLA_NAMES[k]: v.to(DEV) for k, v in g.items()})
        parts = {"norm": norm, "mixer": mixer}
        want = mix
        if kind == "dense":
            parts["feed_forward"] = bench.build("feed_forward", PartSpec("gated_mlp", {"hidden_size": d, "intermediate_size": 40, "activation": "clipped", "limit": 1.0}),
                                                {"gate_proj": f["gate"].to(DEV), "up_proj": f["up"].to(DEV), "down_proj": f["down"].to(DEV)})
            want = mix + N.dense_ff(h, {"f." + k: v.double() for k, v in f.items()}, "f.", {"limit": 1.0})
        elif kind == "moe":
            parts["feed_forward"] = bench.build("feed_forward", PartSpec("routed_experts", moe_params(d, c)), {moe_names(c)[k]: v.to(DEV) for k, v in e.items()})
            want = mix + N.moe(h, {"f." + k: v.double() for k, v in e.items()}, "f.", c)
        block = bench.build_block("parallel", parts, {"residual_mult": m, "has_ffn": kind is not None})
        ctx = bench.prepare([("a", [1] * 20, [])])
        torch.cuda.synchronize()
        out = block.block_forward(x.to(DEV), None, ctx, bench.cache_view(0))
        bench.sync()
        close(out, m * want, dtype, f"feed-forward {kind}")


def test_unsummed_products_of_both_sublayers_reach_the_norm(tmp_path):
    """Wide enough that a decode step's output products are cut over the contraction: their parts, both sublayers' at once,
    are added by the next norm."""
    from imp_b200 import Engine, EngineConfig, StepEntry
    cfg = {"architecture": "Nomanex", "vocab": 64, "width": 512, "norm": {"eps": 1e-5}, "residual_mult": 0.3,
           "embedding": {"bigram": {"buckets": 19, "mul_prev": 3, "mul_cur": 5}},
           "layers": [{"type": "gla", "mixer": gla(8, 64, 128, 8.0, 16), "mlp": dense(2048, 2.0)},
                      {"type": "latent_attention", "mixer": lat(16, 64, 16, 64, 112, 20), "mlp": moe_cfg(4, 2, 256)},
                      {"type": "gla", "mixer": gla(8, 64, 128, 8.0, 16), "mlp": None}]}
    W = make_weights(cfg, 5)
    (tmp_path / "config.json").write_text(json.dumps(file_config(cfg)))
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    Wd = {k: v.double() for k, v in W.items()}
    g = torch.Generator().manual_seed(1)
    seqs = {r: torch.randint(0, 64, (30,), generator=g).tolist() for r in "abc"}
    margins = {r: [] for r in seqs}
    want = {r: N.forward(ids, Wd, cfg, margins=margins[r]) for r, ids in seqs.items()}
    sure = {r: torch.stack(m).min(dim=0).values > 0.03 for r, m in margins.items()}
    eng = Engine.from_folder(str(tmp_path), EngineConfig(compute_dtype="bfloat16", kv_block_size=16, kv_cache_tokens=256, max_batch_size=4, max_seq_len=64,
                                                         max_batch_tokens=128))
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


def test_preemption_recomputes_state_and_predecessor(nomanex_folders):
    """Too few pages for every request at once: the newest is preempted and recomputed, and no token changes."""
    from imp_b200 import Engine, EngineConfig, GenerateParams
    folder, cfg, page, W, reqs, ref, unsure = nomanex_folders["M2"]
    prompts = [reqs["r2"][:20], reqs["r4"][:25], reqs["r5"][:18]]
    outs = []
    for tokens in (1024, 72):
        eng = Engine.from_folder(folder, EngineConfig(compute_dtype="float32", kv_block_size=page, max_batch_size=3, max_seq_len=64,
                                                      kv_cache_tokens=tokens, max_batch_tokens=32))
        outs.append(eng.generate(prompts, GenerateParams(max_tokens=20, temperature=0.0)))
    assert outs[0] == outs[1]


def test_command_line_with_a_checkpoint_and_with_random_weights(nomanex_folders, tmp_path):
    import subprocess
    import sys
    cli = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "imp-cli")
    folder, cfg, page, W, reqs, ref, unsure = nomanex_folders["M3"]
    ids, want = [5, 17, 3], []
    for _ in range(6):
        want.append(int(torch.argmax(N.forward(ids + want, W, cfg)[-1])))
    p = subprocess.run([sys.executable, cli, "--model", folder, "--prompt", "5,17,3", "--max-tokens", "6", "--temperature", "0",
                        "--dtype", "fp32", "--page-size", str(page), "--kv-pages", "64", "--max-seq-len", "128"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [int(x) for x in p.stdout.split()] == want
    only_config = tmp_path / "cfg"
    only_config.mkdir()
    random_cfg = MODELS["M1"][0]
    random_cfg = dict(random_cfg, layers=[dict(l, mixer={("decay_rank" if k == "rank" else k): v for k, v in l["mixer"].items()}) for l in random_cfg["layers"]])
    (only_config / "config.json").write_text(json.dumps(random_cfg))
    b = subprocess.run([sys.executable, cli, "--model", str(only_config), "--random-weights", "--weights-seed", "3", "--kv-pages", "64",
                        "--max-seq-len", "256", "--bench", "--bench-pp", "48", "--max-tokens", "8", "--bench-reps", "2", "--bench-batch", "2"],
                       capture_output=True, text=True, timeout=600)
    assert b.returncode == 0, b.stderr[-2000:]
    assert "pp    96 tokens" in b.stderr and "tg    16 tokens" in b.stderr
