"""Ribovik on the host: config.json keys and refusals, the plan it becomes (a norm behind each sublayer, the head on the
embedding's table), the tensors it expects and the caches its layers ask for; and the plain implementation's own mechanisms
where a fault would be silent.  Needs no GPU."""
import copy
import json
import math

import pytest
import torch

from imp_b200.cache.manager import CacheManager
from imp_b200.config.model_config import ConfigError, RibovikConfig
from imp_b200.config.registry import config_from_dict, known_architectures, load_config, plan_for
from imp_b200.parts.registry import mixer_cache_spec
from plain import ribovik_plain as R

SCALING = {"factor": 4.0, "original": 40, "fast": 3.0, "slow": 0.5}
CFG = {
    "architecture": "Ribovik", "vocab": 103, "width": 72, "norm": {"eps": 2e-5},
    "layers": [
        {"type": "attention", "mixer": {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.3, "mask": {"size": 10},
                                        "rot": {"base": 100.0, "dims": 8, "scaling": SCALING}},
         "mlp": {"kind": "dense", "ff": 100}},
        {"type": "attention", "mixer": {"heads": 3, "kv_heads": 3, "dim": 16, "vdim": 16, "scale": 0.5, "mask": {"size": 33},
                                        "rot": {"base": 7.0, "dims": 16}},
         "mlp": {"kind": "moe", "expert": {"ff": 20, "limit": 1.5}, "router": {"experts": 12, "identity": 3, "top": 5},
                 "shared": {"ff": 28, "limit": 0.5}}},
        {"type": "attention", "mixer": {"heads": 4, "dim": 20}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 1, "dim": 16, "vdim": 8, "scale": 0.25},
         "mlp": {"kind": "moe", "expert": {"ff": 9, "limit": 7.0}, "router": {"experts": 4, "top": 1}, "shared": None}},
    ],
}


def test_architecture_is_known_and_round_trips(tmp_path):
    assert "Ribovik" in known_architectures()
    c = config_from_dict(CFG)
    assert isinstance(c, RibovikConfig)
    assert (c.architecture, c.vocab_size, c.hidden_size, c.num_hidden_layers) == ("Ribovik", 103, 72, 4)
    c.save(str(tmp_path))
    assert load_config(str(tmp_path)) == c
    saved = json.load(open(tmp_path / "config.json"))
    assert saved["layers"][2]["mlp"] is None and saved["layers"][0]["mixer"]["rot"]["scaling"] == SCALING


def test_plan_takes_every_size_and_constant_from_config():
    plan = plan_for(config_from_dict(CFG))
    assert [l.block for l in plan.layers] == ["output_norm"] * 4 and plan.order is None
    l0, l1, l2, l3 = plan.layers
    assert list(l0.parts) == ["mixer", "mixer_post_norm", "feed_forward", "ffn_post_norm"] and list(l2.parts) == ["mixer", "mixer_post_norm"]
    assert l0.block_params == {"has_ffn": True} and l2.block_params == {"has_ffn": False}
    a = l0.mixer
    assert a.kind == "gated_head_attention"
    p = a.params
    assert (p["num_heads"], p["num_kv_heads"], p["head_dim"], p["value_dim"], p["scale"], p["chunk"], p["rot_dims"], p["rot_base"], p["norm_eps"]) == \
        (6, 2, 24, 40, 0.3, 10, 8, 100.0, 2e-5)
    assert (p["qkv_bias"], p["qk_norm"], p["qk_norm_weight"], p["qk_norm_position"], p["rot_pairing"], p["sink"]) == \
        (True, True, False, "after_rotation", "neighbours", True)
    assert p["rot_scaling"] == dict(SCALING, kind="yarn")
    assert a.tensors == {"q_proj": "l0.mix.q", "q_bias": "l0.mix.q.b", "k_proj": "l0.mix.k", "k_bias": "l0.mix.k.b", "v_proj": "l0.mix.v",
                         "v_bias": "l0.mix.v.b", "o_proj": "l0.mix.o"}
    assert "rot_scaling" not in l1.mixer.params and l1.mixer.params["chunk"] == 33
    f = l0.feed_forward
    assert f.kind == "gated_mlp" and (f.params["intermediate_size"], f.params["activation"], f.params["bias"]) == (100, "silu", True)
    e = l1.feed_forward
    assert e.kind == "routed_experts"
    q = e.params
    assert (q["num_experts"], q["num_identity"], q["top_k"], q["expert_size"], q["shared_size"], q["expert"], q["expert_limit"], q["shared_limit"]) == \
        (12, 3, 5, 20, 28, "clipped", 1.5, 0.5)
    assert (q["scores"], q["choice_bias"], q["renormalise"], q["router_bias"], q["shared_gate"]) == ("softmax_all", True, True, False, False)
    for n, name in ((l1.parts["mixer_post_norm"], "l1.norm1"), (l1.parts["ffn_post_norm"], "l1.norm2"), (plan.final_norm, "final.norm")):
        assert n.kind == "rmsnorm" and n.params == {"size": 72, "eps": 2e-5} and n.tensors == {"weight": name}
    assert plan.embedding.kind == "token_embedding" and plan.embedding.params["norm"] is True and plan.embedding.params["norm_eps"] == 2e-5
    assert plan.embedding.tensors == {"weight": "embed", "norm": "embed.norm"} and plan.head.tensors == {"weight": "embed"}


def test_expected_tensors_are_the_checkpoint_names():
    exp = plan_for(config_from_dict(CFG)).expected_tensors()
    shapes = {k: tuple(v.shape) for k, v in exp.items()}
    assert shapes["embed"] == (103, 72) and shapes["embed.norm"] == (72,) and shapes["final.norm"] == (72,) and "head" not in shapes
    assert shapes["l0.mix.q"] == (144, 72) and shapes["l0.mix.q.b"] == (144,) and shapes["l0.mix.k"] == (48, 72) and shapes["l0.mix.v"] == (80, 72)
    assert shapes["l0.mix.v.b"] == (80,) and shapes["l0.mix.o"] == (72, 240) and "l0.mix.o.b" not in shapes
    assert shapes["l0.mlp.gate"] == (100, 72) and shapes["l0.mlp.gate.b"] == (100,) and shapes["l0.mlp.down.b"] == (72,)
    assert shapes["l1.mlp.router"] == (15, 72) and shapes["l1.mlp.correction"] == (15,)
    assert shapes["l1.mlp.e11.gate"] == (20, 72) and shapes["l1.mlp.e11.down"] == (72, 20) and "l1.mlp.e12.gate" not in shapes
    assert shapes["l1.mlp.shared.up"] == (28, 72) and "l1.mlp.shared.up.b" not in shapes and "l1.mlp.e0.gate.b" not in shapes
    for absent in ("l2.norm2", "l2.mlp.gate", "l3.mlp.shared.gate"):
        assert absent not in shapes
    assert shapes["l3.mlp.router"] == (4, 72)


def test_options_that_config_leaves_out_do_not_exist():
    l2 = plan_for(config_from_dict(CFG)).layers[2]
    p = l2.mixer.params
    assert (p["chunk"], p["rot_dims"], p["num_kv_heads"], p["value_dim"]) == (0, 0, 4, 20) and p["scale"] == pytest.approx(20 ** -0.5)
    l3 = plan_for(config_from_dict(CFG)).layers[3]
    assert l3.feed_forward.params["num_identity"] == 0 and "shared_size" not in l3.feed_forward.params


def test_layers_group_by_their_cache_and_chunks_are_given_back():
    plan = plan_for(config_from_dict(CFG))
    specs = [mixer_cache_spec("gated_head_attention", l.mixer.params) for l in plan.layers]
    assert [(s["num_kv_heads"], s["head_dim"], s["window"]) for s in specs] == [(2, 48, -10), (3, 16, -33), (4, 32, 0), (1, 16, 0)]
    mgr = CacheManager(specs, page_size=4, num_pages=16, num_state_slots=2)
    assert len(mgr.info()["paged"]) == 4
    for rid, n in ((1, 41), (2, 3)):
        mgr.add_request(rid)
        mgr.reserve(rid, n)
        mgr.commit(rid, n)
    mgr.check_invariants()
    assert [sum(p >= 0 for p in mgr.block_table(g, 1)) for g in range(4)] == [1, 3, 11, 11]     # 40.., 33.., everything
    mgr.release(1)
    mgr.release(2)
    assert mgr.free_pages() == 16


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][1].update(type="conv"), "unknown layer type 'conv'"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "unknown kind 'gated'"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "6 heads are not a multiple of 4 kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0.0), "scale must be positive"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "'size' must be positive"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims 7 must be even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "dims 26 must be even and at most dim 24"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "must be positive"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(limit=-1.0), "limit must be positive"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=16), "top 16 exceeds the 15 router outputs"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "identity must not be negative"),
    (lambda c: c["layers"][2].pop("mixer"), "mixer"),
    (lambda c: c.update(layers=[]), "non-empty list"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_refusals_name_the_key(edit, text):
    cfg = copy.deepcopy(CFG)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert text in str(e.value)


# ------------------------------------------------------------------ the plain implementation's own mechanisms
def test_plain_yarn_keeps_fast_pairs_and_slows_slow_ones():
    f, stretch = R.yarn_frequencies(100.0, 16, {"factor": 8.0, "original": 100, "fast": 4.0, "slow": 1.0})
    plain = [100.0 ** (-2.0 * i / 16) for i in range(8)]
    turns = [100 * v / (2 * math.pi) for v in plain]                      # a pair's turns over the original length
    lo = math.floor(16 * math.log(100 / (2 * math.pi * 4.0)) / (2 * math.log(100.0)))
    hi = math.ceil(16 * math.log(100 / (2 * math.pi)) / (2 * math.log(100.0)))
    assert (lo, hi) == (2, 5) and turns[2] > 4.0 > turns[3] and turns[4] > 1.0 > turns[5]
    assert f[:3].tolist() == pytest.approx(plain[:3]) and f[5:].tolist() == pytest.approx([v / 8 for v in plain[5:]])
    assert f[3].item() == pytest.approx(plain[3] * (2 / 3) + plain[3] / 8 / 3)
    assert stretch == pytest.approx(0.1 * math.log(8.0) + 1)
    same, one = R.yarn_frequencies(100.0, 16, None)
    assert same.tolist() == pytest.approx(plain) and one == 1.0
    step, _ = R.yarn_frequencies(100.0, 16, {"factor": 2.0, "original": 100, "fast": 1e9, "slow": 5e8})     # both ends before the first pair
    assert step.tolist() == pytest.approx([plain[0]] + [v / 2 for v in plain[1:]])


def test_plain_chunks_are_counted_from_the_sequence_start():
    seen = R.chunk_visible(12, 5)
    for i in range(12):
        assert torch.nonzero(seen[i])[:, 0].tolist() == list(range(i // 5 * 5, i + 1))
    assert int(R.chunk_visible(12, 0)[11].sum()) == 12


def test_plain_sink_takes_its_share():
    s = torch.tensor([[0.0, 0.0, 0.0], [-50.0, 3.0, 1.0], [80.0, 90.0, 0.0]], dtype=torch.float64)
    seen = torch.tensor([[True, True, False], [True, True, True], [True, True, True]])
    p = R.sink_softmax(s, seen)
    assert p[0].tolist() == pytest.approx([1 / 3, 1 / 3, 0.0])
    e = [math.exp(v) for v in (-50.0, 3.0, 1.0)]
    assert p[1].tolist() == pytest.approx([v / (1 + sum(e)) for v in e])
    assert float(p[2].sum()) == pytest.approx(1.0)


def test_plain_route_chooses_with_the_correction_and_weighs_without_it():
    W = {"f.router": torch.eye(6, dtype=torch.float64), "f.correction": torch.tensor([0.0, 0.0, 0.9, 0.0, 0.0, 0.0], dtype=torch.float64)}
    c = {"router": {"experts": 4, "identity": 2, "top": 2}, "expert": {"ff": 1, "limit": 1.0}}
    h = torch.tensor([[1.0, 0.0, -1.0, 0.0, 2.0, 0.0]], dtype=torch.float64)
    idx, w, s = R.route(h, W, "f.", c)
    assert idx[0].tolist() == [2, 4]                                       # the corrected one first, then an identity
    sm = torch.softmax(h[0], dim=0)
    assert torch.allclose(s[0], sm) and w[0].tolist() == pytest.approx([float(sm[2] / (sm[2] + sm[4])), float(sm[4] / (sm[2] + sm[4]))])


def test_plain_identity_expert_gives_the_input():
    d = 6
    W = {"f.router": torch.zeros(3, d, dtype=torch.float64), "f.correction": torch.tensor([0.0, 1.0, 0.0], dtype=torch.float64)}
    for n, shape in (("gate", (2, d)), ("up", (2, d)), ("down", (d, 2))):
        W["f.e0." + n] = torch.randn(*shape, dtype=torch.float64)
    h = torch.randn(4, d, dtype=torch.float64)
    out = R.moe(h, W, "f.", {"router": {"experts": 1, "identity": 2, "top": 1}, "expert": {"ff": 2, "limit": 1.0}})
    assert torch.allclose(out, h)
