"""Nomanex on the host: config.json keys and refusals, the plan it becomes (sublayers side by side behind one norm, layers that
use another layer's weights as a run order), the tensors it expects and the caches its layers and its embedding ask for; and
the plain implementation's own mechanisms where a fault would be silent.  Needs no GPU."""
import copy
import json

import pytest
import torch

from imp_b200.cache.manager import CacheManager
from imp_b200.config.model_config import ConfigError, NomanexConfig
from imp_b200.config.registry import config_from_dict, known_architectures, load_config, plan_for
from imp_b200.parts.registry import mixer_cache_spec
from plain import nomanex_plain as N

CFG = {
    "architecture": "Nomanex", "vocab": 103, "width": 72, "norm": {"eps": 2e-5}, "residual_mult": 0.7,
    "embedding": {"bigram": {"buckets": 57, "mul_prev": 31, "mul_cur": 5}},
    "layers": [
        {"type": "gla", "mixer": {"heads": 3, "dim": 8, "vdim": 24, "tau": 9.0, "decay_rank": 6}, "mlp": {"kind": "dense", "ff": 100, "limit": 1.5}},
        {"type": "latent_attention",
         "mixer": {"heads": 5, "dim": 24, "rot_dim": 8, "vdim": 40, "kv_rank": 50, "scale": 0.2, "mask": {"size": 10}, "rot": {"base": 100.0, "dims": 8}},
         "mlp": {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 12, "top": 3, "groups": {"count": 4, "keep": 2}}}},
        {"type": "gla", "mixer": {"heads": 3, "dim": 8, "vdim": 24, "tau": 9.0}, "mlp": {"kind": "dense", "ff": 100, "limit": 1.5}, "weights_of": 0},
        {"type": "latent_attention", "mixer": {"heads": 2, "dim": 16, "rot_dim": 4, "vdim": 12, "kv_rank": 300, "rot": {"base": 7.0}}, "mlp": None},
        {"type": "latent_attention", "mixer": {"heads": 2, "dim": 16, "rot_dim": 4, "vdim": 12, "kv_rank": 300, "rot": {"base": 7.0}}, "mlp": None,
         "weights_of": 3},
    ],
}


def test_architecture_is_known_and_round_trips(tmp_path):
    assert "Nomanex" in known_architectures()
    c = config_from_dict(CFG)
    assert isinstance(c, NomanexConfig)
    assert (c.architecture, c.vocab_size, c.hidden_size, c.num_hidden_layers) == ("Nomanex", 103, 72, 5)
    assert [c.weights_layer(i) for i in range(5)] == [0, 1, 0, 3, 3] == [N.weights_layer(CFG, i) for i in range(5)]
    c.save(str(tmp_path))
    assert load_config(str(tmp_path)) == c
    saved = json.load(open(tmp_path / "config.json"))
    assert saved["layers"][3]["mlp"] is None and saved["layers"][2]["weights_of"] == 0


def test_plan_takes_every_size_and_constant_from_config():
    plan = plan_for(config_from_dict(CFG))
    assert [l.block for l in plan.layers] == ["parallel"] * 3 and plan.order == [0, 1, 0, 2, 2]
    l0, l1, l2 = plan.layers
    assert list(l0.parts) == ["norm", "mixer", "feed_forward"] and list(l2.parts) == ["norm", "mixer"]
    assert l0.block_params == {"residual_mult": 0.7, "has_ffn": True} and l2.block_params == {"residual_mult": 0.7, "has_ffn": False}
    g = l0.mixer
    assert g.kind == "gated_linear_attention"
    assert (g.params["num_heads"], g.params["key_dim"], g.params["value_dim"], g.params["tau"], g.params["decay_rank"], g.params["norm_eps"]) == (3, 8, 24, 9.0, 6, 2e-5)
    assert g.tensors["decay_down"] == "l0.mix.a1" and g.tensors["decay_bias"] == "l0.mix.a2.b"
    a = l1.mixer
    assert a.kind == "latent_attention"
    assert (a.params["num_heads"], a.params["head_dim"], a.params["rot_dim"], a.params["rot_dims"], a.params["value_dim"], a.params["kv_rank"],
            a.params["q_rank"], a.params["scale"], a.params["window"], a.params["rot_base"], a.params["rot_pairing"], a.params["out_gate"]) == \
        (5, 24, 8, 8, 40, 50, 0, 0.2, 10, 100.0, "neighbours", True)
    assert l2.mixer.params["window"] == 0 and l2.mixer.params["rot_dims"] == 4
    assert l2.mixer.params["scale"] == pytest.approx(20 ** -0.5)
    assert l2.mixer.tensors["q_proj"] == "l3.mix.q", "tensors are named by the layer's place in the configuration"
    d = l0.feed_forward
    assert d.kind == "gated_mlp" and (d.params["intermediate_size"], d.params["activation"], d.params["limit"]) == (100, "clipped", 1.5)
    f = l1.feed_forward
    assert f.kind == "routed_experts"
    assert (f.params["num_experts"], f.params["top_k"], f.params["expert_size"], f.params["expert"], f.params["scores"], f.params["num_groups"],
            f.params["keep_groups"], f.params["group_score"], f.params["router_bias"]) == (12, 3, 20, "relu2", "softmax_all", 4, 2, "max", False)
    for n in (l0.parts["norm"], plan.final_norm):
        assert n.kind == "dynamic_tanh" and n.params["size"] == 72
    assert plan.final_norm.tensors == {"weight": "final.norm", "bias": "final.norm.b", "alpha": "final.norm.alpha"}
    e = plan.embedding
    assert e.kind == "bigram_embedding" and (e.params["buckets"], e.params["mul_prev"], e.params["mul_cur"]) == (57, 31, 5)


def test_expected_tensors_are_the_checkpoint_names():
    exp = plan_for(config_from_dict(CFG)).expected_tensors()
    shapes = {k: tuple(v.shape) for k, v in exp.items()}
    assert shapes["embed"] == (103, 72) and shapes["bigram"] == (58, 72) and shapes["head"] == (103, 72)
    assert shapes["final.norm"] == (72,) and shapes["final.norm.alpha"] == () and shapes["l1.norm1.b"] == (72,)
    assert shapes["l0.mix.q"] == (24, 72) and shapes["l0.mix.v"] == (72, 72) and shapes["l0.mix.g"] == (72, 72) and shapes["l0.mix.norm"] == (24,)
    assert shapes["l0.mix.a1"] == (6, 72) and shapes["l0.mix.a2"] == (24, 6) and shapes["l0.mix.a2.b"] == (24,)
    assert shapes["l1.mix.q"] == (5 * 32, 72) and shapes["l1.mix.dkv"] == (58, 72) and shapes["l1.mix.dkv.norm"] == (50,)
    assert shapes["l1.mix.uk"] == (120, 50) and shapes["l1.mix.uv"] == (200, 50) and shapes["l1.mix.g"] == (200, 72) and shapes["l1.mix.o"] == (72, 200)
    assert shapes["l1.mlp.e11.up"] == (20, 72) and shapes["l1.mlp.e11.down"] == (72, 20) and shapes["l1.mlp.router"] == (12, 72)
    for absent in ("l2.mix.q", "l2.norm1", "l3.mlp.up", "l4.mix.q", "l0.norm2", "l1.mlp.e0.gate"):
        assert absent not in exp
    cfg = copy.deepcopy(CFG)
    del cfg["layers"][0]["mixer"]["decay_rank"]
    exp = plan_for(config_from_dict(cfg)).expected_tensors()
    assert tuple(exp["l0.mix.a1"].shape) == (-1, 72), "the checkpoint's tensor gives the inner size"


def test_options_that_config_leaves_out_do_not_exist():
    cfg = copy.deepcopy(CFG)
    del cfg["embedding"], cfg["residual_mult"], cfg["layers"][1]["mlp"]["router"]["groups"]
    cfg["layers"] = cfg["layers"][:2]
    plan = plan_for(config_from_dict(cfg))
    assert plan.order is None and plan.embedding.kind == "token_embedding" and "bigram" not in plan.expected_tensors()
    assert plan.layers[0].block_params["residual_mult"] == 1.0
    assert (plan.layers[1].feed_forward.params["num_groups"], plan.layers[1].feed_forward.params["keep_groups"]) == (0, 0)


def test_every_run_of_a_layer_owns_its_caches():
    plan = plan_for(config_from_dict(CFG))
    gla = mixer_cache_spec("gated_linear_attention", plan.layers[0].mixer.params)
    assert [t["name"] for t in gla["tensors"]] == ["S"] and gla["tensors"][0]["shape"][0] >= 3 * 8 * 24
    at = mixer_cache_spec("latent_attention", plan.layers[1].mixer.params)
    assert at == {"kind": "paged", "num_kv_heads": 1, "head_dim": 64, "window": 10, "keys_only": True}     # 50 + 8 entries in rows of 64
    wide = mixer_cache_spec("latent_attention", plan.layers[2].mixer.params)
    assert (wide["head_dim"], wide["window"]) == (304, 0)           # beyond what the padded rows are for
    last = {"kind": "state", "tensors": [{"name": "last_token", "shape": [1], "dtype": "int32"}]}
    mgr = CacheManager([gla, at, gla, wide, wide, last], page_size=4, num_pages=32, num_state_slots=2)
    info = mgr.info()
    assert [len(g["layers"]) for g in info["paged"]] == [1, 2] and [len(g["layers"]) for g in info["state"]] == [2, 1]
    for rid, n in ((1, 19), (2, 3)):
        mgr.add_request(rid)
        mgr.reserve(rid, n)
        mgr.commit(rid, n)
    mgr.check_invariants()
    mgr.release(1)
    mgr.release(2)
    assert mgr.free_pages() == 32


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][1].update(type="conv"), "unknown layer type 'conv'"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "unknown kind 'gated'"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0.0), "tau must be positive"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "dims 7 must be even"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5), "count must divide the experts"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=13), "top 13 exceeds the 12 experts"),
    (lambda c: c["layers"][2].update(weights_of=5), "weights_of 5"),
    (lambda c: c["layers"][2].update(weights_of=2), "weights_of 2"),
    (lambda c: c["layers"][2].update(weights_of=1), "is not that of the layer whose weights it uses"),
    (lambda c: c["layers"][0].update(weights_of=2), "circle"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_refusals_name_the_key(edit, text):
    cfg = copy.deepcopy(CFG)
    edit(cfg)
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    assert text in str(e.value)


# ------------------------------------------------------------------ the plain implementation's own mechanisms
def test_plain_bigram_rows():
    c = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert N.bigram_rows([4, 5, 5], c) == [10, (12 + 35) % 10, (15 + 35) % 10]


def test_plain_decay_is_a_root_of_the_sigmoid():
    z = torch.tensor([-3.0, 0.0, 4.0], dtype=torch.float64)
    assert torch.allclose(N.channel_decay(z, 16.0), torch.sigmoid(z) ** (1 / 16.0))


def test_plain_scan_decays_key_rows_before_the_token_joins():
    q = torch.tensor([[0.0, 0.0], [1.0, 1.0]], dtype=torch.float64)
    k = torch.tensor([[1.0, 2.0], [0.0, 10.0]], dtype=torch.float64)
    v = torch.tensor([[1.0], [1.0]], dtype=torch.float64)
    alpha = torch.tensor([[0.1, 0.1], [0.5, 0.25]], dtype=torch.float64)
    assert N.scan_channel_decay(q, k, v, alpha)[1].item() == pytest.approx(0.5 * 1 + 0.25 * 2 + 10)


def test_plain_window_sees_itself_and_size_minus_one_before():
    p = N.windowed_softmax(torch.zeros(12, 12, dtype=torch.float64), 5)
    for i in range(12):
        assert torch.nonzero(p[i] > 0)[:, 0].tolist() == list(range(max(0, i - 4), i + 1))
    assert torch.nonzero(N.windowed_softmax(torch.zeros(12, 12, dtype=torch.float64), 0)[11] > 0).numel() == 12


def test_plain_route_keeps_groups_by_their_largest_score():
    W = {"f.router": torch.eye(8, dtype=torch.float64)}
    c = {"router": {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 1}}}
    h = torch.tensor([[3.0, -5.0, 0.0, 0.0, 2.0, 2.5, 0.0, 0.0]], dtype=torch.float64)   # group 0: the largest score; group 2: the largest pair
    idx, w, s = N.route(h, W, "f.", c)
    assert idx[0].tolist() == [0, 1]
    assert torch.allclose(w[0], torch.softmax(h[0], dim=0)[:2]) and float(w.sum()) < 1
    c["router"]["groups"] = None
    assert sorted(N.route(h, W, "f.", c)[0][0].tolist()) == [0, 5]


def test_plain_clipped_gate():
    g = torch.tensor([5.0, -9.0, 1.0], dtype=torch.float64)
    u = torch.tensor([4.0, -4.0, 0.5], dtype=torch.float64)
    want = [2 * torch.sigmoid(torch.tensor(3.404)).item() * 3, -9 * torch.sigmoid(torch.tensor(-9 * 1.702)).item() * -1, torch.sigmoid(torch.tensor(1.702)).item() * 1.5]
    assert N.clipped_gate(g, u, 2.0).tolist() == pytest.approx(want, rel=1e-5)
