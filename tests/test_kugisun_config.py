"""Kugisun on the CPU: its typed configuration, the parts the registry makes of it, the tensors it declares, and the plain
implementation's own consistency (the delta rule against a closed form, the router by hand)."""
import copy
import math

import pytest
import torch

from llmgen_b200.config.base import ConfigError
from llmgen_b200.parts.registry import model_weight_decls
from llmgen_b200.registry import config_from_dict
from tests import kugisun_util as ku
from tests.plain import kugisun_plain as plain


def spec_of(cfg):
    arch, typed = config_from_dict(cfg)
    return arch.build_spec(typed)


def test_the_registry_finds_the_architecture_and_the_parts_it_is_made_of():
    spec = spec_of(ku.MIXED)
    assert spec.architecture == "Kugisun" and spec.lm_head == spec.embedding == "embed" and spec.position_table == "pos"
    assert spec.residual_streams == 3 and spec.max_positions == 512
    assert [l.kind for l in spec.layers] == ["multi_stream"] * 3
    # five layers of three sets of weights, each with a cache and state number of its own
    assert [item.layer for item in spec.run_order] == [0, 1, 1, 2, 0] and [item.cache for item in spec.run_order] == [0, 1, 2, 3, 4]
    assert all(item.writes_cache for item in spec.run_order)
    assert [l.ffn.kind if l.ffn is not None else None for l in spec.layers] == ["gated_mlp", "routed_mlp", None]
    assert all(l.mixer_norm.weight_offset == 1.0 for l in spec.layers) and spec.final_norm.weight_offset == 1.0
    assert spec.layers[1].mixer_streams.mix == "l1.hc1.mix" and spec.layers[1].ffn_streams.read == "l1.hc2.in" and spec.layers[2].ffn_streams is None
    assert spec.layers[2].mixer_streams.write == "l3.hc1.out"           # the third set of weights belongs to layer 3
    par = spec.layers[0].mixer
    assert par.scales == (0.7, 1.2) and [b.kind for b in par.branches] == ["attention", "head_decay_delta"]
    att, rule = par.branches
    assert (att.num_heads, att.num_kv_heads, att.head_dim, att.v_head_dim, att.scale, att.window) == (4, 2, 16, 24, 0.3, None)
    assert att.q_bias == "l0.mix.left.q.b" and att.v_bias == "l0.mix.left.v.b" and att.o_bias is None and not att.sink and att.q_norm.dim == 16
    assert att.position.rotary_dim == 8 and att.position.pairing == "interleaved" and att.position.theta == 300.0
    assert (rule.num_heads, rule.num_kv_heads, rule.key_dim, rule.value_dim, rule.conv.taps, rule.unit_eps) == (4, 2, 8, 16, 3, 1e-6)
    assert rule.conv.channels == 2 * 2 * 8 + 4 * 16 and rule.out_norm.weight_offset == 0.0
    ffn = spec.layers[1].ffn
    assert (ffn.top_k, len(ffn.experts), ffn.identity_outputs, ffn.groups, ffn.keep_groups, ffn.weight_scale) == (3, 6, 2, 4, 2, 1.7)
    assert ffn.scoring == "softmax" and not ffn.renormalize and not ffn.weight_on_input and ffn.choice_bias == "l1.mlp.correction"
    assert ffn.shared.intermediate_size == 40 and ffn.shared_gate == "l1.mlp.shared.sg"
    odd = spec_of(ku.ODD)
    assert odd.layers[0].mixer.branches[0].position is None and odd.layers[0].ffn.shared is None and odd.layers[0].ffn.shared_gate is None
    assert odd.layers[0].ffn.groups == 1 and odd.layers[0].ffn.identity_outputs == 0 and odd.residual_streams == 1 and odd.layers[0].mixer_streams is not None
    assert [item.layer for item in odd.run_order] == [0, 1, 1, 1]
    bare = spec_of(ku.PLAIN)
    assert bare.layers[0].mixer_streams is None and bare.layers[0].streams == 1 and bare.residual_streams == 1


def test_declared_tensors_have_the_design_s_names_and_shapes():
    shapes = {d.name: tuple(d.shape) for d in model_weight_decls(spec_of(ku.MIXED))}
    assert shapes["embed"] == (97, 48) and shapes["pos"] == (512, 48) and shapes["final.norm"] == (48,) and "head" not in shapes
    assert shapes["l0.hc1.in"] == (3,) and shapes["l0.hc2.out"] == (3,) and shapes["l0.hc1.mix"] == (3, 3)
    assert shapes["l0.mix.left.q"] == (64, 48) and shapes["l0.mix.left.k"] == (32, 48) and shapes["l0.mix.left.v"] == (48, 48)
    assert shapes["l0.mix.left.q.b"] == (64,) and shapes["l0.mix.left.v.b"] == (48,) and shapes["l0.mix.left.k.norm"] == (16,)
    assert shapes["l0.mix.left.o"] == (48, 96) and "l0.mix.left.o.b" not in shapes
    assert shapes["l0.mix.right.q"] == (16, 48) and shapes["l0.mix.right.v"] == (64, 48) and shapes["l0.mix.right.g"] == (64, 48)
    assert shapes["l0.mix.right.b"] == (4, 48) and shapes["l0.mix.right.a"] == (4, 48) and shapes["l0.mix.right.dt_bias"] == (4,)
    assert shapes["l0.mix.right.A_log"] == (4,) and shapes["l0.mix.right.norm"] == (16,) and shapes["l0.mix.right.k.conv"] == (16, 3)
    assert shapes["l0.mix.right.o"] == (48, 64) and shapes["l0.mlp.gate"] == (40, 48) and shapes["l0.mlp.down"] == (48, 40)
    assert shapes["l1.mlp.router"] == (8, 48) and shapes["l1.mlp.correction"] == (8,) and shapes["l1.mlp.e5.down"] == (48, 24) and "l1.mlp.e6.up" not in shapes
    assert shapes["l1.mlp.shared.gate"] == (40, 48) and shapes["l1.mlp.shared.sg"] == (1, 48)
    assert not any(n.startswith(("l2.", "l4.")) for n in shapes)          # layers that use another's weights have none
    assert "l3.norm2" not in shapes and "l3.hc2.in" not in shapes and shapes["l3.hc1.mix"] == (3, 3)
    assert not any(".hc" in d.name for d in model_weight_decls(spec_of(ku.PLAIN)))


def test_the_positions_come_from_the_folder_s_table_when_the_file_does_not_name_them():
    from llmgen_b200.config.kugisun import KugisunConfig
    cfg = copy.deepcopy(ku.MIXED)
    del cfg["max_positions"]
    assert KugisunConfig.fill_from_tensor_shapes(cfg, {"pos": (77, 48)})["max_positions"] == 77 and "max_positions" not in cfg
    assert KugisunConfig.fill_from_tensor_shapes(ku.MIXED, {"pos": (77, 48)})["max_positions"] == 512
    with pytest.raises(ConfigError, match="max_positions"):
        config_from_dict(cfg)


def test_every_problem_of_a_configuration_is_listed_at_once():
    cfg = copy.deepcopy(ku.MIXED)
    cfg["layers"][0]["mixer"]["left"]["kv_heads"] = 3
    cfg["layers"][0]["mixer"]["left"]["rot"]["dims"] = 7
    cfg["layers"][1]["mlp"]["router"]["groups"]["count"] = 3
    cfg["layers"][1]["mlp"]["router"]["top"] = 9
    cfg["layers"][3]["mixer"]["right"]["conv"] = 9
    cfg["layers"][3]["mixer"]["right"].pop("vdim")
    cfg["streams"] = 20
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    text = str(e.value)
    for piece in ("kv_heads", "rot.dims", "3 equal groups", "top 9", "vdim", "streams"):
        assert piece in text, piece
    for change in ({"weights_of": 7}, {"weights_of": 2}, {"mlp": None}):          # nowhere; a circle; an entry that differs
        bad = copy.deepcopy(ku.MIXED)
        bad["layers"][2].update(change)
        with pytest.raises(ConfigError, match="layers\\[2\\]"):
            config_from_dict(bad)


def test_the_plain_delta_rule_agrees_with_a_product_of_matrices():
    """S_t = (I - beta k k^T) g S + beta k v^T, written out from the definition; with beta = 0 nothing is written."""
    torch.manual_seed(0)
    T, H, G, D, E = 7, 4, 2, 5, 3
    q, k = plain.unit(torch.randn(T, G, D, dtype=torch.float64)), plain.unit(torch.randn(T, G, D, dtype=torch.float64))
    v, beta, g = torch.randn(T, H, E, dtype=torch.float64), torch.rand(T, H, dtype=torch.float64), torch.rand(T, H, dtype=torch.float64)
    o, last = plain.delta_memory(q, k, v, beta, g)
    for h in range(H):
        S = torch.zeros(D, E, dtype=torch.float64)
        for t in range(T):
            kk = k[t, h // 2]
            S = (torch.eye(D, dtype=torch.float64) - beta[t, h] * torch.outer(kk, kk)) @ (g[t, h] * S) + beta[t, h] * torch.outer(kk, v[t, h])
            assert float((o[t, h] - q[t, h // 2] @ S).abs().max()) < 1e-12
        assert float((last[h] - S).abs().max()) < 1e-12
    again = plain.delta_memory(q[3:], k[3:], v[3:], beta[3:], g[3:], plain.delta_memory(q[:3], k[:3], v[:3], beta[:3], g[:3])[1])
    assert float((again[0] - o[3:]).abs().max()) < 1e-12
    assert float(plain.delta_memory(q, k, v, 0 * beta, g)[0].abs().max()) == 0.0


def test_the_plain_router_by_hand():
    """Six outputs in three groups: the correction chooses groups and outputs, the scores without it weigh; masked outputs
    are out of the choice even where every correction is far below zero."""
    z = torch.log(torch.tensor([0.30, 0.05, 0.20, 0.15, 0.10, 0.20], dtype=torch.float64))
    r = {"groups": {"count": 3, "keep": 1}, "top": 2, "scale": 2.0}
    best, w = plain.choose(z, torch.zeros(6), r)
    assert best == [0, 1] and abs(w[0] - 0.6) < 1e-12 and abs(w[1] - 0.1) < 1e-12           # the group of 0.30, not the two largest
    best, w = plain.choose(z, torch.tensor([-5.0, -5.0, -5.0, -5.0, -4.0, -5.0]), r)
    assert best == [4, 5] and abs(w[0] - 0.2) < 1e-12 and abs(w[1] - 0.4) < 1e-12
    best, _ = plain.choose(z, torch.zeros(6), {"groups": {"count": 3, "keep": 2}, "top": 3})
    assert sorted(best) == [0, 2, 3]
    best, w = plain.choose(z, torch.zeros(6), {"top": 2})
    assert best[0] == 0 and abs(w[0] - 0.3) < 1e-12 and math.isclose(w[1], 0.2)


def test_the_plain_rotation_turns_neighbours_and_leaves_the_rest():
    x = torch.tensor([1.0, 0.0, 0.0, 2.0, 5.0], dtype=torch.float64)
    y = plain.turn_neighbours(x, 3, {"base": 16.0, "dims": 4})
    a, b = 3.0, 3.0 * 16.0 ** -0.5
    want = [math.cos(a), math.sin(a), -2.0 * math.sin(b), 2.0 * math.cos(b), 5.0]
    assert float((y - torch.tensor(want, dtype=torch.float64)).abs().max()) < 1e-12


def test_profiler_costs_count_the_design_s_products():
    from llmgen_b200.engine.profiler import ModelCost
    cost = ModelCost.from_spec(spec_of(ku.MIXED))
    assert cost.complete and cost.state_bytes > 0 and len(cost.attention) == 5
