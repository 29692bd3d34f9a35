"""Zuvasun on the CPU: its typed configuration, the parts the registry makes of it, the tensors it declares, what layers that
share a cache ask of it, and the plain implementation's own consistency."""
import copy
import math

import pytest
import torch

from llmgen_b200.cache.manager import FULL, WINDOW
from llmgen_b200.config.base import ConfigError
from llmgen_b200.parts.base import KVRequest
from llmgen_b200.parts.registry import model_weight_decls
from llmgen_b200.registry import config_from_dict
from tests import zuvasun_util as zu
from tests.plain import zuvasun_plain as plain


def spec_of(cfg):
    arch, typed = config_from_dict(cfg)
    return arch.build_spec(typed)


def test_the_registry_finds_the_architecture_and_the_parts_it_is_made_of():
    spec = spec_of(zu.MIXED)
    assert spec.architecture == "Zuvasun" and spec.embedding == "embed" and spec.lm_head == "head" and not spec.tied
    assert [layer.kind for layer in spec.layers] == ["parallel_block"] * 4
    assert [layer.mixer.kind for layer in spec.layers] == ["latent_attention", "attention", "latent_attention", "attention"]
    assert [layer.ffn.kind if layer.ffn is not None else None for layer in spec.layers] == ["routed_mlp", "routed_mlp", None, "routed_mlp"]
    assert [(i.layer, i.cache, i.writes_cache) for i in spec.run_order] == [(0, 0, True), (1, 1, True), (2, 0, False), (3, 3, True)]
    assert spec.layers[0].mixer_gain == "l0.ls1" and spec.layers[0].ffn_gain == "l0.ls2" and spec.layers[2].ffn_gain is None
    lat = spec.layers[0].mixer
    assert (lat.num_heads, lat.nope_dim, lat.rope_dim, lat.value_dim, lat.kv_rank, lat.q_rank, lat.window) == (3, 16, 8, 24, 32, 0, 24)
    assert lat.q_proj == "l0.mix.q" and lat.dq_proj is None and lat.kv_norm.dim == 32 and lat.scale == 0.3
    assert lat.position.pairing == "interleaved" and lat.position.yarn == (4.0, 64.0, 8.0, 1.0) and lat.position.scaling is None
    reader = spec.layers[2].mixer
    assert reader.dkv_proj is None and reader.kv_norm is None and reader.window == 41 and reader.value_dim == 10
    att = spec.layers[1].mixer
    assert att.values_from_keys and att.row_norms and att.position is None and att.query_temperature == (0.25, 10.0)
    assert att.q_norm.dim == 64 and att.k_norm.dim == 32 and att.q_bias == "l1.mix.q.b" and att.v_bias is None
    assert spec.layers[3].mixer.query_temperature is None
    ffn = spec.layers[1].ffn
    assert ffn.top_k == 3 and len(ffn.experts) == 5 and ffn.scoring == "softmax" and ffn.renormalize and not ffn.weight_on_input
    assert ffn.choice_bias == "l1.mlp.correction" and ffn.weight_scale == 0.8 and ffn.experts[0].activation == "relu2" and ffn.shared is None
    assert spec_of(zu.ODD).layers[1].mixer.window is None


def test_declared_tensors_have_the_design_s_names_and_shapes():
    shapes = {d.name: tuple(d.shape) for d in model_weight_decls(spec_of(zu.MIXED))}
    assert shapes["embed"] == (97, 48) and shapes["head"] == (97, 48) and shapes["final.norm"] == (48,)
    assert shapes["l0.norm1"] == (48,) and shapes["l0.ls1"] == (48,) and shapes["l0.ls2"] == (48,) and "l0.norm2" not in shapes
    assert shapes["l0.mix.q"] == (72, 48) and shapes["l0.mix.dkv"] == (40, 48) and shapes["l0.mix.dkv.norm"] == (32,)
    assert shapes["l0.mix.uk"] == (48, 32) and shapes["l0.mix.uv"] == (72, 32) and shapes["l0.mix.o"] == (48, 72)
    assert shapes["l1.mix.q"] == (64, 48) and shapes["l1.mix.k"] == (32, 48) and shapes["l1.mix.q.b"] == (64,) and shapes["l1.mix.k.b"] == (32,)
    assert shapes["l1.mix.q.norm"] == (64,) and shapes["l1.mix.k.norm"] == (32,) and "l1.mix.v" not in shapes and shapes["l1.mix.o"] == (48, 64)
    assert shapes["l2.mix.q"] == (40, 48) and shapes["l2.mix.uk"] == (24, 32) and "l2.mix.dkv" not in shapes and "l2.mix.dkv.norm" not in shapes
    assert "l2.ls2" not in shapes and "l2.mlp.router" not in shapes
    assert shapes["l3.mlp.router"] == (3, 48) and shapes["l3.mlp.correction"] == (3,) and shapes["l3.mlp.e2.up"] == (20, 48)
    assert shapes["l3.mlp.e2.down"] == (48, 20) and "l3.mlp.e0.gate" not in shapes
    assert spec_of(zu.MIXED).ignorable_tensors == ("l2.ls2",)


def test_every_problem_of_a_configuration_is_listed_at_once():
    cfg = copy.deepcopy(zu.MIXED)
    cfg["layers"][1]["mixer"]["kv_heads"] = 3
    cfg["layers"][1]["mixer"]["vdim"] = 20
    cfg["layers"][0]["mixer"]["rot"]["dims"] = 6
    cfg["layers"][0]["mixer"]["rot"]["scaling"].pop("fast")
    cfg["layers"][3]["mlp"]["router"]["top"] = 9
    cfg["norm"] = {}
    with pytest.raises(ConfigError) as e:
        config_from_dict(cfg)
    text = str(e.value)
    for piece in ("kv_heads", "vdim 20", "fast", "top 9", "eps"):
        assert piece in text, piece


@pytest.mark.parametrize("change", [{"kv_from": 2}, {"kv_from": 3}, {"kv_from": 1}, {"kv_rank": 16}, {"rot": {"base": 99.0, "dims": 8}}])
def test_a_reader_of_entries_names_an_earlier_layer_that_has_them_in_its_form(change):
    cfg = copy.deepcopy(zu.MIXED)
    cfg["layers"][2]["mixer"].update(change)
    with pytest.raises(ConfigError, match="kv_from"):
        config_from_dict(cfg)


def test_a_reader_of_a_reader_is_refused():
    cfg = copy.deepcopy(zu.MIXED)
    cfg["layers"][3] = copy.deepcopy(cfg["layers"][2])
    cfg["layers"][3]["mixer"]["kv_from"] = 2
    with pytest.raises(ConfigError, match="no latent entries of its own"):
        config_from_dict(cfg)


def test_a_shared_cache_serves_the_widest_view():
    near, wide, full = KVRequest(WINDOW, 24, 1, 40, values=False), KVRequest(WINDOW, 41, 1, 40, values=False), KVRequest(FULL, 0, 1, 40, values=False)
    assert near.shared_with(wide) == wide and wide.shared_with(near) == wide and near.shared_with(near) == near
    assert near.shared_with(full) == full and full.shared_with(near) == full
    assert near.shared_with(KVRequest(WINDOW, 24, 1, 48, values=False)) is None and near.shared_with(KVRequest(WINDOW, 24, 1, 40)) is None


def test_storage_keeps_one_array_and_one_number_per_token_where_keys_are_values():
    from llmgen_b200.cache.storage import CacheStorage, bytes_per_page
    req = KVRequest(FULL, 0, 2, 16, values=False, token_scales=True)
    st = CacheStorage({1: req}, {}, {1: 0}, [5], 8, 2, torch.bfloat16, "cpu")
    cache = st.layer_cache(1, True)
    assert tuple(cache.k.shape) == (5, 2, 8, 16) and cache.v is None
    assert tuple(cache.k_scale.shape) == (5, 8) and cache.k_scale.dtype == torch.float32
    assert bytes_per_page({1: req}, {1: 0}, 0, 8, torch.bfloat16) == 2 * 8 * 16 * 2 + 8 * 4
    assert st.bytes_held() == 5 * (2 * 8 * 16 * 2 + 8 * 4)


@pytest.mark.parametrize("dims,base,yarn", [(8, 100.0, (4.0, 64, 8.0, 1.0)), (48, 1000.0, (2.5, 300, 20.0, 2.0)), (16, 500.0, (1.0, 128, 32.0, 1.0)),
                                            (2, 10.0, (8.0, 32, 4.0, 1.0)), (32, 10000.0, (40.0, 4096, 32.0, 1.0)), (6, 77.0, None)])
def test_rotary_tables_are_the_plain_model_s_angles(dims, base, yarn):
    from llmgen_b200.parts.rope import Rope
    from llmgen_b200.parts.spec import RopeSpec
    cos, sin = Rope(RopeSpec(dims, base, 50, pairing="interleaved", yarn=yarn), None, torch.float32, "cpu").tables()
    rot = {"base": base, "dims": dims}
    if yarn is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    speeds, factor = plain.turning_speeds(rot)
    if yarn is not None and yarn[0] != 1.0 and dims > 2:
        plain_speeds, _ = plain.turning_speeds({"base": base, "dims": dims})
        assert factor > 1.0 and speeds != plain_speeds
    for p in (0, 1, 17, 49):
        for i, f in enumerate(speeds):
            assert abs(float(cos[p, i]) - factor * math.cos(p * f)) < 1e-6 and abs(float(sin[p, i]) - factor * math.sin(p * f)) < 1e-6


def test_some_pairs_keep_their_frequency_some_are_divided_and_some_lie_between():
    speeds, factor = plain.turning_speeds({"base": 1000.0, "dims": 48, "scaling": {"factor": 2.5, "original": 300, "fast": 20.0, "slow": 2.0}})
    base = [1000.0 ** (-2.0 * i / 48) for i in range(24)]
    ratio = [b / s for b, s in zip(base, speeds)]
    assert abs(ratio[0] - 1.0) < 1e-12 and abs(ratio[-1] - 2.5) < 1e-12 and any(1.01 < r < 2.49 for r in ratio)
    assert abs(factor - (1 + 0.1 * math.log(2.5))) < 1e-12


def test_the_plain_model_s_choice_weights_and_temperature_by_hand():
    z = torch.tensor([1.0, 0.0, 2.0, -1.0], dtype=torch.float64)
    s = torch.softmax(z, dim=0)
    best, w = plain.choose(z, torch.zeros(4, dtype=torch.float64), 2, 3.0)
    assert best == [2, 0] and abs(sum(w) - 3.0) < 1e-12 and abs(w[0] - 3.0 * float(s[2] / (s[2] + s[0]))) < 1e-12
    best, w = plain.choose(z, torch.tensor([0.0, 0.0, 0.0, 5.0], dtype=torch.float64), 2, 1.0)        # the correction chooses, the score weighs
    assert best == [3, 2] and abs(w[0] - float(s[3] / (s[3] + s[2]))) < 1e-12
    m = {"q_temp": {"coef": 0.5, "every": 4}}
    assert plain.query_temperature(m, 2) == 1.0 and abs(plain.query_temperature(m, 3) - (1 + 0.5 * math.log(2))) < 1e-12
    assert plain.query_temperature({}, 100) == 1.0


def test_costs_count_what_a_layer_has():
    """FLOPs and bytes per token of MIXED by hand: no value projection where keys are values, no entries where another layer's
    are read, two matrices an expert."""
    from llmgen_b200.engine.profiler import ModelCost
    cost = ModelCost.from_spec(spec_of(zu.MIXED))
    W = 48
    latent0 = W * (3 * 24 + 40 + 3 * 24) + 3 * 32 * (16 + 24)
    att1 = W * (64 + 64 + 32)
    latent2 = W * (2 * 20 + 2 * 10) + 2 * 32 * (12 + 10)
    att3 = W * (48 + 48 + 48)
    ffs = W * (6 + 2 * 2 * 24) + W * (5 + 2 * 3 * 16) + W * (3 + 2 * 3 * 20)
    assert cost.complete and cost.n_mm == latent0 + att1 + latent2 + att3 + ffs + W * 97
    assert [t.window for t in cost.attention] == [24, 0, 41, 0] and [t.stores for t in cost.attention] == [True, True, False, True]
    assert cost.kv_bytes_per_token() == 2 * (40 + 32 + 48)
