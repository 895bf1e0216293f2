"""Tudulix without a GPU: configuration, the run order of a loop, tensor list, refusals, cache needs, and the oracle's
mechanisms on inputs with known answers."""
import copy
import math

import pytest
import torch

import tudulix_tiny as tt
from plain import tudulix_plain as plain
from prelude_b200.config import ConfigError, load_model_config
from prelude_b200.config.spec import (GqaSpec, LatentAttentionSpec, LayerCall, NormSpec, RotaryRatesSpec, RoutedExpertsSpec,
                                      ScaledEmbeddingSpec, looped_order)
from prelude_b200.parts.model import DecoderModel
from prelude_b200.parts.registry import KvPagesNeed
from prelude_b200.weights.loader import WeightStore


def test_every_layer_is_parsed_on_its_own():
    spec = load_model_config(tt.TUDULIX_A).to_model_spec()
    assert spec.architecture == "Tudulix" and spec.vocab_size == 103 and spec.hidden_size == 44
    assert not spec.tie_embeddings and not spec.head.tied and spec.head.name == "head"
    assert spec.embedding == ScaledEmbeddingSpec(103, 44, 3.5, name="embed")
    norm = NormSpec(dim=44, eps=1e-5, suffix="", offset=1.0)
    assert spec.final_norm == NormSpec(dim=44, eps=1e-5, suffix="", offset=1.0, gain=1.7) and spec.final_norm_name == "final.norm"
    assert [type(b.mixer) for b in spec.blocks] == [GqaSpec, LatentAttentionSpec, GqaSpec, LatentAttentionSpec, LatentAttentionSpec]
    assert all(b.kind == "sandwich_residual" and b.mixer_norm == norm and b.mixer_post_norm == norm for b in spec.blocks)
    att = spec.blocks[0].mixer
    assert (att.num_heads, att.num_kv_heads, att.head_dim, att.value_dim, att.softmax_scale, att.window) == (6, 2, 10, 7, 0.4, 9)
    assert att.position == RotaryRatesSpec(dims=6, base=50.0, adjacent=True)
    assert not att.qkv_bias and att.whole_qk_norm_eps is None and not att.sink
    lat = spec.blocks[1].mixer
    assert (lat.num_heads, lat.head_dim, lat.rot_dim, lat.value_dim, lat.kv_rank, lat.softmax_scale, lat.window) == (3, 10, 6, 7, 13, 0.4, 13)
    assert lat.q_rank is None and lat.element_gate and not lat.head_gate and not lat.sink and lat.norm_eps == 1e-5
    assert lat.position == RotaryRatesSpec(dims=6, base=50.0, adjacent=False) and spec.blocks[3].mixer.window is None
    ff = spec.blocks[0].feed_forward
    assert isinstance(ff, RoutedExpertsSpec)
    assert (ff.n_experts, ff.top_k, ff.expert_size, ff.limit, ff.shared_size, ff.shared_limit, ff.alpha) == (5, 2, 11, 0.9, 14, 0.6, 1.702)
    assert (ff.scoring, ff.activation, ff.renormalize, ff.weight_scale, ff.n_groups, ff.router_bias_name, ff.correction_name) == \
        ("softmax_chosen", "clamped_glu", False, 1.0, 1, "router.b", None)
    assert spec.blocks[1].feed_forward.shared_size is None and spec.blocks[2].feed_forward is None and spec.blocks[2].ff_post_norm is None


def test_a_loop_becomes_entries_of_the_run_order():
    def runs(cfg):
        return [(c.block, c.adds_embedding, c.cache, c.writes_cache) for c in load_model_config(cfg).to_model_spec().resolved_order()]

    assert runs(tt.TUDULIX_A) == [(0, False, 0, True), (1, False, 1, True), (2, False, 2, True), (3, False, 3, True), (1, True, 4, True),
                                  (2, False, 5, True), (3, False, 6, True), (1, True, 7, True), (2, False, 8, True), (3, False, 9, True),
                                  (4, False, 10, True)]
    assert [r[:2] for r in runs(tt.TUDULIX_B)] == [(0, False), (1, False), (2, False), (0, True), (1, False), (2, False), (3, False)]
    assert [r[:2] for r in runs(tt.TUDULIX_C)] == [(0, False), (1, False), (2, False)]
    assert [r[:2] for r in runs(tt.TUDULIX_D)] == [(0, False), (1, False)]
    for cfg in (tt.TUDULIX_A, tt.TUDULIX_B, tt.TUDULIX_C, tt.TUDULIX_D):
        assert [r[:2] for r in runs(cfg)] == plain.run_order(cfg)
    assert looped_order(2, 1, 2, 2) == (LayerCall(0), LayerCall(1), LayerCall(1, adds_embedding=True))
    for bad in ((2, 1, 1, 2), (2, 0, 3, 1), (2, -1, 1, 1), (2, 0, 1, 0)):
        with pytest.raises(ValueError):
            looped_order(*bad)


def test_every_pass_has_a_cache_of_its_own():
    model = DecoderModel(load_model_config(tt.TUDULIX_A).to_model_spec())
    needs = model.cache_needs()
    assert len(needs) == 11
    assert needs[0] == KvPagesNeed(2, 10, 9, v_heads=2, v_head_dim=7)
    assert needs[1] == needs[4] == needs[7] == KvPagesNeed(1, 19, 13, v_heads=0, v_head_dim=0)
    assert needs[2] == needs[5] == needs[8] == KvPagesNeed(3, 9, 21)
    assert needs[3] == KvPagesNeed(1, 15, None, v_heads=0, v_head_dim=0)
    caps = model.runtime_caps()
    assert caps.kv_cache and not caps.state_slots and caps.cuda_graph


def test_tensor_list_has_the_designs_names_and_shapes():
    req, opt = DecoderModel(load_model_config(tt.TUDULIX_A).to_model_spec()).tensors()
    want = {"embed": (103, 44), "head": (103, 44), "final.norm": (44,), "l0.norm1": (44,), "l0.norm1b": (44,), "l0.norm2": (44,),
            "l0.norm2b": (44,), "l0.mix.q": (60, 44), "l0.mix.k": (20, 44), "l0.mix.v": (14, 44), "l0.mix.o": (44, 42),
            "l1.mix.q": (48, 44), "l1.mix.dkv": (19, 44), "l1.mix.dkv.norm": (13,), "l1.mix.uk": (30, 13), "l1.mix.uv": (21, 13),
            "l1.mix.g": (21, 44), "l1.mix.o": (44, 21), "l0.mlp.router": (5, 44), "l0.mlp.router.b": (5,), "l0.mlp.e0.gate": (11, 44),
            "l0.mlp.e4.up": (11, 44), "l0.mlp.e4.down": (44, 11), "l0.mlp.shared.gate": (14, 44), "l0.mlp.shared.up": (14, 44),
            "l0.mlp.shared.down": (44, 14)}
    for name, shape in want.items():
        assert tuple(req[name].shape) == shape, name
    assert not opt and req["l0.norm1b"].role == "norm_zero" and req["l1.mix.dkv.norm"].role == "norm"
    assert not any(n.startswith(("l2.norm2", "l2.mlp", "l4.norm2", "l4.mlp", "l1.mlp.shared")) for n in req)


def test_norms_around_a_feed_forward_that_is_not_there_are_passed_over():
    spec = load_model_config(tt.TUDULIX_A).to_model_spec()
    req, opt = DecoderModel(spec).tensors()
    tensors = tt.tensors_of(tt.TUDULIX_A, seed=1)
    tensors["l2.norm2"] = tensors["l2.norm2b"] = torch.zeros(44)
    WeightStore.from_tensors(tensors).check(req, opt, spec.ignored_tensors)
    tensors["l0.norm3"] = torch.ones(44)
    with pytest.raises(ValueError) as e:
        WeightStore.from_tensors(tensors).check(req, opt, spec.ignored_tensors)
    assert "l0.norm3" in str(e.value) and "l2.norm2" not in str(e.value)


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][1].update(type="window"), "unknown layer type"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "at most the 10 elements"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "at most the 6 elements"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "positive integer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "unknown kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top=6 of 5"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(limit=-1.0), "limit"),
    (lambda c: c["loop"].update(start=4), "are not layers of 5"),
    (lambda c: c["loop"].update(stop=6), "are not layers of 5"),
    (lambda c: c["loop"].update(start=-1), "number of a layer"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c.update(loop=3), "must be an object"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "non-empty"),
])
def test_a_configuration_that_cannot_be_run_is_refused_with_the_reason(change, word):
    cfg = copy.deepcopy(tt.TUDULIX_A)
    change(cfg)
    with pytest.raises(ConfigError) as e:
        load_model_config(cfg)
    assert word in str(e.value)


def test_the_feed_forward_hands_its_sum_to_the_norms_that_follow():
    model = DecoderModel(load_model_config(tt.TUDULIX_B).to_model_spec())
    assert all(b.feed_forward.defer_output for b in model.blocks)


# -- the oracle's mechanisms on inputs with known answers ----------------------------------------------------------------
def test_plain_norm_is_stored_around_zero():
    y = plain.norm_around_one(torch.tensor([[3.0, 4.0]], dtype=torch.float64), torch.tensor([0.0, -0.5], dtype=torch.float64), 0.0)
    r = math.sqrt(12.5)
    assert torch.allclose(y, torch.tensor([[3.0 / r, 2.0 / r]], dtype=torch.float64), atol=1e-14)


def test_plain_rotation_in_both_layouts():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=torch.float64)
    c0, s0, c1, s1 = math.cos(3.0), math.sin(3.0), math.cos(0.75), math.sin(0.75)
    y = plain.turn(x, torch.tensor([3]), 4, 16.0, True).reshape(-1)
    assert torch.allclose(y, torch.tensor([1 * c0 - 2 * s0, 2 * c0 + 1 * s0, 3 * c1 - 4 * s1, 4 * c1 + 3 * s1, 5.0], dtype=torch.float64), atol=1e-14)
    y = plain.turn(x, torch.tensor([3]), 4, 16.0, False).reshape(-1)
    assert torch.allclose(y, torch.tensor([1 * c0 - 3 * s0, 2 * c1 - 4 * s1, 3 * c0 + 1 * s0, 4 * c1 + 2 * s1, 5.0], dtype=torch.float64), atol=1e-14)


def test_plain_window_counts_the_token_itself():
    hidden = plain.hidden_keys(6, 3)
    assert [j for j in range(6) if not hidden[5, j]] == [3, 4, 5] and [j for j in range(6) if not hidden[1, j]] == [0, 1]
    assert not plain.hidden_keys(4, None)[3, 0] and plain.hidden_keys(4, None)[0, 1] and plain.hidden_keys(4, 1)[2].tolist() == [True, True, False, True]


def test_plain_clamped_unit():
    a, b = torch.tensor([5.0, -3.0], dtype=torch.float64), torch.tensor([-9.0, 0.5], dtype=torch.float64)
    want = [2.0 / (1 + math.exp(-3.404)) * (-2.0 + 1.0), -3.0 / (1 + math.exp(5.106)) * 1.5]
    assert torch.allclose(plain.clamped_unit(a, b, 2.0), torch.tensor(want, dtype=torch.float64), atol=1e-14)


def test_plain_router_weighs_the_chosen_alone():
    ids, w = plain.route(torch.tensor([[1.0, -2.0, 3.0, 2.5]], dtype=torch.float64), 2)
    assert ids[0].tolist() == [2, 3] and abs(float(w[0, 0]) - 1 / (1 + math.exp(-0.5))) < 1e-14 and abs(float(w.sum()) - 1) < 1e-14
    assert abs(float(plain.route_margin(torch.tensor([[1.0, -2.0, 3.0, 2.5]]), 2)) - 1.5) < 1e-6


def test_plain_loop_adds_the_embedding_before_every_pass_but_the_first():
    """With all sublayers silent (their norms' scales at zero) the stream is the embedding's output times one plus the passes
    behind the first."""
    cfg = tt.TUDULIX_A
    tensors = {k: (torch.full_like(v, -1.0) if k.endswith(("norm1b", "norm2b")) else v) for k, v in tt.tensors_of(cfg, seed=2).items()}
    layers = []
    plain.forward(cfg, tensors, [4, 9], layers_out=layers)
    start = tensors["embed"].double()[[4, 9]] * 3.5
    assert len(layers) == 11
    for n, x in enumerate(layers):
        assert torch.allclose(x, start * (1 if n < 4 else 2 if n < 7 else 3)), n
