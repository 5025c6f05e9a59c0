"""Host-side parts of the Sarizen decoder: the configuration reader and its plan, the tensor names and shapes, what the layers
keep, the stretched rotation's frequencies, and the plain implementation's own mechanisms against brute force."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_sarizen as plain
import sarizen_models as M
from edgelm_b200.cache import SequenceCache
from edgelm_b200.config import ConfigError, config_class_for
from edgelm_b200.engine.model import DecoderModel
from edgelm_b200.parts import KVNeed, StateNeed
from edgelm_b200.parts.rope import rotary_frequencies, rotary_magnitude


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_plan_names_every_tensor_with_its_shape(name):
    cfg = M.CONFIGS[name]
    conf = config_class_for(cfg).from_dict(cfg)
    assert type(conf).__name__ == "SarizenConfig"
    W = M.tensors_for(cfg, 0)
    want = DecoderModel(conf.plan(), torch.float32).expected_weights()
    assert {k: tuple(v) for k, v in want.items()} == {k: tuple(v.shape) for k, v in W.items()}
    again = config_class_for(conf.to_dict()).from_dict(conf.to_dict())
    assert again.plan() == conf.plan()


def test_the_plan_reads_every_constant():
    plan = config_class_for(M.CFG_A).from_dict(M.CFG_A).plan()
    assert plan.hidden_size == 64 and plan.vocab_size == 171 and plan.head["tied_to"] is None
    assert plan.final_norm["scale"] == 0.7 and plan.final_norm["eps"] == 1e-5
    assert [e.layer for e in plan.schedule] == [0, 1, 2, 3] and all(l.block == "parallel_prenorm" for l in plan.layers)
    att = plan.layers[0].mixer
    assert att.kind == "latent_attention" and att["rot_pairs"] == "interleaved" and att["head_gate"] is True
    assert (att["num_heads"], att["head_dim"], att["rot_dim"], att["v_head_dim"], att["kv_rank"]) == (4, 16, 8, 24, 40)
    assert att["scale"] == 0.35 and att["rot_base"] == 700.0 and att["mask"] == {"kind": "window", "size": 21}
    assert att["rot_scaling"] == {"factor": 3.0, "original": 48.0, "fast": 6.0, "slow": 0.5}
    ffn = plan.layers[0].ffn
    assert ffn.kind == "moe" and (ffn["experts"], ffn["top"], ffn["intermediate_size"]) == (6, 2, 24) and ffn["weight_on"] == "input"
    assert ffn["router"] == {"kind": "scored", "score": "sigmoid", "renormalize": False}
    assert ffn["shared"].kind == "swiglu" and ffn["shared"]["intermediate_size"] == 32
    lin = plan.layers[1].mixer
    assert lin.kind == "decay_linear_attention" and (lin["heads"], lin["head_dim"], lin["v_head_dim"]) == (3, 24, 40)
    assert lin["decay"] == (0.3, 0.9, 0.998) and lin["activation"] == "silu" and lin["eps"] == 1e-5
    assert plan.layers[1].ffn.kind == "squared_relu" and plan.layers[1].ffn["intermediate_size"] == 72
    assert plan.layers[3].ffn["shared"] is None and plan.layers[3].ffn["top"] == 3
    b = config_class_for(M.CFG_B).from_dict(M.CFG_B).plan()
    assert b.final_norm["scale"] == 1.0 and b.layers[1].mixer["rot_scaling"] is None and b.layers[1].mixer["mask"]["size"] == 1
    assert b.layers[2].mixer["mask"] is None and b.layers[2].mixer["v_head_dim"] == 12 and b.layers[2].ffn is None and b.layers[2].ffn_norm is None


def test_refusals():
    for change, text in ((lambda c: c["layers"][0].update(type="attention"), "not part of this architecture"),
                         (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "kind 'glu'"),
                         (lambda c: c["layers"][0]["mixer"].pop("scale"), "'scale' is missing"),
                         (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "'kv_rank' is missing"),
                         (lambda c: c["layers"][0]["mixer"].pop("rot"), "'rot'"),
                         (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6), "rot_dim is 8"),
                         (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "'slow' is missing"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "window of 0"),
                         (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "one number per head"),
                         (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decays"),
                         (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "of 6 experts"),
                         (lambda c: c["layers"][0]["mlp"].pop("expert"), "'expert'"),
                         (lambda c: c.pop("norm"), "'norm'"),
                         (lambda c: c.update(logit_scale="big"), "logit_scale")):
        cfg = copy.deepcopy(M.CFG_A)
        change(cfg)
        with pytest.raises(ConfigError, match=text):
            DecoderModel(config_class_for(cfg).from_dict(cfg).plan(), torch.float32)


def test_what_the_layers_keep():
    """Latent rows (key and value at once) in pages for the attention layers, a matrix per head for the linear ones."""
    model = DecoderModel(config_class_for(M.CFG_A).from_dict(M.CFG_A).plan(), torch.bfloat16)
    needs = model.cache_needs()
    assert needs == [KVNeed(1, 48, None, v_head_dim=40, values_in_keys=True), StateNeed((3, 40, 24)),
                     KVNeed(1, 28, None, v_head_dim=24, values_in_keys=True), StateNeed((2, 16, 40))]
    cache = SequenceCache(needs, max_tokens=256, max_positions=1 << 20)
    s = cache.open()
    cache.reserve(s, 130)
    cache.advance(s, 130)
    cache.check()
    assert all(g.n_held[s] == 3 for g in cache.kv_groups)
    cache.close(s)
    cache.check()


def test_a_second_norm_without_a_feed_forward_may_be_stored():
    model = DecoderModel(config_class_for(M.CFG_B).from_dict(M.CFG_B).plan(), torch.float32)
    assert "l2.norm2" in model.ignorable_weights() and "l2.norm2" not in model.expected_weights() and "l1.norm2" not in model.ignorable_weights()


@pytest.mark.parametrize("dims,base,scaling", [(16, 100.0, (3.0, 64, 8.0, 1.0)), (64, 10000.0, (40.0, 4096, 32.0, 1.0)), (6, 50.0, (2.0, 4, 2.0, 1.0)),
                                               (8, 700.0, (5.0, 100000, 1.0, 0.5)), (10, 20.0, (1.0, 500, 20.0, 2.0)), (12, 300.0, None)])
def test_stretched_frequencies(dims, base, scaling):
    """The library's frequencies and lengths against the plain ones: the ramp inside the pairs, before the first (every pair
    stretched) and behind the last (none)."""
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    f, mult = plain.yarn_frequencies(dims, base, sc)
    assert np.allclose(rotary_frequencies(dims, base, sc).numpy(), f, rtol=1e-13, atol=0) and rotary_magnitude(sc) == pytest.approx(mult, abs=1e-15)


def test_stretched_frequencies_by_hand():
    # dims 8, base 16: p(t) = 8 ln(L / (2 pi t)) / (2 ln 16); L = 2 pi 16, fast 16 -> p = 0, slow 1 -> p = 4: ramp 0, 1/4, 1/2, 3/4
    sc = {"factor": 10.0, "original": 2.0 * math.pi * 16.0 * (1 + 1e-12), "fast": 16.0, "slow": 1.0 + 1e-9}
    f, mult = plain.yarn_frequencies(8, 16.0, sc)
    base = np.array([1.0, 0.5, 0.25, 0.125])
    ramp = np.array([0.0, 0.25, 0.5, 0.75])
    assert np.allclose(f, base / 10.0 * ramp + base * (1 - ramp)) and np.isclose(mult, 0.1 * math.log(10.0) + 1.0)


def test_plain_mechanisms_against_brute_force():
    g = np.random.default_rng(3)
    # neighbouring pairs: (0, 1) turns by position * f_0, position 0 only stretches by `mult`
    x = g.normal(size=(3, 1, 4))
    r = plain.rotate_neighbours(x, np.array([0, 3, 11]), np.array([1.0, 0.1]), 1.5)
    assert np.allclose(r[0], 1.5 * x[0])
    a = 11 * 0.1
    assert np.allclose(r[2, 0, 2], 1.5 * (x[2, 0, 2] * np.cos(a) - x[2, 0, 3] * np.sin(a)))
    assert np.allclose(r[2, 0, 3], 1.5 * (x[2, 0, 3] * np.cos(a) + x[2, 0, 2] * np.sin(a)))
    # the window: position 4 with a window of 2 sees 3 and 4; the sink is one more unit of weight without a value, and not scaled
    q, k, v = np.ones((5, 1, 1)), np.zeros((5, 1, 1)), np.arange(5.0).reshape(5, 1, 1)
    o = plain.window_softmax_attention(q, k, v, 9.0, 2, np.array([0.0]))
    assert np.isclose(o[4, 0, 0], (3.0 + 4.0) / 3.0) and np.isclose(o[0, 0, 0], 0.0)
    assert np.isclose(plain.window_softmax_attention(q, k, v, 9.0, 2, np.array([math.log(5.0)]))[4, 0, 0], 7.0 / 7.0)
    assert np.isclose(plain.window_softmax_attention(q, k, v, 9.0, None, None)[4, 0, 0], 2.0)
    # the linear attention as a sum over earlier tokens: o_t = sum_(s <= t) decay^(t - s) (q_t . k_s) v_s
    q, k, v = g.normal(size=(5, 1, 3)), g.normal(size=(5, 1, 3)), g.normal(size=(5, 1, 2))
    o = plain.decayed_linear_attention(q, k, v, np.array([0.8]))
    assert np.allclose(o[3, 0], sum(0.8 ** (3 - s) * (q[3, 0] @ k[s, 0]) * v[s, 0] for s in range(4)))
    # the router: sigmoids of the logits, each by itself, as they are
    chosen, wts = plain.route(np.array([[0.0, -1.0, 2.0, 1.0]]), 2)
    assert chosen.tolist() == [[2, 3]] and np.allclose(wts, [[1 / (1 + math.exp(-2.0)), 1 / (1 + math.exp(-1.0))]])
    # the weight multiplies the expert's input: with one channel silu(w a) * (w b), not w * silu(a) * b
    w = {"router": np.array([[0.0]]), "e0.gate": np.array([[3.0]]), "e0.up": np.array([[2.0]]), "e0.down": np.array([[1.0]])}
    y = plain.moe_ffn(np.array([[1.0]]), w, {"router": {"experts": 1, "top": 1}}, "")
    assert np.isclose(y[0, 0], plain.silu(1.5) * 1.0)
    # squared ReLU
    w = {"up": np.array([[2.0], [-2.0]]), "down": np.array([[1.0, 10.0]])}
    assert np.allclose(plain.squared_relu_ffn(np.array([[1.0], [-3.0]]), w, ""), [[4.0], [360.0]])


def test_plain_model_is_causal_and_sees_its_window():
    cfg = M.CFG_C
    W = M.tensors_for(cfg, 5)
    t = M.tokens(cfg, 20, 0)
    full, runs = plain.forward(cfg, W, t, return_layers=True)
    assert np.allclose(plain.forward(cfg, W, t[:13]), full[:13], atol=1e-9) and runs.shape == (3, 20, 48)
    # an attention layer alone forgets what left its window: the first token changes nothing from position `size` on
    one = {**cfg, "layers": [M.layer(M.latent(2, 8, 4, 8, 12, 50.0, None, 0.4, 6), None)]}
    W = M.tensors_for(one, 6)
    a, b = plain.forward(one, W, t), plain.forward(one, W, [(t[0] + 1) % 120] + t[1:])
    assert np.allclose(a[6:], b[6:], atol=1e-12) and np.abs(a[5] - b[5]).max() > 1e-6
