"""Host-side parts of the Semadra decoder: the configuration reader and its plan, the tensor names and shapes, what the layers
keep, and the plain implementation's own mechanisms against brute force."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_semadra as plain
import semadra_models as M
from edgelm_b200.cache import SequenceCache
from edgelm_b200.config import ConfigError, config_class_for
from edgelm_b200.engine.model import DecoderModel
from edgelm_b200.parts import KVNeed, NeedSet


def conf(cfg):
    return config_class_for(cfg).from_dict(cfg)


@pytest.mark.parametrize("name", sorted(M.CONFIGS))
def test_plan_names_every_tensor_with_its_shape(name):
    cfg = M.CONFIGS[name]
    c = conf(cfg)
    assert type(c).__name__ == "SemadraConfig"
    W = M.tensors_for(cfg, 0)
    want = DecoderModel(c.plan(), torch.float32).expected_weights()
    assert {k: tuple(v) for k, v in want.items()} == {k: tuple(v.shape) for k, v in W.items()}
    assert conf(c.to_dict()).plan() == c.plan()


def test_the_plan_reads_every_constant():
    plan = conf(M.CFG_A).plan()
    assert plan.hidden_size == 64 and plan.vocab_size == 173 and plan.embedding["scale"] == 2.5 and plan.head["tied_to"] == "embed"
    assert plan.final_norm.get("scale") is None and plan.final_norm["offset"] == 1.0 and plan.final_norm["eps"] == 1e-5
    assert [(e.layer, e.reads_cache_of) for e in plan.schedule] == [(0, None), (1, None), (2, 1), (3, None)]
    assert all(l.block == "sublayer_norm" for l in plan.layers)
    for l in plan.layers:
        assert l.mixer_norm["offset"] == 1.0 and l.mixer_norm["scale"] == 0.4 and l.mixer_norm["name"] == "norm1"
    att = plan.layers[0].mixer
    assert att.kind == "masked_attention" and (att["num_heads"], att["num_kv_heads"], att["head_dim"], att["v_head_dim"]) == (4, 2, 16, 24)
    assert att["scale"] == 0.3 and att["mask"] == {"kind": "window", "size": 21, "keep_first": 5} and not att.get("rot_dims")
    assert att["qk_norm"] == {"eps": 1e-5, "over": "projection"} and att["channel_gate"] is True
    lat = plan.layers[2].mixer
    assert lat.kind == "latent_attention" and (lat["num_heads"], lat["head_dim"], lat["rot_dim"], lat["v_head_dim"]) == (9, 8, 0, 12)
    assert (lat["q_rank"], lat["kv_rank"], lat["scale"]) == (28, 40, 0.5) and lat["mask"] == {"kind": "window", "size": 64} and lat["reads_cache"]
    ffn = plan.layers[0].ffn
    assert ffn.kind == "moe" and (ffn["experts"], ffn["top"], ffn["intermediate_size"]) == (8, 2, 24) and ffn.get("weight_on", "output") == "output"
    assert ffn["router"] == {"kind": "scored", "score": "sigmoid", "renormalize": False, "scale": 1.5, "groups": 4, "keep": 2, "group_score": "top2_sum"}
    assert ffn["shared"].kind == "swiglu" and ffn["shared"]["intermediate_size"] == 40
    assert plan.layers[1].ffn.kind == "swiglu" and plan.layers[3].ffn is None and plan.layers[2].ffn["shared"] is None
    for i, l in enumerate(plan.layers):
        (side, norm), = l.options["after"]
        assert side.kind == "token_side" and (side["dim"], side["columns"], side["first_column"]) == (12, 48, 12 * i)
        assert norm["name"] == "side.norm" and norm.get("offset") is None and norm["scale"] == 0.4
    b = conf(M.CFG_B).plan()
    assert b.embedding["scale"] == 1.0 and "after" not in b.layers[0].options and b.layers[1].mixer["mask"] is None
    assert b.layers[3].mixer["mask"]["keep_first"] == 0 and b.layers[0].ffn["router"]["groups"] == 1 and b.layers[0].ffn["router"]["scale"] == 1.0
    assert b.layers[0].mixer["v_head_dim"] == 10 and b.layers[0].mixer_norm["scale"] == 1.0


def test_refusals():
    for change, text in ((lambda c: c["layers"][0].update(type="lightning"), "not part of this architecture"),
                         (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "kind 'glu'"),
                         (lambda c: c["layers"][0]["mixer"].pop("scale"), "'scale' is missing"),
                         (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
                         (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "not a multiple"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "window of 0"),
                         (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "-1 kept"),
                         (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "kv_from 0"),
                         (lambda c: c["layers"][2]["mixer"].update(kv_from=3), "kv_from 3"),
                         (lambda c: c["layers"][2]["mixer"].update(kv_rank=41), "kv_rank differs"),
                         (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "of 8 experts"),
                         (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3), "in 3 groups"),
                         (lambda c: c["layers"][0]["mlp"]["router"]["groups"].pop("keep"), "'keep' is missing"),
                         (lambda c: c["layers"][0]["mlp"].pop("expert"), "'expert'"),
                         (lambda c: c["token_side"].pop("dim"), "'dim' is missing"),
                         (lambda c: c.pop("norm"), "'norm'"),
                         (lambda c: c.update(residual_mult="half"), "residual_mult")):
        cfg = copy.deepcopy(M.CFG_A)
        change(cfg)
        with pytest.raises(ConfigError, match=text):
            DecoderModel(conf(cfg).plan(), torch.float32)


def test_a_query_latent_that_only_the_tensors_size():
    cfg = copy.deepcopy(M.CFG_A)
    for i in (1, 2):
        cfg["layers"][i]["mixer"].pop("q_rank")
    c = conf(cfg).shape_given_sizes({k: v.shape for k, v in M.tensors_for(M.CFG_A, 0).items()})
    assert c.plan() == conf(M.CFG_A).plan()


def test_what_the_layers_keep():
    """Keys and values for the attention layers, latent rows for the latent layers that have one of their own, nothing for a reader."""
    model = DecoderModel(conf(M.CFG_A).plan(), torch.bfloat16)
    kv = lambda *a, **k: NeedSet.of(mixer=KVNeed(*a, **k))
    needs = model.cache_needs()
    assert needs == [kv(2, 16, None, v_head_dim=24), kv(1, 40, None, v_head_dim=40, values_in_keys=True), None, kv(6, 24, None, v_head_dim=8)]
    cache = SequenceCache(needs, max_tokens=256, max_positions=1 << 20)
    s = cache.open()
    cache.reserve(s, 130)
    cache.advance(s, 130)
    cache.check()
    assert all(g.n_held[s] == 3 for g in cache.kv_groups)
    cache.close(s)
    cache.check()


def test_a_second_norm_without_a_feed_forward_may_be_stored():
    model = DecoderModel(conf(M.CFG_A).plan(), torch.float32)
    assert "l3.norm2" in model.ignorable_weights() and "l3.norm2" not in model.expected_weights() and "l1.norm2" not in model.ignorable_weights()


def test_plain_mechanisms_against_brute_force():
    g = np.random.default_rng(3)
    # the mask: position 9 with a window of 3 and 2 kept tokens sees 0, 1 and 7, 8, 9; position 3 all but none twice
    see = plain.visible(10, {"size": 3, "keep_first": 2})
    assert np.nonzero(see[9])[0].tolist() == [0, 1, 7, 8, 9] and np.nonzero(see[3])[0].tolist() == [0, 1, 2, 3]
    assert np.nonzero(plain.visible(10, {"size": 3})[9])[0].tolist() == [7, 8, 9] and plain.visible(5, None)[4].all()
    # equal scores: the mean of the visible values; a query head uses the key head of its group
    q, k, v = np.ones((5, 4, 1)), np.zeros((5, 2, 1)), np.stack([np.arange(5.0), 10 * np.arange(5.0)], 1).reshape(5, 2, 1)
    o = plain.softmax_attention(q, k, v, 3.0, {"size": 2, "keep_first": 1})
    assert np.allclose(o[4, :, 0], [7 / 3, 7 / 3, 70 / 3, 70 / 3])
    # the norm over the whole projection differs from one per head, the gate from one per head
    m = {"heads": 2, "dim": 1, "scale": 1.0}
    W = {"q": np.array([[3.0], [4.0]]), "k": np.eye(2)[:, :1] + 1.0, "v": np.array([[1.0], [1.0]]), "q.norm": np.ones(2), "k.norm": np.ones(2),
         "g": np.array([[0.0], [50.0]]), "o": np.array([[1.0, 10.0]])}
    assert np.isclose(plain.attention_mixer(np.array([[1.0]]), W, m, "", 0.0)[0, 0], 0.5 + 10.0)
    assert np.allclose(plain.rms_norm(np.array([[3.0, 4.0]]), 0.0), np.array([[3.0, 4.0]]) / math.sqrt(12.5))
    # a latent of another layer: keys and values from it, queries from the layer's own input
    c = np.array([[1.0], [2.0]])
    W = {"dq": np.array([[1.0]]), "dq.norm": np.ones(1), "uq": np.array([[0.0]]), "uk": np.array([[1.0]]), "uv": np.array([[5.0]]), "o": np.array([[1.0]])}
    y = plain.latent_attention_mixer(np.array([[1.0], [1.0]]), c, W, {"heads": 1, "dim": 1, "q_rank": 1, "kv_rank": 1, "scale": 1.0}, "", 1e-9)
    assert np.allclose(y[:, 0], [5.0, 7.5])
    # the router: groups of two; group worths 0.9 + 0.1, 0.6 + 0.5, 0.7 + 0.05: the best single score's group is second
    s = np.array([[0.9, 0.1, 0.6, 0.5, 0.7, 0.05]])
    z = np.log(s / (1 - s))
    chosen, wts = plain.route(z, 2, {"count": 3, "keep": 1}, 2.0)
    assert chosen.tolist() == [[2, 3]] and np.allclose(wts, [[1.2, 1.0]])
    chosen, wts = plain.route(z, 3, {"count": 3, "keep": 2}, 1.0)
    assert chosen.tolist() == [[0, 2, 3]] and np.allclose(wts, [[0.9, 0.6, 0.5]])
    assert plain.route(z, 2)[0].tolist() == [[0, 4]]
    # the token input: layer 1's slice of the table, the activation's tanh form, a plain norm weight
    assert np.isclose(plain.gelu_tanh(1.0), 0.8411919906) and np.isclose(plain.gelu_tanh(-2.0), -0.0454023059)
    W = {"side.embed": np.array([[1.0, 2.0], [3.0, 4.0]]), "l1.side.gate": np.array([[1.0]]), "l1.side.proj": np.array([[1.0]]), "l1.side.norm": np.array([0.5])}
    y = plain.token_side(np.array([[1.0]]), [1], W, "l1.", 1, 1, 100.0)
    u = plain.gelu_tanh(1.0) * 4.0
    assert np.isclose(y[0, 0], 0.5 * u / math.sqrt(u * u + 100.0))
    g.normal()


def test_plain_model_is_causal_and_sees_its_window():
    cfg = M.CFG_C
    W = M.tensors_for(cfg, 5)
    t = M.tokens(cfg, 20, 0)
    full, runs = plain.forward(cfg, W, t, return_layers=True)
    assert np.allclose(plain.forward(cfg, W, t[:13]), full[:13], atol=1e-9) and runs.shape == (5, 20, 48)
    # one attention layer forgets a token that left its window, but not one of the kept first ones
    one = M.model(120, 48, 1e-6, [M.layer(M.attention(2, 1, 8, 8, 0.4, 6, 2), None)])
    W = M.tensors_for(one, 6)
    base = plain.forward(one, W, t)
    for at, forgotten in ((2, True), (1, False)):
        moved = np.abs(plain.forward(one, W, t[:at] + [(t[at] + 1) % 120] + t[at + 1:]) - base).max(axis=1)
        assert moved[at + 5] > 1e-6 and (moved[at + 6:] < 1e-12).all() == forgotten
