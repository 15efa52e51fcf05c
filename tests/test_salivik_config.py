"""The Salivik configuration class: what it reads, what it refuses, and the model it
describes (no GPU needed)."""
import copy
import math

import pytest

from janas_b200.config import ConfigError, SalivikConfig, config_from_dict, known_architectures
from janas_b200.weights import expected_tensors
from salivik_models import CONFIGS, tensor_shapes


def test_registered():
    assert "Salivik" in known_architectures()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_list_matches_the_design(name):
    c = config_from_dict(CONFIGS[name])
    assert isinstance(c, SalivikConfig)
    got = {n: tuple(s.shape) for n, s in expected_tensors(c.to_model_spec()).items() if not s.optional}
    assert got == {n: tuple(s) for n, s in tensor_shapes(CONFIGS[name]).items()}


def test_spec_describes_the_layers():
    c = config_from_dict(CONFIGS["SA"])
    assert c.loop == {"start": 1, "stop": 3, "times": 3} and c.norm_eps == 1e-6
    spec = c.to_model_spec()
    assert not spec.tie_embeddings and spec.head_name == "head" and spec.embedding_name == "embed"
    assert spec.embedding_norm.kind == "rmsnorm" and spec.embedding_norm_name == "embed.norm"
    assert spec.join_name == "loop.in"
    assert [(e.layer, e.join_embedding) for e in spec.run_order] == \
        [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False)]
    assert all(e.cache_of is None and not e.add_embedding for e in spec.run_order)
    l0, l1, l2 = spec.layers
    for l in spec.layers:
        assert l.block == "prenorm" and l.post_mixer_norm is None and l.post_ffn_norm is None
        assert l.mixer_norm.kind == "rmsnorm" and l.mixer_norm.get("names")["weight"] == ""
    m = l0.mixer
    assert m.kind == "latent_attention" and m.get("gate") is False and m.get("sink") is True and m.get("window") == 37
    pos = m.get("position")
    assert pos.kind == "rope_neox" and pos.get("rotary_dim") == 8
    assert pos.get("yarn") == {"factor": 4.0, "fast": 3.0, "original": 40.0, "slow": 0.5}
    unit = {"alpha": 1.702, "limit": 0.8, "shift": 1.0}
    assert l0.feed_forward.kind == "swiglu" and l0.feed_forward.get("unit") == unit
    m = l1.mixer
    assert m.kind == "sink_attention" and m.get("values_are_keys") is True and m.get("sink_score") == 0.0
    assert m.get("gate") is True and m.get("window") == 64 and m.get("position").get("rotary_dim") == 16
    assert m.get("position").get("yarn") is None
    f = l1.feed_forward
    assert f.kind == "routed" and f.get("experts") == 6 and f.get("top") == 2 and f.get("gated") is True
    assert f.get("score") == "chosen_softmax" and f.get("router_bias") is True and f.get("correction") is None
    assert f.get("unit")["limit"] == 1.5 and f.get("shared_unit")["limit"] == 0.7 and f.get("shared_ff") == 40
    m = l2.mixer
    assert m.kind == "decay_attention" and m.get("activation") == "none" and m.get("gate") == "silu"
    assert m.get("head_norm") is True and abs(m.get("key_scale") - 0.25) < 1e-12 and m.get("decay") == [0.5, 0.97, 0.999]
    assert l2.feed_forward.get("shared_ff") is None
    spec.validate()
    # what a model leaves out is off: no loop, no rotation, no window, no feed-forward
    e = config_from_dict(CONFIGS["SE"])
    assert e.loop is None
    se = e.to_model_spec()
    assert se.join_name == "" and [r.layer for r in se.run_order] == [0, 1, 2]
    assert se.layers[0].mixer.get("position").kind == "none" and se.layers[0].mixer.get("window") == 0
    assert se.layers[1].feed_forward is None and se.layers[1].ffn_norm is None


def test_spec_as_json_and_back():
    from janas_b200.config import ModelSpec
    for c in CONFIGS.values():
        spec = config_from_dict(c).to_model_spec()
        again = ModelSpec.from_json(spec.to_json())
        assert again.to_json() == spec.to_json() and again.run_order == spec.run_order
        again.validate()


def test_round_trip():
    for name, c in CONFIGS.items():
        d = config_from_dict(c).to_dict()
        assert config_from_dict(d).to_dict() == d
        assert d["vocab"] == c["vocab"] and d["width"] == c["width"] and d["loop"] == c.get("loop")
        for a, b in zip(d["layers"], c["layers"]):
            assert a["type"] == b["type"]
            for k, v in b["mixer"].items():
                assert a["mixer"][k] == v, (name, k)
            if b["mlp"] is None:
                assert a["mlp"] is None
            else:
                for k, v in b["mlp"].items():
                    assert a["mlp"][k] == v, (name, k)


def test_yarn_frequencies_by_hand():
    """The plain form's ramp: eight frequencies of which the first stay, the last are divided by the
    factor, and the ones between lie on the ramp."""
    import plain_salivik as ps
    rot = {"base": 10000.0, "dims": 16, "scaling": {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}}
    f = ps.frequencies(rot).tolist()
    base = [10000.0 ** (-i / 8) for i in range(8)]
    lo = math.floor(8 * math.log(2048 / (2 * math.pi * 32)) / math.log(10000.0))
    hi = math.ceil(8 * math.log(2048 / (2 * math.pi)) / math.log(10000.0))
    assert (lo, hi) == (2, 6)
    for i in range(8):
        ramp = min(max((i - 2) / 4, 0), 1)
        assert abs(f[i] - base[i] * ((1 - ramp) + ramp / 8)) < 1e-6 * base[i]
    assert abs(ps.amplitude(rot) - (0.1 * math.log(8) + 1)) < 1e-12


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0].update(type="mingru"), "mixers"),
    (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda d: d["layers"][1]["mixer"].update(vdim=16), "vdim"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=26), "at most"),
    (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=10), "at most"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0), "scaling"),
    (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda d: d["layers"][0]["mixer"].update(kv_rank=510), "512"),
    (lambda d: d["layers"][1]["mixer"].update(dim=600, vdim=600), "512"),
    (lambda d: d["layers"][2]["mixer"].update(decay=[0.5]), "decay"),
    (lambda d: d["layers"][2]["mixer"].pop("decay"), "decay"),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda d: d["layers"][1]["mlp"]["shared"].update(ff=0), "shared"),
    (lambda d: d["layers"][1]["mlp"]["expert"].update(limit=-1), "limit"),
    (lambda d: d["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda d: d["layers"][0]["mlp"].update(kind="relu"), "dense"),
    (lambda d: d["loop"].update(stop=4), "loop"),
    (lambda d: d["loop"].update(stop=1), "loop"),
    (lambda d: d["loop"].update(times=0), "loop"),
    (lambda d: d.pop("norm"), "norm"),
    (lambda d: d["layers"][1]["mixer"].pop("scale"), "scale"),
])
def test_refusals(change, word):
    d = copy.deepcopy(CONFIGS["SA"])
    change(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert word in str(e.value)


def test_a_join_needs_its_matrix():
    """A run order with a join, and a model that names no matrix for it, is refused."""
    spec = config_from_dict(CONFIGS["SA"]).to_model_spec()
    j = spec.to_json()
    j.pop("join_name")
    from janas_b200.config import ModelSpec
    with pytest.raises(ConfigError) as e:
        ModelSpec.from_json(j).validate()
    assert "join" in str(e.value)
