"""The Dafalix configuration class: what it reads, what it refuses, and the model it
describes (no GPU needed)."""
import copy

import pytest
import torch

from janas_b200.config import ConfigError, DafalixConfig, ModelSpec, config_from_dict, known_architectures
from janas_b200.weights import expected_tensors
from dafalix_models import CONFIGS, tensor_shapes


def test_registered():
    assert "Dafalix" in known_architectures()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_list_matches_the_design(name):
    c = config_from_dict(CONFIGS[name])
    assert isinstance(c, DafalixConfig)
    listed = expected_tensors(c.to_model_spec())
    got = {n: tuple(s.shape) for n, s in listed.items() if not s.optional}
    assert got == {n: tuple(s) for n, s in tensor_shapes(CONFIGS[name]).items()}
    # what surrounds an absent feed-forward may stand in a file; the head is the embedding table
    absent = [f"l{i}." for i, l in enumerate(CONFIGS[name]["layers"]) if l["mlp"] is None]
    leaves = ("norm2", "norm2.b", "ls2", "hc2.in", "hc2.out", "hc2.mix")
    assert {n for n, s in listed.items() if s.optional} == {"head"} | {p + x for p in absent for x in leaves}


def test_spec_describes_the_layers():
    c = config_from_dict(CONFIGS["FA"])
    assert c.loop == {"start": 1, "stop": 3, "times": 3} and c.streams == 3 and c.residual_mult == 0.8
    spec = c.to_model_spec()
    assert spec.tie_embeddings and spec.embedding_name == "embed" and spec.streams == 3 and spec.embedding_norm is None
    assert [e.layer for e in spec.run_order] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert all(e.cache_of is None and not e.add_embedding and not e.join_embedding for e in spec.run_order)
    for l in spec.layers:
        assert l.block == "streams" and l.block_params["streams"] == 3 and l.block_params["residual_mult"] == 0.8
        assert l.mixer_norm.kind == "layernorm" and l.mixer_norm.get("names") == {"weight": "", "bias": "b"}
        assert l.mixer_norm.get("eps") == 1e-6
    m = spec.layers[0].mixer
    assert m.kind == "mlstm" and m.get("head_dim") == 16 and m.get("v_head_dim") == 24 and m.get("gate_cap") == 8.0
    m = spec.layers[1].mixer
    assert m.kind == "pair" and m.get("join") == "sum" and m.get("left_scale") == 0.7 and m.get("right_scale") == 1.2
    a, r = m.get("left"), m.get("right")
    assert a.kind == "sink_attention" and a.get("window") == 37 and a.get("v_head_dim") == 16 and a.get("sink") is None
    pos = a.get("position")
    assert pos.kind == "rope_neox" and pos.get("rotary_dim") == 16 and pos.get("linear_factor") == 2.5
    assert r.kind == "rglru" and r.get("width") == 48 and r.get("blocks") == 3 and r.get("conv_taps") == 4
    f = spec.layers[2].feed_forward
    assert f.kind == "routed" and f.get("experts") == 5 and f.get("top") == 3 and f.get("weight_on_input") is True
    assert f.get("score") == "sigmoid" and f.get("gated") is True and f.get("correction") is None
    spec.validate()
    # what a model leaves out is off: no loop, no rotation, no window, no feed-forward
    e = config_from_dict(CONFIGS["FE"])
    assert e.loop is None
    se = e.to_model_spec()
    assert [r.layer for r in se.run_order] == [0, 1, 2]
    assert se.layers[0].mixer.get("left").get("position") is None and se.layers[0].mixer.get("left").get("window") == 0
    assert se.layers[1].feed_forward is None and se.layers[1].ffn_norm is None


def test_spec_as_json_and_back():
    for c in CONFIGS.values():
        spec = config_from_dict(c).to_model_spec()
        again = ModelSpec.from_json(spec.to_json())
        assert again.to_json() == spec.to_json() and again.run_order == spec.run_order and again.streams == c["streams"]
        again.validate()


def test_round_trip():
    for name, c in CONFIGS.items():
        d = config_from_dict(c).to_dict()
        assert config_from_dict(d).to_dict() == d
        assert d["loop"] == c.get("loop")
        for k in ("vocab", "width", "streams", "residual_mult", "norm", "layers"):
            assert d[k] == c[k], (name, k)


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0].update(type="mingru"), "mixers"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"].update(dims=26), "at most"),
    (lambda d: d["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "factor"),
    (lambda d: d["layers"][1]["mixer"]["left"]["mask"].update(size=0), "mask.size"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(dim=600), "512"),
    (lambda d: d["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda d: d["layers"][1]["mixer"].pop("right"), "right"),
    (lambda d: d["layers"][1]["mixer"]["right"].update(blocks=5), "divide"),
    (lambda d: d["layers"][1]["mixer"]["right"].update(conv=0), "conv"),
    (lambda d: d["layers"][0]["mixer"].update(dim=1025), "1024"),
    (lambda d: d["layers"][0]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda d: d["layers"][0]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "moe"),
    (lambda d: d["loop"].update(stop=5), "loop"),
    (lambda d: d["loop"].update(stop=1), "loop"),
    (lambda d: d["loop"].update(times=0), "loop"),
    (lambda d: d.update(streams=0), "streams"),
    (lambda d: d.update(streams=33), "streams"),
    (lambda d: d.pop("norm"), "norm"),
])
def test_refusals(change, word):
    d = copy.deepcopy(CONFIGS["FA"])
    change(d)
    with pytest.raises(ConfigError) as e:
        config_from_dict(d)
    assert word in str(e.value)


def test_streams_and_arrangement_go_together():
    """Several streams take no second embedding output, and their count is the layers' own."""
    j = config_from_dict(CONFIGS["FE"]).to_model_spec().to_json()
    j["run_order"][1]["add_embedding"] = True
    with pytest.raises(ConfigError) as e:
        ModelSpec.from_json(j).validate()
    assert "streams" in str(e.value)
    j = config_from_dict(CONFIGS["FE"]).to_model_spec().to_json()
    j["streams"] = 3
    with pytest.raises(Exception) as e:
        expected_tensors(ModelSpec.from_json(j))
    assert "streams" in str(e.value)


def test_plain_recurrences_by_hand():
    """The plain forms on numbers small enough to follow."""
    import plain_dafalix as pd
    # one head, one value: a forget gate of one and inputs of weight one are a running sum
    o, (m, n, S) = pd.mlstm_scan(torch.ones(3, 1, 1), torch.ones(3, 1, 1), torch.tensor([1.0, 2.0, 6.0]).view(3, 1, 1),
                                 torch.zeros(3, 1), torch.zeros(3, 1))
    assert torch.allclose(o.flatten(), torch.tensor([1.0, 1.5, 3.0]), atol=1e-5) and float(m) == 0.0 and float(n) == 3.0
    # a strong input gate raises the maximum and drowns what came before
    i = torch.tensor([[0.0], [9.0]])
    o, (m, _, _) = pd.mlstm_scan(torch.ones(2, 1, 1), torch.ones(2, 1, 1), torch.tensor([1.0, 5.0]).view(2, 1, 1), i, torch.zeros(2, 1))
    assert float(m) == 9.0 and abs(float(o[1]) - 5.0) < 1e-2
    # r = 0: nothing decays and nothing enters; a large lam: the state is the input alone
    u = torch.tensor([[2.0], [3.0]])
    S, _ = pd.lru_scan(u, torch.zeros(2, 1), torch.ones(2, 1), torch.zeros(1), torch.tensor([7.0]))
    assert torch.equal(S, torch.full((2, 1), 7.0))
    S, _ = pd.lru_scan(u, torch.ones(2, 1), torch.ones(2, 1), torch.full((1,), 30.0))
    assert torch.allclose(S, u)
    # streams: from and to are not the same
    X = torch.tensor([[[1.0], [10.0]]])
    out = pd.write_streams(X, torch.tensor([[100.0]]), torch.tensor([[0.0, 1.0], [2.0, 0.0]]), torch.tensor([1.0, 0.0]), 0.5)
    assert out.flatten().tolist() == [70.0, 1.0]
