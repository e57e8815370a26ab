"""The Laperax design's configuration, layout and cache plan, on the host."""
import json

import pytest
import torch

from plain import laperax_plain as P
from test_gpu_laperax import _att, _config, _del, _moe, _ret


def _layers():
    return [_ret(), _att(), _del(mlp=None), _att(size=None, rot=None), _ret(heads=1, decay=[1.0], rot=None)]


def _edit(config, path, value=None, delete=False):
    bad = json.loads(json.dumps(config))
    node = bad
    for key in path[:-1]:
        node = node[key]
    if delete:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return bad


def test_config_errors_name_the_key():
    from picolm_b200.config import ConfigError, config_from_dict
    good = _config(_layers())
    assert config_from_dict(good).to_dict() == good
    ret, att, dlt = (("layers", i, "mixer") for i in range(3))
    for path, value, word in ((("layers", 0, "type"), "lstm", "lstm"), (att + ("kv_heads",), 3, "kv_heads"), (att + ("scale",), 0, "scale"),
                              (att + ("mask", "size"), 0, "size"), (att + ("rot", "dims"), 7, "dims"), (att + ("rot", "dims"), 18, "dims"),
                              (att + ("rot", "base"), 0, "base"), (ret + ("rot", "base"), "x", "base"), (ret + ("decay",), [0.5], "decay"),
                              (ret + ("decay",), 0.5, "decay"), (ret + ("decay",), [0.5, 1.5, 0.1], "decay"), (ret + ("vdim",), "x", "vdim"),
                              (dlt + ("conv",), 0, "conv"), (dlt + ("kv_heads",), 3, "kv_heads"), (("layers", 0, "mlp", "kind"), "odd", "odd"),
                              (("layers", 1, "mlp", "router", "top"), 9, "top"), (("layers", 1, "mlp", "expert", "ff"), 0, "ff"),
                              (("layers", 0, "mlp", "router", "scale"), "x", "scale"), (("logit_softcap",), 0, "logit_softcap"),
                              (("logit_scale",), "x", "logit_scale"), (("norm", "eps"), -1, "eps"), (("width",), 0, "width"), (("layers",), [], "layers")):
        with pytest.raises(ConfigError, match=word):
            config_from_dict(_edit(good, path, value))
    for path in (("norm", "eps"), ("vocab",), ("logit_scale",), ("logit_softcap",), ret + ("decay",), ret + ("dim",), ret + ("rot", "dims"), att + ("scale",),
                 att + ("mask", "size"), dlt + ("conv",), ("layers", 0, "mlp", "expert"), ("layers", 1, "mlp", "router", "experts"),
                 ("layers", 1, "mlp", "router", "scale")):
        with pytest.raises(ConfigError, match=str(path[-1])):
            config_from_dict(_edit(good, path, delete=True))


def test_layout_and_cache_plan():
    """One norm a layer; keys and values for the attention layers alone (a group by its window and head sizes), the
    recurrences' states (the delta rule's with the convolution's last inputs) for the others; a layer without
    feed-forward has no tensors of one."""
    from picolm_b200.config import config_from_dict, spec_of
    from picolm_b200.engine.model import Model
    spec = spec_of(config_from_dict(_config(_layers())))
    assert [layer.arrangement for layer in spec.layers] == ["parallel_norm"] * 5
    assert set(spec.layers[0].parts) == {"mixer_norm", "mixer", "feed_forward"} and set(spec.layers[2].parts) == {"mixer_norm", "mixer"}
    model = Model(spec, None)
    names = model.expected_tensors()
    assert {"embed", "embed.norm", "head", "final.norm", "l0.norm1", "l0.mix.g", "l0.mlp.router", "l1.mlp.e4.down", "l1.mix.o", "l2.mix.q.conv",
            "l2.mix.A_log", "l2.mix.norm"} <= set(names)
    assert not any(n.startswith("l2.mlp") or "norm2" in n or n.endswith(("gate", "q.norm", "k.norm")) for n in names)
    assert "l0.mix.norm" not in names and "l1.mix.g" not in names
    assert names["l2.mix.a"].shape == (4, 40) and names["l2.mix.dt_bias"].shape == (4,) and names["l2.mix.g"].shape == (80, 40)
    assert names["l2.mix.v.conv"].shape == (80, 3) and names["l1.mix.o"].shape == (40, 96) and names["l0.mix.o"].shape == (40, 60)
    specs = model.cache_specs()
    assert [(s.kind, s.window) for s in specs if s.kind == "kv"] == [("kv", 21), ("kv", None)]
    assert [s.shape for s in specs if s.kind == "state"] == [(3 * 12 * 20,), (4 * 12 * 20 + 2 * (2 * 24 + 80),), (12 * 20,)]


def test_parts_refuse_what_does_not_fit():
    from picolm_b200.config.spec import PartSpec
    from picolm_b200.parts.base import build_part
    base = {"hidden_size": 40, "heads": 2, "dim": 8, "vdim": 8, "decay": [0.5, 0.5], "eps": 1e-6}
    build_part("mixer", PartSpec("retention", base), None)
    rope = {"head_dim": 8, "rotary_dim": 8, "theta": 10.0, "scaling": None, "max_positions": 64}
    for bad in (dict(base, decay=[0.5]), dict(base, position=PartSpec("rope", dict(rope, pairing="adjacent")))):
        with pytest.raises(ValueError):
            build_part("mixer", PartSpec("retention", bad), None)
    moe = {"hidden_size": 40, "experts": 3, "top": 1, "expert_size": 8, "route_scale": 1.0, "router_name": "router", "expert_prefix": "e",
           "up_name": "up", "down_name": "down", "activation": "relu2"}
    build_part("feed_forward", PartSpec("routed_mlp", moe), None)
    for bad in (dict(moe, activation="tanh"), dict(moe, shared={"size": 8, "prefix": "shared", "gate": None})):
        with pytest.raises(ValueError):
            build_part("feed_forward", PartSpec("routed_mlp", bad), None)
    with pytest.raises(ValueError):
        build_part("embedding", PartSpec("token_embedding", {"vocab_size": 5, "hidden_size": 4, "name": "e", "scale": 2.0,
                                                             "norm": {"name": "n", "eps": 1e-6}}), None)


def test_plain_functions_on_small_cases():
    """The plain implementation's own pieces on values worked out by hand."""
    assert P.window_mask(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert P.window_mask(3, None).int().tolist() == [[1, 0, 0], [1, 1, 0], [1, 1, 1]]
    o = P.decayed_scan(torch.ones(3, 1, 1), torch.tensor([1.0, 2.0, 3.0]).view(3, 1, 1), torch.ones(3, 1, 1), [0.5])
    assert o.flatten().tolist() == [1.0, 2.5, 4.25]
    ids, w = P.choose(torch.tensor([[0.0, 3.0, 3.0, -1.0]]), 2, 1.5)
    assert ids.tolist() == [[1, 2]] and torch.allclose(w, torch.tensor([[0.75, 0.75]]))
    assert torch.allclose(P.squash(torch.tensor([0.0, 1e9, -1e9, 0.01]), 2.0), torch.tensor([0.0, 2.0, -2.0, 0.01]), atol=1e-6)
    x = torch.tensor([3.0, 5.0, 4.0, 7.0]).view(1, 1, 4)
    quarter = P.rotate(x, [1], 2, 123.0)                     # one pair (components 0 and 1) by one radian
    c, s = torch.cos(torch.tensor(1.0)), torch.sin(torch.tensor(1.0))
    assert torch.allclose(quarter.flatten(), torch.stack([3 * c - 5 * s, 5 * c + 3 * s, torch.tensor(4.0), torch.tensor(7.0)]), atol=1e-6)
    # one decay of a half, unit write strength: S = 1, then 0.5 + (4 - 0.5) = 4
    o = P.delta_rule(torch.ones(2, 1), torch.ones(2, 1), torch.tensor([[1.0], [4.0]]), torch.tensor([0.3, 0.5]), torch.ones(2))
    assert o.flatten().tolist() == [1.0, 4.0]
    assert torch.allclose(P.short_conv(torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[10.0, 1.0]])).flatten(), torch.tensor([1.0, 12.0, 24.0]))


def test_builders_round_trip():
    from picolm_b200.config import config_from_dict
    for layers in ([_ret(mlp=_moe(3, 1, 8, 0.25))], [_att(size=None, mlp=None)], [_del(conv=1)]):
        cfg = _config(layers)
        assert config_from_dict(cfg).to_dict() == cfg
