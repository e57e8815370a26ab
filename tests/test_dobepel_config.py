"""The Dobepel design's configuration, layout and cache plan, on the host."""
import json
import math

import pytest
import torch

from plain import dobepel_plain as P
from test_gpu_dobepel import _config, _dense, _layer, _left, _moe, _right


def _layers():
    return [_layer(), _layer(_left(size=None), mlp="moe"), _layer(_left(heads=6, kv_heads=3, size=9, keep=0), _right(heads=1, decay=[1.0]), mlp=None)]


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
    left, right = ("layers", 0, "mixer", "left"), ("layers", 0, "mixer", "right")
    for path, value, word in ((("layers", 0, "type"), "lstm", "lstm"), (left + ("kv_heads",), 3, "kv_heads"), (left + ("scale",), 0, "scale"),
                              (left + ("mask", "size"), 0, "size"), (left + ("mask", "keep_first"), -1, "keep_first"),
                              (right + ("decay",), [0.5], "decay"), (right + ("decay",), 0.5, "decay"), (right + ("decay",), [0.5, 1.5, 0.1], "decay"),
                              (right + ("vdim",), "x", "vdim"), (("layers", 0, "mlp", "kind"), "odd", "odd"),
                              (("layers", 1, "mlp", "router", "top"), 9, "top"), (("layers", 1, "mlp", "shared", "ff"), 0, "shared"),
                              (("embedding", "bigram", "buckets"), 0, "buckets"), (("embedding", "bigram", "mul_cur"), "x", "mul_cur"),
                              (("residual_mult",), "x", "residual_mult"), (("width",), 0, "width"), (("layers",), [], "layers")):
        with pytest.raises(ConfigError, match=word):
            config_from_dict(_edit(good, path, value))
    for path in (("norm", "eps"), ("vocab",), ("embedding", "bigram"), left + ("dim",), left + ("mask", "size"), right + ("decay",),
                 ("layers", 0, "mlp", "ff"), ("layers", 1, "mlp", "expert"), ("layers", 1, "mlp", "router", "experts")):
        with pytest.raises(ConfigError, match=str(path[-1])):
            config_from_dict(_edit(good, path, delete=True))
    assert config_from_dict(_edit(good, ("residual_mult",), delete=True)).residual_mult == 1.0
    assert config_from_dict(_edit(good, left + ("mask", "keep_first"), delete=True)).layers[0].mixer["left"]["mask"]["keep_first"] == 0


def test_layout_and_cache_plan():
    """Every layer keeps keys and values (its own group by its window, what it keeps of the first tokens and its head
    sizes) and the recurrence's state; the embedding keeps the token before, behind the layers' caches; a layer without
    feed-forward has neither norms nor tensors of one."""
    from picolm_b200.config import config_from_dict, spec_of
    from picolm_b200.engine.model import Model
    spec = spec_of(config_from_dict(_config(_layers(), mult=0.25)))
    assert [layer.arrangement for layer in spec.layers] == ["sandwich_norm"] * 3
    assert spec.layers[0].part("mixer_post_norm").params["scale"] == 0.25 and "scale" not in spec.layers[0].part("mixer_norm").params
    slopes = spec.layers[2].part("mixer").params["left"].params["slopes"]
    assert slopes == [2.0 ** (-8.0 * (h + 1) / 6) for h in range(6)]
    model = Model(spec, None)
    names = model.expected_tensors()
    assert {"embed", "bigram", "head", "final.norm", "l0.norm1b", "l0.norm2b", "l0.mlp.up", "l1.mlp.router.b", "l1.mlp.e4.down", "l1.mlp.shared.up",
            "l2.mix.left.out", "l2.mix.right.norm", "l2.mix.right.g"} <= set(names)
    assert names["bigram"].shape == (54, 40) and names["l0.mix.left.o"].shape == (40, 96) and names["l0.mix.right.o"].shape == (40, 60)
    assert not any(n.startswith(("l2.mlp", "l2.norm2")) for n in names) and "l0.mlp.gate" not in names
    specs = model.cache_specs()
    assert [(s.kind, s.window, s.keep_first) for s in specs if s.kind == "kv"] == [("kv", 21, 5), ("kv", None, 0), ("kv", 9, 0)]
    assert [s.shape for s in specs if s.kind == "state"] == [(3 * 12 * 20,), (3 * 12 * 20,), (12 * 20,), (1,)]
    assert specs[-1].dtype == "int32" and model._embedding_caches == [(6, True)]


def test_kept_pages_stay_when_the_window_moves_on():
    from picolm_b200.cache import CacheSpec, SequenceCache
    spec = CacheSpec.kv(1, 16, window=100, keep_first=65)
    other = CacheSpec.kv(1, 16, window=100)
    assert spec.group_key() != other.group_key()
    with pytest.raises(ValueError):
        CacheSpec.kv(1, 16, keep_first=3)
    cache = SequenceCache([spec, other], max_tokens=64 * 20, max_seqs=2, kv_dtype=torch.float32, device="cpu", allocate_storage=False)
    s = cache.allocate()
    for _ in range(10):
        cache.reserve([(s, 64)])
        cache.advance(s, 64)
        cache.check()
    kept, plain = cache.kv_groups[0].pages[s], cache.kv_groups[1].pages[s]
    # 640 tokens: the next query sees from 541 on, which lies on page 8
    assert [bool(p) for p in kept] == [True, True] + [False] * 6 + [True, True]
    assert [bool(p) for p in plain] == [False] * 8 + [True, True]
    cache.release(s)
    cache.check()


def test_plain_functions_on_small_cases():
    """The plain implementation's own pieces on values worked out by hand."""
    assert P.pair_rows([4, 0, 6], 10, 3, 2) == [10, (12 + 0) % 10, (0 + 12) % 10]
    assert P.head_slopes(4) == [0.25, 0.0625, 0.015625, 0.00390625]
    ok = P.window_mask(6, 2, 1)
    assert ok.int().tolist() == [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0], [1, 0, 0, 1, 1, 0], [1, 0, 0, 0, 1, 1]]
    assert all(bool(ok[i, j]) == P.visible(i, j, 2, 1) for i in range(6) for j in range(6))
    ids, w = P.choose(torch.tensor([[1.0, 3.0, 3.0, 0.0]]), 2)
    assert ids.tolist() == [[1, 2]] and torch.allclose(w, torch.tensor([[0.5, 0.5]]))
    o, S = P.decayed_scan(torch.ones(3, 1, 1), torch.tensor([1.0, 2.0, 3.0]).view(3, 1, 1), torch.ones(3, 1, 1), [0.5])
    assert o.flatten().tolist() == [1.0, 2.5, 4.25] and S.item() == 4.25
    assert abs(P.gelu_erf(torch.tensor(1.0)).item() - 0.5 * (1 + math.erf(1 / math.sqrt(2)))) < 1e-6


def test_decay_table_is_exact_to_float32():
    from picolm_b200.ops import decay_powers
    d = [0.999, 0.3, 1.0, 0.0]
    table = decay_powers(d)
    assert table.shape == (4, 65) and table.dtype == torch.float32
    exact = torch.tensor(d, dtype=torch.float32).double()[:, None] ** torch.arange(65)
    assert ((table.double() - exact).abs() <= 6e-8 * exact).all() and table[3, 0] == 1.0


def test_dense_and_routed_builders_round_trip():
    from picolm_b200.config import config_from_dict
    for mlp in (_dense(48), _moe(experts=3, top=1, shared=None), None):
        cfg = _config([_layer(mlp=mlp)])
        assert config_from_dict(cfg).to_dict() == cfg
