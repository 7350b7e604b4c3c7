"""Lidizen's configuration, tensor names and cache needs, and its plain implementation's mechanisms
against hand-made cases. No GPU."""

import json
import math

import pytest
import torch

import plain_lidizen as plain
from atomserve_b200.cache.manager import CacheManager
from atomserve_b200.config.model_config import ModelConfigError
from atomserve_b200.config.registry import config_from_dict
from atomserve_b200.parts.base import KVCacheSpec
from atomserve_b200.parts.model import build_model
from atomserve_b200.weights.loader import WeightsError, load_model
from atomserve_b200.weights.random_init import write_model_folder
from gefilix_helpers import write_folder
from tiny_lidizen import LIDIZEN

F64 = torch.float64


@pytest.mark.parametrize("name", list(LIDIZEN))
def test_configuration_round_trips_and_names_the_plain_tensors(name):
    cfg, _ = LIDIZEN[name]
    arch, config = config_from_dict(json.loads(json.dumps(cfg)))
    assert arch.name == "Lidizen" and config.to_dict() == cfg
    model = build_model(arch.build_spec(config))
    assert {s.name: tuple(s.shape) for s in model.tensor_specs()} == plain.tensor_shapes(cfg)


def test_what_each_layer_keeps_and_mixes():
    arch, config = config_from_dict(LIDIZEN["a"][0])
    spec = arch.build_spec(config)
    assert config.first_value_layer() == 1
    assert [layer.mixer.params["value_mix"] for layer in spec.layers] == [None, "first", None, "mixed"]
    needs = build_model(spec).cache_requirements()
    assert len(needs) == 5 and needs[4][0] is None and needs[4][1][0].dtype == torch.int32  # the embedding's last token
    assert [(n[0].window, n[0].keep_first, n[0].tensors[0].width) for n in needs[:4]] == [(10, 3, 24), (33, 18, 40), (None, 0, 16), (7, 40, 40)]


def test_unread_tensors_of_a_checkpoint(tmp_path):
    """A factor for values that nothing mixes and the norm of a missing feed-forward may lie in the
    file; anything else that the model does not know may not."""
    cfg, _ = LIDIZEN["d"]
    w = plain.random_checkpoint(cfg, 1)
    extra = {"l0.mix.vmix": torch.tensor(0.5), "l0.norm2": torch.ones(100), "l0.hc2.in": torch.ones(5)}
    load_model(write_folder(cfg, {**w, **extra}, tmp_path / "a"), "float32", "cpu")
    with pytest.raises(WeightsError, match="l1.mix.sink"):
        load_model(write_folder(cfg, {**w, "l1.mix.sink": torch.ones(10)}, tmp_path / "b"), "float32", "cpu")
    del w["l1.mix.vmix"]
    with pytest.raises(WeightsError, match="l1.mix.vmix"):
        load_model(write_folder(cfg, w, tmp_path / "c"), "float32", "cpu")


def test_random_weights_make_a_folder_that_loads(tmp_path):
    _, config = config_from_dict(LIDIZEN["b"][0])
    folder = write_model_folder(config, 5, tmp_path / "m", "float32")
    _, again, model = load_model(folder, "float32", "cpu")
    assert again == config
    mix = model.blocks[1].feed_forward_norm.w_mix
    assert mix.shape == (1, 1) and 0.3 < float(mix) < 1.7


@pytest.mark.parametrize("change,words", [
    (lambda c: c["layers"][0].__setitem__("type", "attention_2"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 4), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), "even"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "positive"),
    (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("keep_first", -1), "negative"),
    (lambda c: c["layers"][3]["mixer"].__setitem__("vdim", 39), "values"),
    (lambda c: c["layers"][1]["mlp"]["router"].__setitem__("top", 6), "cannot choose"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "glu"), "dense"),
    (lambda c: c["embedding"]["bigram"].__setitem__("buckets", 0), "buckets"),
    (lambda c: c.__setitem__("streams", 0), "streams"),
    (lambda c: c.pop("streams"), "streams"),
])  # fmt: skip
def test_rejections(change, words):
    cfg = json.loads(json.dumps(LIDIZEN["a"][0]))
    change(cfg)
    with pytest.raises(ModelConfigError, match=words):
        config_from_dict(cfg)


def test_kept_pages_stay_while_a_window_passes():
    """Pages of 4, a window of 6, the first 5 positions kept: two pages stay for good, those the window
    has passed go back and are handed out again."""
    cache = CacheManager([(KVCacheSpec(1, 8, 6, keep_first=5), [])], 4, 7, 2)
    rc = cache.new_request()
    assert cache.admit(rc)
    for start, n in [(0, 9), (9, 3)] + [(p, 1) for p in range(12, 60)]:
        assert cache.reserve(rc, start, n)
        table = rc.block_tables[0]
        first = max(0, start - 5) // 4
        assert all(b >= 0 for b in table[:2]) and all(b >= 0 for b in table[first:])
        assert all(b < 0 for b in table[2:first])
    assert sum(b >= 0 for b in rc.block_tables[0]) <= 5
    cache.free(rc)
    assert cache.groups[0].allocator.num_free == 7


def test_visibility_by_hand():
    ok = plain.visible(8, dict(size=2, keep_first=2))
    assert ok[7].tolist() == [True, True, False, False, False, False, True, True]
    assert ok[1].tolist() == [True, True] + [False] * 6
    assert plain.visible(5, dict(size=1)).sum() == 5 and plain.visible(5, None).sum() == 15


def test_mixing_of_heads_is_linear_in_the_queries():
    """The identity the engine rests on: mixed scores are scores of mixed queries, part by part."""
    g = torch.Generator().manual_seed(0)
    H, G, d, n = 6, 3, 5, 4
    q, k, talk = torch.randn(n, H, d, generator=g).double(), torch.randn(n, G, d, generator=g).double(), torch.randn(H, H, generator=g).double()
    scores = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(2, dim=1))
    parts = torch.stack([torch.einsum("hg,igd->ihd", talk[:, 2 * c : 2 * c + 2], q[:, 2 * c : 2 * c + 2]) for c in range(G)], dim=2)
    assert torch.allclose(plain.mix_heads(scores, talk), torch.einsum("ihcd,jcd->hij", parts, k))


def test_streams_by_hand():
    X = torch.tensor([[[1.0], [10.0]]], dtype=F64)
    assert plain.gather_streams(X, torch.tensor([2.0, 0.5])).item() == 7.0
    new = plain.advance_streams(X, torch.tensor([[100.0]], dtype=F64), torch.tensor([1.0, 2.0]), torch.tensor([[1.0, 3.0], [5.0, 7.0]]))
    assert new.flatten().tolist() == [1 + 50 + 100, 3 + 70 + 200]  # mix is indexed [from, to]


def test_rotation_and_routing_by_hand():
    x = torch.tensor([[[1.0, 0.0, 0.0, 1.0, 5.0]]], dtype=F64)
    out = plain.rotate_pairs(x, torch.tensor([3]), 100.0, 4)[0, 0]
    want = [math.cos(3.0), math.sin(3.0), -math.sin(0.3), math.cos(0.3), 5.0]
    assert torch.allclose(out, torch.tensor(want, dtype=F64))
    w = {"router": torch.tensor([[1.0], [0.0], [2.0]]), "router.b": torch.tensor([0.0, 3.0, 0.0])}
    chosen, weights = plain.route(torch.tensor([[1.0]], dtype=F64), w, 2)
    assert chosen.tolist() == [[1, 2]] and torch.allclose(weights, torch.softmax(torch.tensor([[3.0, 2.0]], dtype=F64), -1))
