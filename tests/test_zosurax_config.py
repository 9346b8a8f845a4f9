"""The Zosurax configuration, model description and cache bookkeeping, without a GPU."""
import copy

import pytest
import torch

from tensorline_b200.cache import PagedKV, SlotState
from tensorline_b200.config import ConfigError
from tensorline_b200.config.zosurax import ZosuraxConfig
from tensorline_b200.models import build_model, expected_tensors
from tensorline_b200.models.registry import architecture, registered_architectures
from tensorline_b200.models.zosurax import describe_zosurax
from tensorline_b200.ops_attention_mix import plan_ranges, row_tiles
from tensorline_b200.parts import Runtime
from tests.plain import zosurax_plain
from tests.tiny_zosurax import CONFIGS


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_round_trip_and_registry(name):
    cfg = ZosuraxConfig.from_dict(CONFIGS[name])
    assert cfg.to_json_dict() == CONFIGS[name]
    assert "Zosurax" in registered_architectures() and architecture("Zosurax").config_class is ZosuraxConfig
    assert cfg.vocab_size == CONFIGS[name]["vocab"] and cfg.hidden_size == CONFIGS[name]["width"]
    spec = describe_zosurax(cfg)
    assert [(e.layer, e.add_row) for e in spec.run] == zosurax_plain.order(CONFIGS[name])
    assert [e.add_start for e in spec.run] == [bool(r) for _, r in zosurax_plain.order(CONFIGS[name])]      # every pass but the first
    assert spec.tie_word_embeddings and cfg.num_parameters() > 0


def test_tensor_names_and_shapes():
    names = expected_tensors(ZosuraxConfig.from_dict(CONFIGS["Z1"]))
    want = {"embed": (131, 48), "loop.step": (2, 48), "final.norm": (48,), "l0.norm1": (48,), "l0.ls1": (48,), "l0.shift": (48,),
            "l0.mix.q": (24, 48), "l0.mix.f": (24, 48), "l0.mix.f.b": (24,), "l0.mix.lower": (24,), "l0.mix.v": (48, 48),
            "l0.mix.norm": (16,), "l0.mix.o": (48, 48),
            "l1.mix.q": (96, 48), "l1.mix.k": (32, 48), "l1.mix.v": (48, 48), "l1.mix.q.norm": (16,), "l1.mix.k.norm": (16,),
            "l1.mix.o": (48, 144), "l1.norm2": (48,), "l1.ls2": (48,), "l1.mlp.up": (40, 48), "l1.mlp.down": (48, 40),
            "l2.mix.q": (32, 48), "l2.mix.talk": (4, 4), "l2.mix.o": (48, 32), "l3.ls2": (48,)}
    for k, shape in want.items():
        assert tuple(names[k].shape) == shape and not names[k].optional, k
    for k in ("l0.norm2", "l0.ls2", "head"):                   # not needed; stored ones are left alone
        assert names[k].optional, k
    for absent in ("l0.mix.k", "l0.mix.g", "l2.mix.q.norm", "l1.mix.talk", "l1.mlp.gate", "l1.mix.q.b"):
        assert absent not in names, absent
    assert "loop.step" not in expected_tensors(ZosuraxConfig.from_dict(CONFIGS["Z3"]))


def test_what_the_cache_manager_is_asked_for():
    rt = Runtime(torch.device("cpu"), torch.float32, 8)
    needs = build_model(ZosuraxConfig.from_dict(CONFIGS["Z1"]), rt).cache_needs()
    entries = [i for i, _ in zosurax_plain.order(CONFIGS["Z1"])]
    assert entries == [0, 1, 2, 1, 2, 3]
    for i in range(len(entries)):                              # every pass has caches and states of its own
        assert needs[(i, "shift")] == SlotState((48,), "float32")
    assert needs[(1, "mixer")] == needs[(3, "mixer")] == PagedKV(2, 24) and needs[(2, "mixer")] == PagedKV(2, 8)
    assert isinstance(needs[(0, "mixer")], SlotState) and needs[(0, "mixer")].dtype == "float32"
    rt16 = Runtime(torch.device("cpu"), torch.bfloat16, 8)     # bfloat16 pages: multiples of 16, of 64 where the heads are mixed
    n16 = build_model(ZosuraxConfig.from_dict(CONFIGS["Z1"]), rt16).cache_needs()
    assert n16[(1, "mixer")] == PagedKV(2, 32) and n16[(2, "mixer")] == PagedKV(2, 64)


def test_row_tiles_of_prompt_portions():
    """Every row tile appears once, with the key tiles up to its last row's position, longest first, in launches of a bounded
    number of (row tile, key tile) pairs."""
    q_start, start = [0, 300, 301, 429], [0, 900, 70]
    launches = row_tiles(q_start, start, [0, 2], 7)
    seen = {}
    for tiles, parts, unit_tile in launches:
        assert parts.tolist() == [[i, p] for i, t in enumerate(tiles) for p in range(-(-int(t[3]) // 8))]
        units = 0
        for i, (b, t, first, kt) in enumerate(tiles.tolist()):
            assert first == units and unit_tile[first:first + kt].tolist() == [i] * kt
            units += kt
            last = start[b] + min(q_start[b + 1] - q_start[b], 128 * (t + 1)) - 1
            assert kt == last // 64 + 1 and (b, t) not in seen
            seen[(b, t)] = kt
        assert units == len(unit_tile) and (units <= 7 or len(tiles) == 1)
    assert sorted(seen) == [(0, 0), (0, 1), (0, 2), (2, 0)]
    flat = [int(x[3]) for t, _, _ in launches for x in t]
    assert flat == sorted(flat, reverse=True)


@pytest.mark.parametrize("n,nkv,group,d,span", [(1, 4, 4, 128, 2304), (8, 4, 4, 128, 2304), (64, 16, 1, 64, 9000), (1, 1, 1, 64, 1), (2, 2, 3, 256, 131072)])
def test_ranges_of_a_decode_step_cover_the_keys(n, nkv, group, d, span):
    rng, splits = plan_ranges(n, nkv, group, d, span, sms=148)
    assert rng % 64 == 0 and 64 <= rng <= 256 and rng * splits >= span > rng * (splits - 1)


def test_blocks_of_a_request_in_the_one_launch_decode():
    from tensorline_b200.ops_attention_mix import plan_cluster
    assert [plan_cluster(n, 16, 4, 128, 2304, sms=148) for n in (1, 6, 7, 12, 13, 37, 38, 74)] == [16, 16, 8, 8, 4, 4, 2, 2]
    assert plan_cluster(8, 16, 16, 64, 4096, sms=148) == 0     # every head its own keys, four thousand of them: every SM is wanted
    assert plan_cluster(1, 64, 8, 128, 65536, sms=148) == 0    # the weights would not fit


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "delta", "type"), (("layers", 1, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 1, "mixer", "rot", "dims"), 5, "dims"), (("layers", 1, "mixer", "rot", "dims"), 18, "dims"),
    (("layers", 1, "mlp", "kind"), "moe", "kind"), (("loop", "stop"), 9, "loop"), (("loop", "times"), 0, "times"),
    (("layers", 0, "mixer", "dim"), 0, "dim"), (("norm", "eps"), 0.0, "eps"), (("layers",), [], "layers"),
])
def test_errors_name_their_key(path, value, word):
    raw = copy.deepcopy(CONFIGS["Z1"])
    node = raw
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        ZosuraxConfig.from_dict(raw)


def test_a_missing_key_is_an_error():
    for path in (("vocab",), ("norm",), ("layers", 0, "mixer", "vdim"), ("layers", 1, "mixer", "scale"), ("layers", 1, "mlp", "ff"), ("loop", "start")):
        raw = copy.deepcopy(CONFIGS["Z1"])
        node = raw
        for k in path[:-1]:
            node = node[k]
        del node[path[-1]]
        with pytest.raises(ConfigError):
            ZosuraxConfig.from_dict(raw)


def test_a_loop_over_no_layers_runs_every_layer_once():
    raw = copy.deepcopy(CONFIGS["Z1"])
    raw["loop"] = {"start": 2, "stop": 2, "times": 3}
    cfg = ZosuraxConfig.from_dict(raw)
    assert cfg.run_order() == [(i, None) for i in range(4)] == zosurax_plain.order(raw)
    assert tuple(expected_tensors(cfg)["loop.step"].shape) == (3, 48)


def test_chunks_of_a_step():
    from tensorline_b200.ops import channel_chunks
    rows, carried = channel_chunks([0, 1, 301, 429, 558], 128)
    assert rows.tolist() == [[0, 0, 1, 0], [1, 0, 3, 1], [1, 1, 3, 1], [1, 2, 3, 1], [2, 0, 1, 4], [3, 0, 2, 5], [3, 1, 2, 5]]
    assert carried.tolist() == [1, 5]
