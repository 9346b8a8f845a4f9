"""The Fimolix configuration, model description and cache bookkeeping, without a GPU."""
import copy

import pytest
import torch

from tensorline_b200.cache import CacheManager, PagedKV, SlotState
from tensorline_b200.config import ConfigError
from tensorline_b200.config.fimolix import FimolixConfig
from tensorline_b200.models import build_model, expected_tensors
from tensorline_b200.models.fimolix import describe_fimolix
from tensorline_b200.models.registry import architecture, registered_architectures
from tensorline_b200.parts import Runtime
from tests.plain.fimolix_plain import PlainFimolix, greedy_generate, logits_of
from tests.tiny_fimolix import CONFIGS, write_tiny_fimolix


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_round_trip_and_registry(name):
    cfg = FimolixConfig.from_dict(CONFIGS[name])
    assert cfg.to_json_dict() == CONFIGS[name]
    assert "Fimolix" in registered_architectures() and architecture("Fimolix").config_class is FimolixConfig
    assert cfg.vocab_size == CONFIGS[name]["vocab"] and cfg.hidden_size == CONFIGS[name]["width"]
    spec = describe_fimolix(cfg)
    assert [e.layer for e in spec.run] == list(range(len(cfg.layers)))
    assert [e.reads_cache_of for e in spec.run] == [l["mixer"].get("kv_from") for l in CONFIGS[name]["layers"]]
    assert spec.tie_word_embeddings and cfg.num_parameters() > 0


def test_tensor_names_and_shapes():
    names = expected_tensors(FimolixConfig.from_dict(CONFIGS["F1"]))
    want = {"embed": (131, 48), "final.norm": (48,), "l0.norm1": (48,), "l0.norm2": (48,), "l0.mix.q": (36, 48), "l0.mix.dkv": (24, 48),
            "l0.mix.dkv.norm": (20,), "l0.mix.uk": (24, 20), "l0.mix.uv": (36, 20), "l0.mix.sink": (3,), "l0.mix.g": (3, 48),
            "l0.mix.o": (48, 36), "l0.mlp.up": (40, 48), "l0.mlp.down": (48, 40),
            "l1.mix.q": (96, 48), "l1.mix.k": (32, 48), "l1.mix.v": (48, 48), "l1.mix.q.conv": (96, 3), "l1.mix.k.conv": (32, 3),
            "l1.mix.v.conv": (48, 3), "l1.mix.q.norm": (8,), "l1.mix.k.norm": (8,), "l1.mix.lq1": (8,), "l1.mix.lk2": (8,), "l1.mix.o": (48, 144),
            "l2.mix.uk": (60, 20), "l2.mix.uv": (40, 20), "l2.mix.sink": (5,), "l2.mix.g": (5, 48)}
    for k, shape in want.items():
        assert tuple(names[k].shape) == shape and not names[k].optional, k
    for k in ("l2.norm2", "l3.norm2", "head"):                 # not needed; stored ones are left alone
        assert names[k].optional, k
    for absent in ("l2.mix.dkv", "l2.mix.dkv.norm", "l2.mlp.up", "l0.mlp.gate", "l0.mix.k", "l1.mix.sink", "l1.mix.g"):
        assert absent not in names, absent
    assert tuple(expected_tensors(FimolixConfig.from_dict(CONFIGS["F2"]))["l0.mix.q.conv"].shape) == (96, 1)      # one tap is a factor


def test_what_the_cache_manager_is_asked_for():
    rt = Runtime(torch.device("cpu"), torch.float32, 8)
    needs = build_model(FimolixConfig.from_dict(CONFIGS["F1"]), rt).cache_needs()
    assert needs[0] == PagedKV(1, 24, 37, shared_values=True)           # its own queries see 9 keys, its reader's 37
    assert 2 not in needs and needs[4] == PagedKV(1, 32, 5, shared_values=True)
    assert needs[(1, "kv")] == PagedKV(2, 24) and needs[(1, "rows")] == SlotState((2, 176), "float32")
    assert needs[(3, "kv")] == PagedKV(1, 24) and needs[(3, "rows")] == SlotState((3, 136), "float32")
    n2 = build_model(FimolixConfig.from_dict(CONFIGS["F2"]), Runtime(torch.device("cpu"), torch.bfloat16, 8)).cache_needs()
    assert n2[1] == PagedKV(1, 48, 50, shared_values=True)              # narrower readers change nothing
    assert (0, "rows") not in n2 and n2[(0, "kv")] == PagedKV(3, 48) and n2[(3, "rows")].dtype == "bfloat16"


def test_a_cache_keeps_what_its_readers_see():
    a = PagedKV(1, 8, 10, shared_values=True)
    assert a.widened(PagedKV(1, 8, 25, shared_values=True)).window == 25 and a.widened(PagedKV(1, 8, 4, shared_values=True)) == a
    assert a.widened(PagedKV(1, 8, None, shared_values=True)).window is None
    c = PagedKV(2, 8, None, chunk=6)
    assert c.widened(PagedKV(2, 8, None, chunk=6)) == c and c.widened(PagedKV(2, 8, None, chunk=7)) == PagedKV(2, 8)
    assert PagedKV(2, 8, 5, keep_first=3).widened(PagedKV(2, 8, 9, keep_first=1)) == PagedKV(2, 8, 9, keep_first=3)
    with pytest.raises(ValueError):
        a.widened(PagedKV(1, 16, 25, shared_values=True))
    # pages of the wider window stay while the request moves on
    cm = CacheManager({0: a.widened(PagedKV(1, 8, 25, shared_values=True))}, page_size=4, num_pages=20, max_num_seqs=1, max_model_len=80,
                      prefix_caching=False)
    assert cm.admit("x") == 0 and cm.grow("x", 0, 40)
    cm.advance("x", 40, None)                                  # position 40 reads 16 .. 40 through the wider window
    assert [p >= 0 for p in cm.pages("x", 0)] == [False] * 4 + [True] * 6
    cm.check()


def test_ranges_of_keys_for_heads_whose_block_fills_an_sm():
    """One key/value head of 256: clusters of more than nine blocks only while at most seven of them run."""
    from tensorline_b200.ops_attention import plan_splits
    assert plan_splits(7, 1, 16, 2111, 256, sms=148) == (192, 11) and plan_splits(8, 1, 16, 2111, 256, sms=148) == (256, 9)
    assert plan_splits(12, 1, 16, 2111, 256, sms=148)[1] <= 9
    assert plan_splits(2, 4, 7, 4096, 128, sms=148)[1] == 16             # narrower heads: two blocks an SM, as they were


@pytest.mark.parametrize("path,value,word", [
    (("layers", 1, "type"), "hgrn2", "type"), (("layers", 1, "mixer", "kv_heads"), 4, "kv_heads"), (("layers", 0, "mixer", "rot", "dims"), 3, "dims"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"), (("layers", 0, "mixer", "mask", "size"), 0, "size"), (("layers", 1, "mixer", "softcap"), 0.0, "softcap"),
    (("layers", 1, "mixer", "conv"), 0, "conv"), (("layers", 2, "mixer", "kv_from"), 2, "kv_from"), (("layers", 2, "mixer", "kv_from"), 1, "kv_from"),
    (("layers", 2, "mixer", "kv_rank"), 21, "kv_rank"), (("layers", 2, "mixer", "rot", "base"), 999.0, "rot"), (("norm", "eps"), -1.0, "eps"),
    (("layers", 4, "mixer", "kv_from"), 2, "kv_from"),
])
def test_errors_name_their_key(path, value, word):
    raw = copy.deepcopy(CONFIGS["F1"])
    node = raw
    for k in path[:-1]:
        node = node[k]
    node[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        FimolixConfig.from_dict(raw)


def test_a_missing_key_is_an_error():
    for path in (("vocab",), ("norm",), ("layers", 1, "mixer", "diff"), ("layers", 1, "mixer", "softcap"), ("layers", 0, "mixer", "mask"),
                 ("layers", 0, "mixer", "rot"), ("layers", 0, "mixer", "kv_rank"), ("layers", 0, "mlp", "ff")):
        raw = copy.deepcopy(CONFIGS["F1"])
        node = raw
        for k in path[:-1]:
            node = node[k]
        del node[path[-1]]
        with pytest.raises(ConfigError):
            FimolixConfig.from_dict(raw)


def test_the_plain_model_is_causal_and_reads_its_weights(tmp_path):
    plain = PlainFimolix(write_tiny_fimolix("F2", tmp_path / "m"))
    toks = [5, 17, 3, 44, 80, 2, 9]
    whole = logits_of(plain, toks)
    assert torch.allclose(logits_of(plain, toks[:4]), whole[:4], atol=1e-12)
    assert greedy_generate(plain, toks, 1) == [int(whole[-1].argmax())]
