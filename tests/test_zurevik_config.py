"""Zurevik's configuration reader and its model as data, without a GPU: every size and constant comes from the document, a
missing or malformed key is refused by name, the document is written back as it was read, a layer that reads another
layer's keys and values becomes a schedule entry that reads the lender's cache, and the parts ask for the design's tensor names and
for the right kinds of cache.  The plain implementation's pieces are held to hand-made cases here too."""
from __future__ import annotations

import copy
import math

import pytest
import torch

from hyperion_b200.config import ConfigError, ZurevikConfig
from hyperion_b200.models import DecoderModel, architecture_of, get_architecture
from hyperion_b200.parts import PagedTokens
from plain import zurevik_plain as plain

DOCUMENT = {
    "architecture": "Zurevik", "vocab": 77, "width": 40, "embedding": {"scale": 3.5}, "norm": {"eps": 1e-5}, "logit_softcap": 20.0,
    "layers": [
        {"type": "attention_2", "mixer": {"heads": 6, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.3, "mask": {"size": 50}},
         "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2}}},
        {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 10, "vdim": 14, "scale": 0.25, "mask": {"size": 30, "keep_first": 3}, "diff": 0.4},
         "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 3, "top": 3}}},
        {"type": "attention_2", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.2, "mask": {"size": 70}, "kv_from": 0}, "mlp": None},
        {"type": "attention", "mixer": {"heads": 3, "kv_heads": 1, "dim": 16, "vdim": 32, "scale": 0.2, "mask": {"size": 9, "keep_first": 0}, "diff": 0.2}, "mlp": None},
        {"type": "attention_2", "mixer": {"heads": 2, "kv_heads": 2, "dim": 32, "vdim": 32, "scale": 0.1, "mask": {"size": 16}},
         "mlp": {"kind": "moe", "expert": {"ff": 16}, "router": {"experts": 2, "top": 1}}},
        {"type": "attention_2", "mixer": {"heads": 6, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.3, "mask": {"size": 20}, "kv_from": 0}, "mlp": None},
    ],
}


def test_the_document_is_read_and_written_back():
    entry = architecture_of(DOCUMENT)
    assert entry.name == "Zurevik"
    config = entry.read_config(DOCUMENT)
    assert entry.write_config(config) == DOCUMENT
    assert (config.vocab, config.width, config.eps, config.embedding_scale, config.logit_softcap) == (77, 40, 1e-5, 3.5, 20.0)
    a = config.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.diff, a.window, a.keep_first) == (4, 2, 10, 14, 0.25, 0.4, 30, 3)
    b = config.layers[2].mixer
    assert (b.heads, b.kv_heads, b.dim, b.vdim, b.scale, b.window, b.kv_from) == (4, 2, 12, 20, 0.2, 70, 0)
    assert config.layers[2].mlp is None and (config.layers[0].mlp.ff, config.layers[0].mlp.experts, config.layers[0].mlp.top) == (24, 5, 2)
    assert [config.cache_window(i) for i in (0, 4)] == [70, 16]  # the lender keeps what its widest reader sees
    bare = copy.deepcopy(DOCUMENT)
    del bare["embedding"], bare["logit_softcap"], bare["layers"][2]["mixer"]["mask"], bare["layers"][1]["mixer"]["mask"]["keep_first"]
    config = ZurevikConfig.from_dict(bare)
    assert config.embedding_scale == 1.0 and config.logit_softcap == 0.0 and config.layers[1].mixer.keep_first == 0
    assert config.layers[2].mixer.window == 0 and config.cache_window(0) == 0  # one reader sees every key


@pytest.mark.parametrize("path, value, key", [
    (("vocab",), 0, "vocab"), (("width",), None, "width"), (("norm", "eps"), -1.0, "norm.eps"), (("embedding", "scale"), "big", "embedding.scale"),
    (("logit_softcap",), -2.0, "logit_softcap"), (("layers", 0, "type"), "lstm", "layers[0].type"), (("layers", 0, "mixer", "kv_heads"), 4, "layers[0].mixer.kv_heads"),
    (("layers", 0, "mixer", "mask", "size"), 0, "layers[0].mixer.mask.size"), (("layers", 0, "mixer", "scale"), None, "layers[0].mixer.scale"),
    (("layers", 1, "mixer", "mask", "keep_first"), -1, "layers[1].mixer.mask.keep_first"), (("layers", 1, "mixer", "diff"), None, "layers[1].mixer.diff"),
    (("layers", 1, "mixer", "dim"), 0, "layers[1].mixer.dim"), (("layers", 2, "mixer", "kv_from"), 1, "layers[2].mixer.kv_from"),
    (("layers", 2, "mixer", "kv_from"), 4, "layers[2].mixer.kv_from"), (("layers", 5, "mixer", "kv_from"), 2, "layers[5].mixer.kv_from"),
    (("layers", 5, "mixer", "kv_from"), 4, "layers[5].mixer.kv_from"), (("layers", 5, "mixer", "kv_from"), "first", "layers[5].mixer.kv_from"),
    (("layers", 5, "mixer", "vdim"), 12, "layers[5].mixer.kv_from"), (("layers", 0, "mlp", "kind"), "dense", "layers[0].mlp.kind"),
    (("layers", 0, "mlp", "router", "top"), 6, "layers[0].mlp.router.top"), (("layers", 0, "mlp", "expert"), None, "layers[0].mlp.expert"),
])
def test_a_bad_value_is_refused_by_name(path, value, key):
    document = copy.deepcopy(DOCUMENT)
    at = document
    for step in path[:-1]:
        at = at[step]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError) as refused:
        ZurevikConfig.from_dict(document)
    assert refused.value.key == key


def test_the_model_as_data_asks_for_the_designs_tensors_and_caches():
    entry = get_architecture("Zurevik")
    model = DecoderModel(entry.build_spec(entry.read_config(DOCUMENT)), torch.float32, torch.device("meta"))
    wanted = {name: tuple(spec.shape) for name, spec in model.expected_tensors().items()}
    assert wanted["embed"] == wanted["head"] == (77, 40) and wanted["final.norm"] == (40,)
    assert wanted["l0.mix.q"] == (72, 40) and wanted["l0.mix.q.b"] == (72,) and wanted["l0.mix.k"] == (24, 40) and wanted["l0.mix.v"] == (40, 40)
    assert wanted["l0.mix.v.b"] == (40,) and wanted["l0.mix.sink"] == (6,) and wanted["l0.mix.g"] == (6, 40) and wanted["l0.mix.o"] == (40, 120)
    assert wanted["l1.mix.q"] == (80, 40) and wanted["l1.mix.k"] == (40, 40) and wanted["l1.mix.v"] == (28, 40) and wanted["l1.mix.g"] == (56, 40)
    assert wanted["l1.mix.q.norm"] == wanted["l1.mix.k.norm"] == wanted["l1.mix.lq1"] == wanted["l1.mix.lk2"] == (10,) and "l1.mix.q.b" not in wanted
    assert {name for name in wanted if name.startswith("l2.mix.")} == {"l2.mix." + n for n in ("q", "q.b", "sink", "g", "o")}  # no keys and values of its own
    assert wanted["l2.mix.q"] == (48, 40) and wanted["l2.mix.o"] == (40, 80)
    assert wanted["l0.mlp.router"] == (5, 40) and wanted["l0.mlp.router.b"] == (5,) and wanted["l0.mlp.e4.up"] == (24, 40) and wanted["l0.mlp.e4.down"] == (40, 24)
    assert "l0.mlp.e5.up" not in wanted and "l2.norm2" not in wanted and wanted["l0.norm2"] == (40,) and "l2.norm2" in model.spec.tolerated
    assert [(run.layer, run.reads_cache_of) for run in model.spec.schedule] == [(0, None), (1, None), (2, 0), (3, None), (4, None), (5, 0)]
    users = dict(model.cache_users())
    assert set(users) == {0, 1, 3, 4}
    assert users[0] == PagedTokens((2,), (32,), 70)  # keys of 12 and values of 20 side by side, for the widest reader
    assert users[1] == PagedTokens((2,), (34,), 30, keep_first=3)  # a head's two keys of 10 and its value of 14
    assert users[3] == PagedTokens((2, 1), (32,), 9)  # two keys as wide as a value: the layout every attention of the package uses
    assert users[4] == PagedTokens((2, 2), (32,), 16)


def test_the_plain_pieces_on_cases_made_by_hand():
    # a window of two beside one kept first token
    assert plain.sees(4, 2, 1).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [1, 1, 1, 0], [1, 0, 1, 1]]
    assert plain.sees(3, None).int().tolist() == [[1, 0, 0], [1, 1, 0], [1, 1, 1]]
    # the sink takes its share of the denominator and nothing else
    scores = torch.tensor([[[0.0, math.log(2.0)]]], dtype=torch.float64)
    p = plain.softmax_with_sink(scores, torch.tensor([math.log(5.0)], dtype=torch.float64))
    assert torch.allclose(p, torch.tensor([[[1 / 8, 2 / 8]]], dtype=torch.float64))
    assert torch.allclose(plain.softmax_with_sink(scores, None), torch.tensor([[[1 / 3, 2 / 3]]], dtype=torch.float64))
    # the router: the bias lifts output 0 above output 1; the weights are a softmax over the two chosen, biases included
    w = {"router": torch.eye(3, dtype=torch.float64), "router.b": torch.tensor([2.0, 0.0, 0.0], dtype=torch.float64)}
    chosen, weight = plain.route(torch.tensor([[0.0, 1.0, 3.0]], dtype=torch.float64), w, "", 2)
    assert chosen.tolist() == [[2, 0]] and torch.allclose(weight, torch.softmax(torch.tensor([[3.0, 2.0]], dtype=torch.float64), dim=-1))
    # the second map's weight
    w = {name: torch.tensor([v], dtype=torch.float64) for name, v in (("lq1", 2.0), ("lk1", 0.5), ("lq2", 1.0), ("lk2", 0.0))}
    assert math.isclose(float(plain.map_weight(w, "", 0.25)), math.e - 1.0 + 0.25)
    assert torch.allclose(plain.soft_cap(torch.tensor([1e9, 0.0]), 7.0), torch.tensor([7.0, 0.0]))
