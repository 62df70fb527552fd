"""Biropel's configuration reader and its model as data, without a GPU: every size and constant comes from the document, a
missing or malformed key is refused by name, the document is written back as it was read, a layer that reads another
layer's keys and values becomes a schedule entry that reads the lender's cache, and the parts ask for the design's tensor names and
for the right kinds of cache.  The frequencies of the stretched rotation and the plain implementation's pieces are held to hand-made cases here too."""
from __future__ import annotations

import copy
import math

import pytest
import torch

from hyperion_b200.config import BiropelConfig, ConfigError
from hyperion_b200.models import DecoderModel, architecture_of, get_architecture
from hyperion_b200.parts import PagedTokens, PartSpec, RequestState
from hyperion_b200.parts.base import POSITIONS, BuildContext, make
from hyperion_b200.parts.rope import slowed_frequencies
from plain import biropel_plain as plain

SCALING = {"factor": 8.0, "original": 256.0, "fast": 16.0, "slow": 2.0}
DOCUMENT = {
    "architecture": "Biropel", "vocab": 77, "width": 40, "streams": 5, "norm": {"eps": 1e-5},
    "layers": [
        {"type": "parallel_2", "mlp": {"kind": "dense", "ff": 56},
         "mixer": {"left": {"heads": 6, "kv_heads": 2, "dim": 12, "vdim": 20, "scale": 0.3, "softcap": 9.0, "q_temp": {"coef": 0.25, "every": 10}},
                   "right": {"heads": 3, "dim": 10, "vdim": 14, "gate_cap": 6.0}}},
        {"type": "attention", "mlp": None,
         "mixer": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.25, "mask": {"size": 30}, "rot": {"dims": 6, "base": 500.0}}},
        {"type": "parallel", "mlp": {"kind": "dense", "ff": 24},
         "mixer": {"left": {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 8, "scale": 0.4, "mask": {"size": 11}, "softcap": 4.0, "rot": {"dims": 8, "base": 1e4, "scaling": SCALING}},
                   "right": {"heads": 4, "vdim": 6, "state": 9, "groups": 2, "norm_groups": 3, "conv": 3}}},
        {"type": "attention", "mlp": {"kind": "dense", "ff": 8},
         "mixer": {"heads": 2, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.2, "mask": {"size": 70}, "rot": {"dims": 6, "base": 500.0}, "kv_from": 1}},
        {"type": "attention", "mlp": {"kind": "dense", "ff": 8}, "mixer": {"heads": 2, "kv_heads": 1, "dim": 10, "vdim": 7, "scale": 0.2}},
    ],
}


def test_the_document_is_read_and_written_back():
    entry = architecture_of(DOCUMENT)
    assert entry.name == "Biropel"
    config = entry.read_config(DOCUMENT)
    assert entry.write_config(config) == DOCUMENT
    assert (config.vocab, config.width, config.streams, config.eps) == (77, 40, 5, 1e-5)
    left = config.layers[0].mixer.left
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.window, left.softcap, left.rot) == (6, 2, 12, 20, 0.3, 0, 9.0, None)
    assert (left.q_temp.coef, left.q_temp.every) == (0.25, 10)
    right = config.layers[0].mixer.right
    assert (right.heads, right.dim, right.vdim, right.gate_cap) == (3, 10, 14, 6.0)
    rot = config.layers[2].mixer.left.rot
    assert (rot.dims, rot.base, rot.scaling.factor, rot.scaling.original, rot.scaling.fast, rot.scaling.slow) == (8, 1e4, 8.0, 256.0, 16.0, 2.0)
    assert config.layers[2].mixer.right.norm_groups == 3 and config.layers[1].ff is None and config.layers[3].mixer.kv_from == 1
    assert [config.cache_window(i) for i in (1, 4)] == [70, 0]  # the lender keeps what its widest reader sees
    open_reader = copy.deepcopy(DOCUMENT)
    del open_reader["layers"][3]["mixer"]["mask"]
    assert BiropelConfig.from_dict(open_reader).cache_window(1) == 0


@pytest.mark.parametrize("path, value, key", [
    (("vocab",), 0, "vocab"), (("width",), None, "width"), (("streams",), None, "streams"), (("streams",), 1.5, "streams"), (("norm", "eps"), -1.0, "norm.eps"),
    (("layers", 0, "type"), "lstm", "layers[0].type"), (("layers", 0, "mixer", "left"), None, "layers[0].mixer.left"),
    (("layers", 0, "mixer", "left", "kv_heads"), 4, "layers[0].mixer.left.kv_heads"), (("layers", 0, "mixer", "left", "softcap"), 0, "layers[0].mixer.left.softcap"),
    (("layers", 0, "mixer", "left", "q_temp", "every"), 0, "layers[0].mixer.left.q_temp.every"), (("layers", 0, "mixer", "left", "q_temp", "coef"), None, "layers[0].mixer.left.q_temp.coef"),
    (("layers", 0, "mixer", "left", "kv_from"), 0, "layers[0].mixer.left.kv_from"), (("layers", 0, "mixer", "right", "gate_cap"), -3.0, "layers[0].mixer.right.gate_cap"),
    (("layers", 0, "mixer", "right", "dim"), None, "layers[0].mixer.right.dim"), (("layers", 1, "mixer", "mask", "size"), 0, "layers[1].mixer.mask.size"),
    (("layers", 1, "mixer", "rot", "dims"), 18, "layers[1].mixer.rot.dims"), (("layers", 1, "mixer", "rot", "dims"), 5, "layers[1].mixer.rot.dims"),
    (("layers", 1, "mixer", "rot", "base"), None, "layers[1].mixer.rot.base"), (("layers", 1, "mixer", "scale"), None, "layers[1].mixer.scale"),
    (("layers", 2, "mixer", "left", "rot", "scaling", "slow"), None, "layers[2].mixer.left.rot.scaling.slow"),
    (("layers", 2, "mixer", "left", "rot", "base"), 1.0, "layers[2].mixer.left.rot.base"), (("layers", 2, "mixer", "right", "groups"), 3, "layers[2].mixer.right.groups"),
    (("layers", 2, "mixer", "right", "norm_groups"), 5, "layers[2].mixer.right.norm_groups"), (("layers", 2, "mixer", "right", "conv"), 0, "layers[2].mixer.right.conv"),
    (("layers", 3, "mixer", "kv_from"), 2, "layers[3].mixer.kv_from"), (("layers", 3, "mixer", "kv_from"), 3, "layers[3].mixer.kv_from"),
    (("layers", 3, "mixer", "kv_from"), "first", "layers[3].mixer.kv_from"), (("layers", 3, "mixer", "vdim"), 12, "layers[3].mixer.kv_from"),
    (("layers", 4, "mixer", "kv_from"), 3, "layers[4].mixer.kv_from"), (("layers", 0, "mlp", "kind"), "moe", "layers[0].mlp.kind"), (("layers", 0, "mlp", "ff"), None, "layers[0].mlp.ff"),
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
        BiropelConfig.from_dict(document)
    assert refused.value.key == key


def test_the_model_as_data_asks_for_the_designs_tensors_and_caches():
    entry = get_architecture("Biropel")
    model = DecoderModel(entry.build_spec(entry.read_config(DOCUMENT)), torch.float32, torch.device("meta"))
    wanted = {name: tuple(spec.shape) for name, spec in model.expected_tensors().items()}
    assert wanted["embed"] == wanted["head"] == (77, 40) and wanted["embed.norm"] == wanted["final.norm"] == (40,)
    for name in ("l0.hc1", "l0.hc2", "l1.hc1"):
        assert wanted[name + ".in"] == wanted[name + ".out"] == (5,) and wanted[name + ".mix"] == (5, 5)
    assert "l1.hc2.in" not in wanted and "l1.norm2" not in wanted and {"l1.norm2", "l1.hc2.in", "l1.hc2.out", "l1.hc2.mix"} == set(model.spec.tolerated)
    assert {name for name in wanted if name.startswith("l0.mix.left.")} == {"l0.mix.left." + n for n in ("q", "k", "v", "o", "out")}
    assert wanted["l0.mix.left.q"] == (72, 40) and wanted["l0.mix.left.v"] == (40, 40) and wanted["l0.mix.left.o"] == (40, 120) and wanted["l0.mix.left.out"] == (40,)
    assert wanted["l0.mix.right.q"] == (30, 40) and wanted["l0.mix.right.v"] == wanted["l0.mix.right.g"] == (42, 40) and wanted["l0.mix.right.norm"] == (42,)
    assert wanted["l0.mix.right.i"] == wanted["l0.mix.right.f"] == (3, 40) and wanted["l0.mix.right.i.b"] == wanted["l0.mix.right.f.b"] == (3,)
    assert wanted["l0.mlp.up"] == (56, 40) and wanted["l0.mlp.down"] == (40, 56)
    assert wanted["l1.mix.q.b"] == (64,) and wanted["l1.mix.v.b"] == (32,) and wanted["l1.mix.g"] == (64, 40) and "l1.mix.o.b" not in wanted
    assert wanted["l2.mix.right.in"] == (2 * 24 + 2 * 2 * 9 + 4, 40) and wanted["l2.mix.right.conv"] == (60, 3) and wanted["l2.mix.right.norm"] == (24,)
    assert {name for name in wanted if name.startswith("l3.mix.")} == {"l3.mix." + n for n in ("q", "q.b", "g", "o")}  # no keys and values of its own
    assert [(run.layer, run.reads_cache_of) for run in model.spec.schedule] == [(0, None), (1, None), (2, None), (3, 1), (4, None)]
    users = dict(model.cache_users())
    assert set(users) == {(0, 0), (0, 1), 1, (2, 0), (2, 1), 4}
    assert users[(0, 0)] == PagedTokens((2,), (32,), 0)  # keys of 12 and values of 20 side by side
    assert users[(0, 1)] == RequestState((3 * 15 * 12 + 4,))  # 14 values and the sum of keys of each head, then the running maxima
    assert users[1] == PagedTokens((2, 2), (16,), 70)  # for the widest reader
    assert users[(2, 0)] == PagedTokens((2, 1), (8,), 11)
    assert users[(2, 1)] == RequestState((4 * 6 * 12 + 2 * 60,))
    with pytest.raises(ValueError):
        many = {**DOCUMENT, "streams": 17}
        DecoderModel(entry.build_spec(entry.read_config(many)), torch.float32, torch.device("meta"))


def test_frequencies_of_the_stretched_rotation():
    """Against the plain formula, and at the ramp's ends: fast pairs keep their frequency, slow ones are divided by the factor."""
    for dims, base, factor, original, fast, slow in ((64, 1e4, 4.0, 512.0, 32.0, 1.0), (8, 500.0, 8.0, 256.0, 16.0, 2.0), (2, 100.0, 2.0, 64.0, 4.0, 1.0), (96, 1e6, 1.0, 100.0, 8.0, 1.0),
                                                     (20, 10.0, 16.0, 8.0, 2.0, 1.0)):
        want, amplitude = plain.frequencies({"dims": dims, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}})
        assert torch.allclose(slowed_frequencies(dims, base, factor, original, fast, slow), torch.tensor(want, dtype=torch.float64), rtol=1e-12)
        build = BuildContext(dtype=torch.float32, device=torch.device("cpu"), max_positions=10, shared={})
        part = make(POSITIONS, PartSpec("rope_half_slowed", "", {"dims": dims, "base": base, "factor": factor, "original": original, "fast": fast, "slow": slow}), build)
        assert part.half and part.dims == dims and math.isclose(part.amplitude, amplitude) and torch.allclose(part.inv_freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6)
    slowed = slowed_frequencies(64, 1e4, 4.0, 512.0, 32.0, 1.0)
    kept = torch.tensor([1e4 ** (-2 * i / 64) for i in range(32)], dtype=torch.float64)
    assert torch.allclose(slowed[:3], kept[:3]) and torch.allclose(slowed[-8:], kept[-8:] / 4)
    assert ((slowed <= kept * (1 + 1e-12)) & (slowed >= kept / 4 * (1 - 1e-12))).all()


def test_the_plain_pieces_on_cases_made_by_hand():
    assert plain.sees(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    f64 = dict(dtype=torch.float64)
    # the mixing matrix is indexed [from, to]
    w = {"c.in": torch.tensor([1.0, 10.0], **f64), "c.out": torch.tensor([3.0, 0.0], **f64), "c.mix": torch.tensor([[1.0, 2.0], [0.0, 5.0]], **f64)}
    streams = torch.tensor([[[1.0]], [[2.0]]], **f64)
    assert plain.read_streams(streams, w, "c.").tolist() == [[21.0]]
    assert plain.write_streams(streams, torch.tensor([[7.0]], **f64), w, "c.").tolist() == [[[22.0]], [[12.0]]]
    # a quarter turn of one pair, entry i with entry i + dims / 2, the rest untouched
    x = torch.tensor([[[0.0, 0.0, 9.0]], [[1.0, 2.0, 9.0]]], **f64)
    turned = plain.rotate(x, {"dims": 2, "base": 7.0})
    assert torch.allclose(turned[1, 0], torch.tensor([math.cos(1) - 2 * math.sin(1), 2 * math.cos(1) + math.sin(1), 9.0], **f64))
    # the temperature rises where position + 1 reaches a multiple of its step
    t = plain.temperature(7, {"coef": 2.0, "every": 3}, torch.float64)
    assert torch.allclose(t, torch.tensor([1.0, 1.0] + [1.0 + 2 * math.log(2)] * 3 + [1.0 + 2 * math.log(3)] * 2, **f64))
    # the convolution's last column multiplies the current token
    y = plain.causal_convolution(torch.tensor([[1.0], [2.0], [3.0]], **f64), torch.tensor([[10.0, 1.0]], **f64), torch.tensor([0.5], **f64))
    assert y[:, 0].tolist() == [1.5, 12.5, 23.5]
    # a memory whose gates are always open: the running maximum starts at 0, so a first token behind a log input gate of -1 is not lifted to 1
    w = {n: torch.ones(1, 1, **f64) for n in ("q", "k", "v", "o")}
    w.update({"i": torch.zeros(1, 1, **f64), "f": torch.zeros(1, 1, **f64), "g": torch.zeros(1, 1, **f64), "i.b": torch.tensor([-1.0], **f64), "f.b": torch.tensor([1e9], **f64),
              "norm": torch.ones(1, **f64)})
    i, f = plain.matrix_memory_gates(torch.ones(1, 1, **f64), w, "", 1e6)
    assert math.isclose(float(i), -1.0, rel_tol=1e-6) and float(f) == 0.0
    out = plain.matrix_memory(torch.full((1, 1), 0.5, **f64), w, "", {"heads": 1, "dim": 1, "vdim": 1, "gate_cap": 1e6}, 1.0)
    o = math.exp(-1) * 0.5 * 0.5 * 0.5 / (1.0 + 1e-6)  # exp(-m) = 1 is above |n . q|
    assert math.isclose(float(out), o / math.sqrt(o * o + 1.0) * 0.5, rel_tol=1e-6)
