"""Zurevik on the GPU against the plain implementation (``tests/plain/zurevik_plain.py``): every mechanism alone, whole prompts against
token-by-token decoding, portions down to two tokens, batches of unequal requests against each alone, pages that are freed
and taken again while the first ones stay, keys just inside and just outside a window and the kept first tokens, at page borders and
far away, the sink, long decoding, sizes that differ in every respect between the configurations, layers that read another layer's keys and
values through windows of their own, and greedy generation through ``Engine.generate``.

The configurations and weights are made here.  Weights are drawn so that a fault shows: matrices of N(0, gain^2 / in) make the attention
peaked, sinks are of the size of the scores, and where a test is about one key a marker token, whose key points where the last query points,
makes that key's score stand out.  In the whole models the routers' biases settle which experts are chosen (steps that the small logits beside
them cannot cross) while the weights still follow the logits, so that a bfloat16 run sends every token where exact arithmetic does.  float32
runs are held to 3e-4 of the largest logit, which no wrong key, window or lost page survives; bfloat16 runs to 5e-2 of a row's
root-mean-square logit.
"""
from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from plain import zurevik_plain as plain

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOLERANCE = {"float32": 3e-4, "bfloat16": 5e-2}


# ------------------------------------------------------------------------------------------ configurations
def mask_of(window, keep=None):
    if window is None:
        return {}
    return {"mask": {"size": window} if keep is None else {"size": window, "keep_first": keep}}


def differential(heads, kv_heads, dim, vdim, scale, diff, window=None, keep=0):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff, **mask_of(window, keep)}


def sinks(heads, kv_heads, dim, vdim, scale, window=None, kv_from=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, **mask_of(window)}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return "attention_2", mixer


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(kind_and_mixer, mlp=None):
    return {"type": kind_and_mixer[0], "mixer": kind_and_mixer[1], "mlp": mlp}


def document(width, vocab, layers, eps=1e-5, embed=1.0, cap=30.0):
    doc = {"architecture": "Zurevik", "vocab": vocab, "width": width, "embedding": {"scale": embed}, "norm": {"eps": eps}, "layers": layers}
    if cap is not None:
        doc["logit_softcap"] = cap
    return doc


# Two models that differ in every size, in the order of their layers, in eps, in the embedding's scale and the cap; keys and values of unequal
# size and of shapes that the tensor-core kernels take, one key/value head for six and one per head, windows that are no multiple of a page (40,
# 7, 9, 100) and none, three kept first tokens, more of them than a page holds and none, a layer that reads another's keys through a wider and one that reads
# them through a narrower window, one to four experts per token, layers without a feed-forward.
CONFIGS = {
    "A": document(64, 131, [layer(sinks(4, 2, 24, 16, 0.3, window=20), moe(72, 5, 2)),
                            layer(differential(4, 2, 12, 20, 0.35, 0.3, window=40, keep=3), moe(24, 4, 3)),
                            layer(sinks(2, 2, 24, 16, 0.25, window=45, kv_from=0)),
                            layer(differential(3, 3, 8, 16, 0.4, 0.6, window=9, keep=19), moe(20, 3, 1)),
                            layer(sinks(6, 2, 24, 16, 0.2, window=7, kv_from=0), moe(16, 2, 2))], eps=2e-3, embed=4.0, cap=12.0),
    "B": document(96, 211, [layer(differential(6, 1, 64, 128, 0.12, 0.25, window=100, keep=5), moe(60, 6, 4)),
                            layer(sinks(6, 3, 64, 64, 0.1, window=33), moe(28, 7, 2)),
                            layer(differential(4, 4, 24, 48, 0.2, 0.8, window=24)),
                            layer(sinks(3, 3, 64, 64, 0.15, window=80, kv_from=1), moe(40, 1, 1)),
                            layer(differential(2, 1, 20, 12, 0.3, 0.1), moe(16, 3, 2)),
                            layer(sinks(8, 8, 16, 16, 0.25), moe(16, 4, 2))], eps=1e-6, embed=1.7, cap=50.0),
}
# One layer each: a mechanism alone (no feed-forward unless the feed-forward is what stands alone).
ALONE = {
    "differential": document(48, 97, [layer(differential(4, 2, 24, 20, 0.3, 0.3, window=24, keep=4))]),
    # two keys as wide as a value: in bfloat16 these take the tensor-core kernels of heads of 48, 64 and 128 (the last with the kernel whose
    # two halves are the maps)
    "differential_48": document(48, 97, [layer(differential(4, 2, 24, 48, 0.12, 0.3, window=24, keep=4))], cap=None),
    "differential_64": document(64, 97, [layer(differential(2, 2, 32, 64, 0.1, 0.7, window=24, keep=4))], embed=0.6),
    "differential_128": document(64, 97, [layer(differential(6, 2, 64, 128, 0.2, 0.3, window=24, keep=4))]),
    "differential_128_wide": document(64, 61, [layer(differential(4, 4, 64, 128, 0.1, 0.45, window=130, keep=70))]),
    "differential_open": document(40, 61, [layer(differential(3, 3, 32, 64, 0.2, 0.3))]),
    "sinks": document(48, 97, [layer(sinks(4, 2, 24, 20, 0.1, window=24))]),
    "sinks_48": document(48, 97, [layer(sinks(6, 2, 48, 48, 0.2, window=24))], cap=None),
    "sinks_64": document(64, 97, [layer(sinks(4, 2, 64, 64, 0.15, window=24))]),
    "sinks_128": document(64, 61, [layer(sinks(6, 2, 128, 128, 0.1, window=100))]),
    "sinks_open": document(40, 61, [layer(sinks(3, 3, 16, 16, 0.5))]),
    "shared": document(64, 97, [layer(sinks(4, 2, 64, 64, 0.15, window=10)), layer(sinks(2, 2, 64, 64, 0.03, window=24, kv_from=0))], embed=0.5),
    "experts": document(48, 97, [layer(sinks(2, 2, 8, 8, 0.5, window=8), moe(36, 6, 3))]),
    "experts_all": document(40, 61, [layer(sinks(2, 2, 8, 8, 0.5, window=8), moe(20, 5, 5))]),
    # one expert per token: a choice that flips swaps the whole feed-forward
    "experts_one": document(40, 61, [layer(sinks(2, 2, 8, 8, 0.5, window=8), moe(12, 4, 1))]),
}


def make_weights(doc: dict, seed: int, gain: float = 1.5, decided: bool = False) -> dict[str, torch.Tensor]:
    """bfloat16 tensors under the design's names: matrices N(0, gain^2 / in), norm weights around 1, biases and sinks of the size of what they
    stand beside.  ``decided``: the routers' biases are steps of 1.5 in a random order and their matrices small, so that the biases alone settle which
    experts are chosen while the weights still follow the logits."""
    from hyperion_b200.models import DecoderModel, get_architecture

    entry = get_architecture("Zurevik")
    model = DecoderModel(entry.build_spec(entry.read_config(doc)), torch.float32, torch.device("meta"))
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, wanted in model.expected_tensors().items():
        shape = tuple(wanted.shape)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif name.endswith("router.b"):
            t = 1.5 * torch.randperm(shape[0], generator=g).float() if decided else torch.randn(shape, generator=g)
        elif last == "router":  # undecided: few tokens whose best experts lie so close that a rounding upstream swaps them
            t = torch.randn(shape, generator=g) * ((0.2 if decided else 3.0 * gain) / shape[-1] ** 0.5)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = torch.randn(shape, generator=g) * (0.6 / shape[-1] ** 0.25)
        elif last == "sink":
            t = 1.0 + torch.randn(shape, generator=g)
        elif last == "b":
            t = 0.5 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * (gain / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16)
    return out


def align_keys_with_queries(doc: dict, weights: dict[str, torch.Tensor]) -> None:
    """Make one score stand out: keys are made by the matrices (biases, norms) that make the queries (every key head takes its first query
    head's), so a key made from the same token as the query meets it with cosine 1, where other keys' cosines are about 1 / sqrt(dim)."""
    for index, entry in enumerate(doc["layers"]):
        m, p = entry["mixer"], f"l{index}.mix."
        if p + "k" not in weights:
            continue
        rep, rows = m["heads"] // m["kv_heads"], m["dim"] * (2 if entry["type"] == "attention" else 1)
        weights[p + "k"] = weights[p + "q"].view(m["heads"], rows, -1)[::rep].reshape(m["kv_heads"] * rows, -1).clone()
        if entry["type"] == "attention":
            weights[p + "k.norm"] = weights[p + "q.norm"].clone()
            # the second map's queries look elsewhere: where both maps see the marker alike, their difference hides how much
            q = weights[p + "q"].view(m["heads"], 2, m["dim"], -1).clone()
            q[:, 1] = q[:, 1].flip(1)
            weights[p + "q"] = q.reshape(weights[p + "q"].shape)
        else:
            weights[p + "k.b"] = weights[p + "q.b"].view(m["heads"], rows)[::rep].reshape(-1).clone()
    # the last token of the vocabulary is the marker, the one before it the query: the marker's embedding is mostly the
    # query's, so its key points where the query points, and partly its own, so its value is another
    own = torch.randn(weights["embed"].shape[1], generator=torch.Generator().manual_seed(99))
    weights["embed"][-1] = ((2.0 * weights["embed"][-2].float() + own) / 5 ** 0.5).to(torch.bfloat16)


MARKED = ("differential", "differential_48", "differential_64", "differential_128", "sinks", "sinks_48", "sinks_64", "differential_open", "sinks_open", "shared")


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from hyperion_b200.weights import write_file

    root = tmp_path_factory.mktemp("zurevik_models")
    made = {}
    for index, (name, doc) in enumerate({**CONFIGS, **ALONE}.items()):
        folder = root / name
        folder.mkdir()
        (folder / "config.json").write_text(json.dumps(doc))
        weights = make_weights(doc, 23 + index, gain=1.2 if name in CONFIGS else 1.5, decided=name in CONFIGS)
        if name in MARKED:
            align_keys_with_queries(doc, weights)
        write_file(folder / "model.safetensors", weights)
        made[name] = folder
    return made


_plain_cache: dict = {}


def plain_logits(folder: Path, ids) -> np.ndarray:
    key = (str(folder), tuple(ids))
    if key not in _plain_cache:
        config, weights = plain.read_model_folder(folder)
        _plain_cache[key] = plain.forward(config, weights, list(ids)).numpy()
    return _plain_cache[key]


def ids_for(seed: int, count: int, vocab: int) -> list[int]:
    return torch.randint(0, vocab, (count,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine_for(folder, dtype, **options):
    from hyperion_b200.api import Engine

    options.setdefault("page_size", 16)
    options.setdefault("max_tokens", 1024)
    options.setdefault("max_requests", 4)
    return Engine.from_folder(folder, dtype=dtype, **options)


def row_errors(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    got, want = np.atleast_2d(got), np.atleast_2d(want)
    return np.sqrt(((got - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean(axis=1))


def relative_error(got: np.ndarray, want: np.ndarray) -> float:
    """The largest difference against the largest logit: the sharp measure, which a float32 run meets.  For bfloat16 results the worst row's
    root-mean-square difference against its root-mean-square logit."""
    sharp = float(np.abs(got - want).max() / np.abs(want).max())
    return sharp if sharp <= TOLERANCE["float32"] else float(row_errors(got, want).max())


def assert_close(got: np.ndarray, want: np.ndarray, dtype: str, what=None, routed: bool = False, deep: bool = False) -> None:
    """``routed`` (a router that follows its input): in bfloat16 a token whose best experts lie close together may go to another expert than in exact
    arithmetic: up to a fifth of the rows may be off.  ``deep`` (a model of several layers): three rows in a hundred may be off.  Either way the
    middle row stays within half the tolerance (a fault of a kernel or a cache moves every row).  float32 is held to its line without
    exceptions."""
    assert np.isfinite(got).all(), what
    if (routed or deep) and dtype == "bfloat16":
        errors = row_errors(got, want)
        over, middle = float((errors > TOLERANCE[dtype]).mean()), float(np.median(errors))
        assert over <= (0.2 if routed else 0.03) and middle <= TOLERANCE[dtype] / 2, (what, over, middle)
        return
    error = relative_error(got, want)
    assert error <= TOLERANCE[dtype], (what, error)


def run_cut(engine, name, ids, sizes) -> np.ndarray:
    """One request in portions of the given sizes (cycled), every position's logits."""
    from hyperion_b200.engine.batch import StepEntry

    rows, at, k = [], 0, 0
    while at < len(ids):
        n = min(sizes[k % len(sizes)], len(ids) - at)
        k += 1
        rows.append(engine.step([StepEntry(name, ids[at:at + n], list(range(n)))]).cpu().numpy().copy())
        at += n
    engine.finish(name)
    engine.check()
    return np.concatenate(rows)


# ------------------------------------------------------------------------------------------ every mechanism alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_layer_of_each_kind(folders, name, dtype):
    """A model of one layer (two where one reads the other's keys): the whole prompt at once, again in portions of 5, 2, 1, 9 tokens, and
    over larger pages."""
    vocab = ALONE[name]["vocab"]
    ids = ids_for(3, 75, vocab)
    want = plain_logits(folders[name], ids)
    routed = any(entry["mlp"] is not None for entry in ALONE[name]["layers"])
    for page_size in (8, 64):
        engine = engine_for(folders[name], dtype, page_size=page_size)
        assert_close(run_cut(engine, "w", ids, [len(ids)]), want, dtype, "whole", routed)
        assert_close(run_cut(engine, "p", ids, [5, 2, 1, 9]), want, dtype, "portions", routed)


def test_which_kernels_a_shape_takes(folders):
    for name, fast in (("differential", False), ("differential_48", True), ("differential_128", True), ("sinks", False), ("sinks_48", True), ("sinks_64", True)):
        for dtype in ("float32", "bfloat16"):
            assert engine_for(folders[name], dtype).model.layers[0].mixer.fast == (fast and dtype == "bfloat16"), (name, dtype)


def test_router_bias_and_softmax_over_the_chosen():
    """The router alone against the plain function, and the same bits whether a token comes alone or with hundreds."""
    from hyperion_b200.ops import moe as ops_moe

    g = torch.Generator().manual_seed(11)
    for experts, top, hidden in ((11, 5, 40), (1, 1, 24), (33, 33, 37), (5, 2, 130), (64, 8, 256)):
        x = torch.randn(600, hidden, generator=g)
        w = {"router": torch.randn(experts, hidden, generator=g) * 0.3, "router.b": torch.randn(experts, generator=g)}
        want_chosen, want_weight = plain.route(x.double(), {k: v.double() for k, v in w.items()}, "", top)
        router, bias = w["router"].cuda(), w["router.b"].cuda()
        for dtype in (torch.float32, torch.bfloat16):
            rows = x.to(dtype).cuda()
            chosen, weight = ops_moe.route_softmax(rows, router, bias, top)
            if dtype == torch.float32:
                assert torch.equal(chosen.cpu().long(), want_chosen)
                assert (weight.cpu().double() - want_weight).abs().max() <= 2e-6
            assert (weight.sum(dim=1) - 1).abs().max() <= 1e-5
            few_chosen, few_weight = ops_moe.route_softmax(rows[37:40], router, bias, top)
            assert torch.equal(few_chosen, chosen[37:40]) and torch.equal(few_weight, weight[37:40])
    # equal logits: the lowest index first
    chosen, weight = ops_moe.route_softmax(torch.zeros(3, 8).cuda(), torch.zeros(6, 8).cuda(), None, 4)
    assert chosen.cpu().tolist() == [[0, 1, 2, 3]] * 3 and torch.equal(weight.cpu(), torch.full((3, 4), 0.25))


@pytest.mark.parametrize("hidden", [8, 40, 130, 516, 2048, 4100])
def test_the_sum_of_two_sublayers_and_two_norms(hidden):
    """Dense sublayer outputs, a product in split-K pieces, expert rows with weights, either alone, rows picked out, one norm and two."""
    from hyperion_b200 import ops
    from hyperion_b200.ops import moe as ops_moe
    from hyperion_b200.ops.gemm import SplitSum

    g = torch.Generator().manual_seed(hidden)
    tokens, experts, top, eps = 21, 5, 3, 1e-5
    h = 3 * torch.randn(tokens, hidden, generator=g)
    w1, w2 = 1 + 0.2 * torch.randn(hidden, generator=g), 1 + 0.2 * torch.randn(hidden, generator=g)
    for dtype, tolerance in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        a, b = torch.randn(tokens, hidden, generator=g).to(dtype), torch.randn(tokens, hidden, generator=g).to(dtype)
        pieces = torch.randn(4, tokens, hidden, generator=g)
        chosen = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).int()
        weights = torch.rand(tokens, top, generator=g)
        where = ops_moe.plan(chosen.cuda(), None, experts)
        y = torch.randn(where.capacity, hidden, generator=g).to(dtype)
        picked = (y.double()[where.slot_of.cpu().long()].view(tokens, top, hidden) * weights.double()[:, :, None]).sum(dim=1)
        rows_of = ops_moe.WeightedRows(y.cuda(), where, weights.cuda(), a.cuda())
        firsts = {"none": (None, 0), "dense": (a.cuda(), a.double()), "pieces": (SplitSum(pieces.cuda(), None, dtype), pieces.double().sum(dim=0))}
        seconds = {"none": (None, 0), "dense": (b.cuda(), b.double()), "experts": (rows_of, picked)}
        for (first_name, (first, first_want)) in firsts.items():
            for (second_name, (second, second_want)) in seconds.items():
                stream = h.cuda()
                x1, x2 = ops.add_pair_norms(stream, first, second, w1.cuda(), w2.cuda(), eps, dtype)
                total = h.double() + (first_want + second_want)
                assert (stream.cpu().double() - total).abs().max() <= 1e-5 * total.abs().max(), (first_name, second_name)
                for got, w in ((x1, w1), (x2, w2)):
                    want = plain.rms_norm(total, w.double(), eps)
                    assert got.dtype == dtype and (got.cpu().double() - want).abs().max() <= tolerance * want.abs().max(), (first_name, second_name)
                rows = torch.tensor([20, 3, 3], dtype=torch.int32)
                stream = h.cuda()
                one, none = ops.add_pair_norms(stream, first, second, w1.cuda(), None, eps, dtype, rows.cuda())
                assert none is None and torch.equal(stream.cpu(), h)
                assert (one.cpu().double() - plain.rms_norm(total, w1.double(), eps)[rows.long()]).abs().max() <= tolerance * total.abs().max()


def test_the_cap_of_the_logits():
    from hyperion_b200 import ops

    g = torch.Generator().manual_seed(3)
    for rows, columns in ((1, 1), (3, 517), (5, 4096)):
        x = 60 * torch.randn(rows, columns, generator=g)
        got = ops.soft_cap_(x.cuda(), 17.0).cpu().double()
        assert (got - plain.soft_cap(x.double(), 17.0)).abs().max() <= 1e-5
    with pytest.raises(ops.KernelError):
        ops.soft_cap_(x.cuda().bfloat16(), 17.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_heads_are_normed_biased_and_stored(dtype):
    """Queries to a buffer, keys of one and of two maps and values to pages in either arrangement, sizes that are and are not whole 16-byte
    pieces, with and without norms and a bias."""
    from hyperion_b200 import ops

    g = torch.Generator().manual_seed(7)
    tolerance = 2e-6 if dtype == torch.float32 else 1e-2
    for heads, kv_heads, d, e, maps, norm, bias in ((4, 2, 24, 48, 2, True, False), (3, 1, 7, 5, 2, True, True), (6, 3, 64, 64, 1, False, True), (2, 2, 64, 128, 2, True, False),
                                                    (1, 1, 200, 40, 1, True, True), (2, 1, 1, 1, 2, True, False)):
        for tokens in (3, 530):
            page, pages = 8, 80
            qw, kw, vw, pad = heads * maps * d, kv_heads * maps * d, kv_heads * e, 3
            x = torch.randn(tokens, qw + kw + vw + pad, generator=g)
            b = torch.randn(qw + kw + vw, generator=g) if bias else None
            wq, wk = (1 + 0.2 * torch.randn(d, generator=g), 1 + 0.2 * torch.randn(d, generator=g)) if norm else (None, None)
            cache = torch.zeros((pages, 2, kv_heads, page, e) if maps * d == e else (pages, kv_heads, page, maps * d + e), dtype=dtype).cuda()
            table = torch.randperm(pages, generator=g).int().view(1, pages)
            positions = (torch.arange(tokens, dtype=torch.int32) + 5).clamp(max=page * pages - 1)
            q = torch.empty(tokens, qw, dtype=dtype).cuda()
            ops.heads_store(x.cuda(), 0, qw, qw + kw, heads, kv_heads, d, e, positions.cuda(), q_out=q, maps=maps, bias=b.cuda() if bias else None,
                            q_norm=wq.cuda() if norm else None, k_norm=wk.cuda() if norm else None, eps=1e-5, cache=cache, block_table=table.cuda(),
                            token_row=torch.zeros(tokens, dtype=torch.int32).cuda(), page_size=page)
            full = x[:, :qw + kw + vw].double() + (b.double() if bias else 0)
            wanted_q, wanted_k = full[:, :qw].reshape(tokens, heads * maps, d), full[:, qw:qw + kw].reshape(tokens, kv_heads, maps, d)
            if norm:
                wanted_q, wanted_k = plain.rms_norm(wanted_q, wq.double(), 1e-5), plain.rms_norm(wanted_k, wk.double(), 1e-5)
            wanted_v = full[:, qw + kw:].reshape(tokens, kv_heads, e)
            assert (q.cpu().double().view(tokens, heads * maps, d) - wanted_q).abs().max() <= tolerance * wanted_q.abs().max()
            where = table[0, (positions // page).long()].long()
            slot = (positions % page).long()
            host = cache.cpu().double()
            if maps * d == e:
                got_k, got_v = host[where, 0, :, slot], host[where, 1, :, slot]
            else:
                both = host[where, :, slot]
                got_k, got_v = both[..., :maps * d], both[..., maps * d:]
            last = slice(None) if tokens < page * pages - 5 else slice(0, page * pages - 6)
            assert (got_k.reshape(tokens, kv_heads, maps, d) - wanted_k)[last].abs().max() <= tolerance * wanted_k.abs().max()
            assert (got_v - wanted_v)[last].abs().max() <= tolerance * wanted_v.abs().max()


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_against_token_by_token_and_portions(folders, name, dtype):
    vocab = CONFIGS[name]["vocab"]
    ids = ids_for(5, 150, vocab)
    want = plain_logits(folders[name], ids)
    engine = engine_for(folders[name], dtype, page_size=8 if name == "A" else 16)
    results = {"whole": run_cut(engine, "w", ids, [len(ids)]), "single": run_cut(engine, "s", ids, [1]),
               "pairs": run_cut(engine, "p", ids, [2]), "mixed sizes": run_cut(engine, "m", ids, [7, 2, 16, 3, 33, 1, 1, 64])}
    for how, got in results.items():
        assert_close(got, want, dtype, how, deep=True)
        if dtype == "float32":
            assert np.array_equal(got, results["whole"]), how  # float32: the same bits however the work is cut


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_requests_together_over_pages_that_are_used_again(folders, name, dtype):
    """Six requests of unequal length through a cache of 3 slots and too few pages for all: portions of some beside single tokens of
    others, a request sitting out now and then; as one ends, the next takes its pages."""
    from hyperion_b200.engine.batch import StepEntry

    vocab = CONFIGS[name]["vocab"]
    lengths = [90, 41, 130, 17, 66, 101]
    requests = {f"r{i}": ids_for(50 + i, n, vocab) for i, n in enumerate(lengths)}
    want = {rid: plain_logits(folders[name], ids) for rid, ids in requests.items()}
    engine = engine_for(folders[name], dtype, page_size=16, max_tokens=3 * 144, max_requests=3)
    waiting, live, sizes, k, step = list(requests), {}, [5, 2, 19, 3, 8, 2, 30, 4], 0, 0
    got_rows, want_rows, owners = [], [], {}
    while waiting or live:
        while waiting and len(live) < 3:
            live[waiting.pop(0)] = 0
        entries = []
        for j, rid in enumerate(list(live)):
            ids, at = requests[rid], live[rid]
            if (step + j) % 5 == 4 and len(live) > 1:
                continue
            n = 1 if at >= len(ids) - 10 else min(sizes[k % len(sizes)], len(ids) - 10 - at)
            k += 1
            entries.append(StepEntry(rid, ids[at:at + n], list(range(n))))
        logits = engine.step(entries).cpu().numpy()
        row = 0
        for entry in entries:
            at = live[entry.request]
            n = len(entry.tokens)
            got_rows.append(logits[row:row + n])
            want_rows.append(want[entry.request][at:at + n])
            row += n
            live[entry.request] = at + n
            for group in range(len(engine.cache.paged)):
                for page in engine.cache.table(group, entry.request):
                    if page >= 0:
                        owners.setdefault((group, page), set()).add(entry.request)
            if at + n == len(requests[entry.request]):
                engine.finish(entry.request)
                del live[entry.request]
        step += 1
    engine.check()
    engine.cache.check()
    assert_close(np.concatenate(got_rows), np.concatenate(want_rows), dtype, deep=True)
    for group in range(len(engine.cache.paged)):  # in every group some page served more than one request
        assert max(len(users) for (g, _), users in owners.items() if g == group) >= 2


def test_pages_of_a_window_go_back_and_those_of_the_first_tokens_stay(folders):
    """A request of 300 tokens through one layer with a window of 24 and four kept first tokens over pages of 8, in a pool of eight pages."""
    from hyperion_b200.engine.batch import StepEntry

    name = "differential_48"
    ids = ids_for(17, 300, ALONE[name]["vocab"])
    want = plain_logits(folders[name], ids)
    for dtype in ("float32", "bfloat16"):
        engine = engine_for(folders[name], dtype, page_size=8, max_tokens=64)
        got = []
        for at in range(0, 300, 20):
            got.append(engine.step([StepEntry("r", ids[at:at + 20], list(range(20)))]).cpu().numpy().copy())
            held = [b for b, page in enumerate(engine.cache.table(0, "r")) if page >= 0]
            assert held[0] == 0 and len(held) <= 5, held
        engine.check()
        assert_close(np.concatenate(got), want, dtype)


def _marked(seed: int, length: int, vocab: int, places) -> list[int]:
    """Random tokens that end in the query token, with the marker at the given positions and nowhere else."""
    ids = ids_for(seed, length, vocab - 2)  # the last two tokens of the vocabulary are kept for the marked places
    ids[-1] = vocab - 2
    for place in places:
        ids[place] = vocab - 1
    return ids


def _as_a_prompt_and_decoded(engine, ids, want, dtype, what):
    """The last row of the whole prompt, of two portions, and of a tail of 30 tokens decoded one by one."""
    from hyperion_b200.engine.batch import StepEntry

    whole = engine.step([StepEntry("w", ids, [len(ids) - 1])]).cpu().numpy()[0]
    engine.finish("w")
    assert relative_error(whole, want[-1]) <= TOLERANCE[dtype], (what, "whole")
    head = len(ids) - 30
    engine.step([StepEntry("d", ids[:head], [])])
    for at in range(head, len(ids)):
        last = engine.step([StepEntry("d", [ids[at]], [0])]).cpu().numpy()[0].copy()
        assert relative_error(last, want[at]) <= TOLERANCE[dtype], (what, at)
    engine.finish("d")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["differential", "differential_48", "differential_64", "differential_128", "sinks", "sinks_48", "sinks_64", "shared"])
def test_keys_just_inside_and_just_outside_the_window(folders, name, dtype):
    """A window of 24 positions over pages of 8: a marker whose key scores high against the last query stands 23 places back (the last key the
    window keeps), 24 places back (the first it does not), one place, one page and two pages back, and 22 and 25; the prompts end at and around
    multiples of a page.  In ``shared`` the window is the borrowing layer's, wider than the one of the layer that owns the keys."""
    vocab, window = ALONE[name]["vocab"], 24
    engine = engine_for(folders[name], dtype, page_size=8)
    for length in (120, 121, 71):
        for back in (1, 8, 16, window - 2, window - 1, window, window + 1):
            ids = _marked(700 + length + back, length, vocab, [length - 1 - back])
            _as_a_prompt_and_decoded(engine, ids, plain_logits(folders[name], ids), dtype, (length, back))
    engine.check()
    # the marked key and the window's edge matter: the plain logits move by many float32 tolerances when the key is taken away, and
    # a window that is one place longer or shorter moves them too
    seen, unseen = _marked(1, 120, vocab, [119 - (window - 1)]), _marked(1, 120, vocab, [119 - window])
    without = list(seen)
    without[119 - (window - 1)] = 0
    base = plain_logits(folders[name], seen)[-1]
    assert relative_error(plain_logits(folders[name], without)[-1], base) > 50 * TOLERANCE["float32"]
    config, weights = plain.read_model_folder(folders[name])
    for ids, size in ((seen, window - 1), (unseen, window + 1)):
        other = json.loads(json.dumps(config))
        other["layers"][-1]["mixer"]["mask"]["size"] = size
        assert relative_error(plain.forward(other, weights, ids).numpy()[-1], plain_logits(folders[name], ids)[-1]) > 50 * TOLERANCE["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["differential", "differential_48", "differential_64", "differential_128"])
def test_the_kept_first_tokens_and_the_next_ones(folders, name, dtype):
    """Four first tokens stay visible beside a window of 24: the marker stands at positions 0 and 3 (seen from everywhere), 4 and 5 (lost with the
    window), with prompts so short that window and kept tokens meet or overlap, and so long that pages between them have gone."""
    vocab = ALONE[name]["vocab"]
    engine = engine_for(folders[name], dtype, page_size=8)
    for length in (31, 33, 200, 321):
        for place in (0, 3, 4, 5):
            ids = _marked(900 + length + place, length, vocab, [place])
            _as_a_prompt_and_decoded(engine, ids, plain_logits(folders[name], ids), dtype, (length, place))
    engine.check()
    config, weights = plain.read_model_folder(folders[name])
    for place, keep in ((3, 3), (4, 5)):  # one kept token fewer loses the marker at 3, one more finds the one at 4
        ids = _marked(5, 200, vocab, [place])
        other = json.loads(json.dumps(config))
        other["layers"][0]["mixer"]["mask"]["keep_first"] = keep
        assert relative_error(plain.forward(other, weights, ids).numpy()[-1], plain_logits(folders[name], ids)[-1]) > 50 * TOLERANCE["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["differential_open", "sinks_open"])
def test_a_key_far_away_among_hundreds(folders, name, dtype):
    """No window: the marker stands 1, 7, 8, 9, 64, 300 and 690 places behind the last query among 700 tokens, as a whole prompt and with
    the tail decoded."""
    vocab = ALONE[name]["vocab"]
    engine = engine_for(folders[name], dtype, page_size=8, max_tokens=1536)
    for back in (1, 7, 8, 9, 64, 300, 690):
        ids = _marked(800 + back, 700, vocab, [699 - back])
        want = plain_logits(folders[name], ids)
        _as_a_prompt_and_decoded(engine, ids, want, dtype, back)
    engine.check()
    without = list(ids)
    without[699 - 690] = 0
    assert relative_error(plain_logits(folders[name], without)[-1], plain_logits(folders[name], ids)[-1]) > 50 * TOLERANCE["float32"]


def test_sink_gate_and_both_maps_matter(folders):
    """What the runs above are held to moves by many tolerances when the sink is left out, the gate is, the second map's weight is that of ``diff``
    alone, or the head norm's factor is left out."""
    for name, tensor, value in (("sinks", "l0.mix.sink", -30.0), ("sinks", "l0.mix.g", 0.0), ("differential", "l0.mix.g", 0.0), ("differential", "l0.mix.lq1", 0.0),
                                ("differential", "l0.mix.lk2", 0.0), ("sinks", "l0.mix.k.b", 0.0), ("sinks", "l0.mix.v.b", 0.0), ("experts", "l0.mlp.router.b", 0.0)):
        ids = ids_for(3, 75, ALONE[name]["vocab"])
        config, weights = plain.read_model_folder(folders[name])
        weights[tensor] = torch.full_like(weights[tensor], value)
        assert relative_error(plain.forward(config, weights, ids).numpy(), plain_logits(folders[name], ids)) > 50 * TOLERANCE["float32"], (name, tensor)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_first_tokens_and_long_decoding(folders, name, dtype):
    from hyperion_b200.engine.batch import StepEntry

    vocab = CONFIGS[name]["vocab"]
    ids = ids_for(8, 400, vocab)
    want = plain_logits(folders[name], ids)
    engine = engine_for(folders[name], dtype, page_size=32, max_tokens=512)
    rows = []
    for token in ids:  # position 0 alone, then every other one: a one-token prompt and 399 decoded tokens
        rows.append(engine.step([StepEntry("r", [token], [0])]).cpu().numpy()[0].copy())
    engine.finish("r")
    pair = engine.step([StepEntry("pair", ids[:2], [0, 1])]).cpu().numpy().copy()
    engine.finish("pair")
    engine.check()
    single = np.stack(rows)
    assert_close(single, want, dtype, deep=True)
    assert_close(single[:8], want[:8], dtype, "the first tokens")
    assert_close(pair, want[:2], dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["differential_64", "differential_128", "differential_128_wide", "sinks_64", "sinks_128"])
def test_windows_in_the_tensor_core_kernels(folders, name, dtype):
    """450 tokens: as one prompt (tiles whose queries' windows begin in the middle of a key tile, kept first tokens that fill part of one or more
    than one page), in two portions and a tail decoded token by token (the split-key kernel), and three requests of unequal progress side by side."""
    from hyperion_b200.engine.batch import StepEntry

    vocab = ALONE[name]["vocab"]
    ids = ids_for(77, 450, vocab)
    want = plain_logits(folders[name], ids)
    engine = engine_for(folders[name], dtype, max_tokens=2048)
    assert_close(run_cut(engine, "w", ids, [len(ids)]), want, dtype, "whole")
    got = [engine.step([StepEntry("d", ids[:300], list(range(300)))]).cpu().numpy().copy()]
    got.append(engine.step([StepEntry("d", ids[300:420], list(range(120)))]).cpu().numpy().copy())
    for at in range(420, 450):
        got.append(engine.step([StepEntry("d", [ids[at]], [0])]).cpu().numpy().copy())
    engine.finish("d")
    assert_close(np.concatenate(got), want, dtype, "two portions and a decoded tail")
    engine.step([StepEntry("a", ids[:199], []), StepEntry("b", ids[:30], [])])
    got = engine.step([StepEntry("a", [ids[199]], [0]), StepEntry("b", ids[30:330], list(range(300))), StepEntry("c", ids[:2], [0, 1])]).cpu().numpy()
    engine.check()
    assert_close(got, np.concatenate([want[199:200], want[30:330], want[:2]]), dtype, "side by side")


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_through_the_scheduler(folders, name):
    from hyperion_b200.sampling import SamplingParams

    vocab = CONFIGS[name]["vocab"]
    prompts = [ids_for(300 + i, n, vocab) for i, n in enumerate([5, 37, 1, 80, 23])]
    config, weights = plain.read_model_folder(folders[name])

    def greedy(prompt, count):
        ids = list(prompt)
        for _ in range(count):
            ids.append(int(plain.forward(config, weights, ids)[-1].argmax()))
        return ids[len(prompt):]

    want = [greedy(prompt, 6) for prompt in prompts]
    engine = engine_for(folders[name], "float32", max_tokens=3 * 128, max_requests=3)
    got = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True), max_batch_tokens=48, prefill_chunk_busy=16)
    assert got == want
    engine = engine_for(folders[name], "bfloat16", max_tokens=3 * 128, max_requests=3)
    got = engine.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True), max_batch_tokens=48, prefill_chunk_busy=16)
    assert all(len(tokens) == 6 for tokens in got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_through_the_command(folders, dtype, tmp_path):
    """bin/trace_run on a model of this design: two requests side by side, one ends, a third takes its place."""
    name, vocab = "A", CONFIGS["A"]["vocab"]
    a, b, c = ids_for(1, 70, vocab), ids_for(2, 33, vocab), ids_for(3, 50, vocab)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [39]}, {"id": "b", "tokens": b[:31], "want": [0, 30]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[40:42], "want": [0, 1]}, {"id": "b", "tokens": b[31:32], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[32:], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c, "want": [49]}, {"id": "a", "tokens": a[42:], "want": [27]}], "end": ["a", "c"]}]
    text = "".join(json.dumps(s) + "\n" for s in steps)
    done = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folders[name]), "--dtype", dtype, "--out", str(tmp_path),
                           "--max-tokens", "192"], input=text, capture_output=True, text=True, timeout=900)
    assert done.returncode == 0, done.stderr[-3000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done ")] == [f"done {i}" for i in range(4)]
    ref = {"a": plain_logits(folders[name], a), "b": plain_logits(folders[name], b), "c": plain_logits(folders[name], c)}
    read = lambda step: np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(-1, vocab)
    expected = {0: [ref["a"][39], ref["b"][0], ref["b"][30]], 1: [ref["a"][40], ref["a"][41], ref["b"][31]], 2: [ref["b"][32]],
                3: [ref["c"][49], ref["a"][69]]}
    for step, rows in expected.items():
        assert_close(read(step), np.stack(rows), dtype, step)


def test_the_command_line_writes_a_random_model_and_generates_with_it(tmp_path):
    """``python -m hyperion_b200 random`` from a config.json of this design, then ``generate`` on the folder it wrote:
    the tokens are the plain implementation's greedy ones."""
    config = tmp_path / "config.json"
    config.write_text(json.dumps(CONFIGS["A"]))
    folder = tmp_path / "model"
    run = lambda *args: subprocess.run([sys.executable, "-m", "hyperion_b200", *args], capture_output=True, text=True, timeout=900, cwd=ROOT)
    done = run("random", "--config", str(config), "--out", str(folder), "--seed", "5", "--std", "0.3")
    assert done.returncode == 0, done.stderr[-2000:]
    prompt = ids_for(71, 19, CONFIGS["A"]["vocab"])
    done = run("generate", "-m", str(folder), "--dtype", "float32", "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "5", "--temperature", "0",
               "--ignore-eos", "--max-batch", "2")
    assert done.returncode == 0, done.stderr[-2000:]
    got = json.loads(done.stdout.strip().splitlines()[-1])
    plain_config, weights = plain.read_model_folder(folder)
    ids = list(prompt)
    for _ in range(5):
        ids.append(int(plain.forward(plain_config, weights, ids)[-1].argmax()))
    assert got["tokens"] == ids[len(prompt):] and got["finish_reason"] == "length"


# ------------------------------------------------------------------------------------------ configurations drawn at random
def _random_document(seed: int) -> dict:
    """A model whose every size, option and constant is drawn: widths, heads and groupings, head sizes that the tensor-core kernels take and
    others, windows, kept tokens, experts, layers without a feed-forward, layers that read an earlier layer's keys, in any order."""
    import random

    r = random.Random(seed)
    layers: list = []
    for _ in range(r.randint(2, 6)):
        mlp = moe(r.choice([8, 20, 36]), *(lambda n: (n, r.randint(1, n)))(r.randint(1, 9))) if r.random() < 0.75 else None
        lenders = [i for i, entry in enumerate(layers) if entry["type"] == "attention_2" and "kv_from" not in entry["mixer"]]
        kv = r.choice([1, 2, 3])
        heads, window = kv * r.choice([1, 2, 3]), r.choice([None, r.randint(1, 70), r.randint(1, 70)])
        kind = r.choice(["differential", "differential", "sinks", "sinks", "shared"])
        if kind == "shared" and lenders:
            source = r.choice(lenders)
            m = layers[source]["mixer"]
            layers.append(layer(sinks(m["kv_heads"] * r.choice([1, 2]), m["kv_heads"], m["dim"], m["vdim"], r.choice([0.1, 0.3]), window=window, kv_from=source), mlp))
        elif kind == "differential":
            dim = r.choice([4, 8, 12, 16, 24, 32, 64])
            vdim = r.choice([2 * dim, 2 * dim, dim, 12, 20])
            layers.append(layer(differential(heads, kv, dim, vdim, r.choice([0.1, 0.3, dim ** -0.5]), r.choice([0.0, 0.2, 0.5, 0.9]), window=window,
                                             keep=r.choice([0, 1, 4, 17, 40])), mlp))
        else:
            dim = r.choice([8, 16, 20, 32, 48, 64])
            layers.append(layer(sinks(heads, kv, dim, r.choice([dim, dim, 12, 24]), r.choice([0.1, 0.3, dim ** -0.5]), window=window), mlp))
    return document(r.choice([32, 40, 54, 64, 80, 128]), r.randint(40, 300), layers, eps=r.choice([1e-6, 1e-5, 1e-3]), embed=r.choice([0.5, 1.0, 9.0]),
                    cap=r.choice([None, 5.0, 30.0]))


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Ten models drawn at random, in float32 against the plain implementation: a whole prompt, the same in portions, and two requests of
    unequal progress side by side; in bfloat16 the middle row of the whole prompt and of the portions."""
    from hyperion_b200.engine.batch import StepEntry
    from hyperion_b200.weights import write_file

    doc = _random_document(seed)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(doc))
    write_file(folder / "model.safetensors", make_weights(doc, 100 + seed, gain=1.2, decided=True))
    ids, other = ids_for(seed, 90, doc["vocab"]), ids_for(seed + 50, 37, doc["vocab"])
    want, want_other = plain_logits(folder, ids), plain_logits(folder, other)
    engine = engine_for(folder, "float32", page_size=8, max_tokens=512)
    assert_close(run_cut(engine, "w", ids, [len(ids)]), want, "float32", ("whole", doc))
    assert_close(run_cut(engine, "p", ids, [3, 1, 2, 17]), want, "float32", ("portions", doc))
    engine.step([StepEntry("a", ids[:61], []), StepEntry("b", other[:5], [])])
    got = engine.step([StepEntry("a", [ids[61]], [0]), StepEntry("b", other[5:], list(range(32)))]).cpu().numpy()
    engine.check()
    assert_close(got, np.concatenate([want[61:62], want_other[5:]]), "float32", ("side by side", doc))
    engine = engine_for(folder, "bfloat16", page_size=8, max_tokens=512)
    for sizes in ([len(ids)], [3, 1, 2, 17]):
        errors = row_errors(run_cut(engine, "w", ids, sizes), want)
        assert np.median(errors) <= TOLERANCE["bfloat16"], (float(np.median(errors)), sizes, doc)


def test_sizes_of_one(tmp_path):
    """Every size that can be one is one (heads, key and value sizes, a window of one position, one kept token, one expert, an inner size of one):
    whole, in portions and token by token, in both precisions."""
    from hyperion_b200.weights import write_file

    docs = {
        "ones": document(8, 17, [layer(differential(1, 1, 1, 2, 1.0, 0.3, window=1, keep=1), moe(1, 1, 1)), layer(sinks(1, 1, 1, 1, 1.0, window=1), moe(4, 2, 1)),
                                 layer(sinks(1, 1, 1, 1, 0.5, window=2, kv_from=1))], eps=1e-4),
        "many": document(24, 50, [layer(differential(16, 1, 8, 16, 0.3, 0.5, window=33, keep=2), moe(8, 30, 6)), layer(sinks(12, 1, 16, 16, 0.25, window=5), moe(8, 9, 8))]),
    }
    for name, doc in docs.items():
        folder = tmp_path / name
        folder.mkdir()
        (folder / "config.json").write_text(json.dumps(doc))
        write_file(folder / "model.safetensors", make_weights(doc, 7, gain=1.2, decided=True))
        ids = ids_for(1, 90, doc["vocab"])
        want = plain_logits(folder, ids)
        for dtype in ("float32", "bfloat16"):
            engine = engine_for(folder, dtype, page_size=8, max_tokens=512)
            for sizes in ([len(ids)], [3, 1, 2, 17], [1]):
                assert_close(run_cut(engine, "w", ids, sizes), want, dtype, (name, sizes), deep=True)
