"""A plain, slow implementation of the Zurevik decoder: whole sequences, no cache, no batching, one
function per mechanism, torch on the CPU in float64 (or the dtype asked for).

It shares no code with the package: it reads the model folder with its own safetensors reader.
Notation: T tokens, W the model width, H query heads, G key/value heads, d the query/key size of a head
(of one map of it), e the value size.  Weights are stored [out, in].

The stream starts as embed[token] * scale.  A layer's two sublayers read the same stream through a norm each and
are added to it together:
    x <- x + (mixer(norm1(x)) + ff(norm2(x)))
The logits are cap * tanh((head . norm(x)) / cap).
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import torch

DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "F64": torch.float64, "I32": torch.int32, "I64": torch.int64}


def read_safetensors(path: Path) -> dict[str, torch.Tensor]:
    blob = Path(path).read_bytes()
    (length,) = struct.unpack("<Q", blob[:8])
    header = json.loads(blob[8 : 8 + length])
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        begin, end = meta["data_offsets"]
        raw = bytearray(blob[8 + length + begin : 8 + length + end])
        out[name] = torch.frombuffer(raw, dtype=DTYPES[meta["dtype"]]).reshape(meta["shape"]).clone() if raw else torch.zeros(meta["shape"], dtype=DTYPES[meta["dtype"]])
    return out


def read_model_folder(folder: Path) -> tuple[dict, dict[str, torch.Tensor]]:
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


# ------------------------------------------------------------------------------------------ small pieces
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * weight


def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def sees(T: int, window: int | None, keep_first: int = 0) -> torch.Tensor:
    """[T, T] bool: whether position i sees position j: the last ``window`` positions up to itself (None: all of them), and the first
    ``keep_first`` positions of the sequence whatever their distance."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if window is None else i - j < window
    return (j <= i) & (near | (j < keep_first))


def softmax_with_sink(scores: torch.Tensor, sink: torch.Tensor | None) -> torch.Tensor:
    """Softmax over the last dimension of [H, T, T]; ``sink`` [H]: one more term exp(sink) in a head's denominators."""
    if sink is None:
        return torch.softmax(scores, dim=-1)
    most = torch.maximum(scores.amax(dim=-1, keepdim=True), sink[:, None, None])
    p = torch.exp(scores - most)
    return p / (p.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - most))


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor, sink: torch.Tensor | None = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; query head h reads key/value head h // (H / G)."""
    rep = q.shape[1] // k.shape[1]
    scores = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, dim=1)) * scale
    weights = softmax_with_sink(scores.masked_fill(~seen[None], float("-inf")), sink)
    return torch.einsum("hij,jhe->ihe", weights, v.repeat_interleave(rep, dim=1))


def map_weight(w: dict, p: str, diff: float) -> torch.Tensor:
    """What the second map's output is multiplied by before it is taken off the first's: one number per layer."""
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


# ------------------------------------------------------------------------------------------ mixers
def differential_attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """Two softmax maps per head over the same values, the second taken off the first times a learned number; the head's result is
    divided by its root mean square, scaled by 1 - diff and gated entry by entry."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w[p + "q"].T).reshape(T, H, 2, d), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].T).reshape(T, G, 2, d), w[p + "k.norm"], eps)
    v = (h @ w[p + "v"].T).reshape(T, G, e)
    mask = m.get("mask")
    seen = sees(T, None if mask is None else mask["size"], 0 if mask is None else mask.get("keep_first", 0))
    first = attend(q[:, :, 0], k[:, :, 0], v, m["scale"], seen)
    second = attend(q[:, :, 1], k[:, :, 1], v, m["scale"], seen)
    o = unit_rms(first - map_weight(w, p, m["diff"]) * second, eps) * (1.0 - m["diff"])
    return (o.reshape(T, H * e) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def keys_and_values(h: torch.Tensor, w: dict, p: str, m: dict) -> tuple[torch.Tensor, torch.Tensor]:
    T, G = h.shape[0], m["kv_heads"]
    return (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, m["dim"]), (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, m["vdim"])


def sink_attention(h: torch.Tensor, w: dict, p: str, m: dict, k: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
    """Windowed attention with biases, a sink in the softmax and one gate per head, over keys and values that may be another layer's."""
    T, H = h.shape[0], m["heads"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, m["dim"])
    mask = m.get("mask")
    o = attend(q, k, v, m["scale"], sees(T, None if mask is None else mask["size"]), w[p + "sink"])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * m["vdim"]) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forward
def route(h: torch.Tensor, w: dict, p: str, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """([T, top] chosen experts, [T, top] their weights): the largest logits with the router's bias, a softmax over the chosen ones only."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    best = z.topk(top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def expert_ff(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return torch.relu(h @ w[p + "up"].T).pow(2) @ w[p + "down"].T


def experts_ff(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    chosen, weight = route(h, w, p, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, choice = (chosen == e).nonzero(as_tuple=True)
        if len(rows):
            out.index_add_(0, rows, weight[rows, choice][:, None] * expert_ff(h[rows], w, f"{p}e{e}."))
    return out


# ------------------------------------------------------------------------------------------ the model
def forward(config: dict, weights: dict[str, torch.Tensor], token_ids, dtype=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the stream after every layer."""
    w = {name: (t.to(dtype) if t.is_floating_point() else t) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    ids = torch.as_tensor(token_ids, dtype=torch.long)
    x = w["embed"][ids] * config["embedding"]["scale"]
    lent: dict[int, tuple[torch.Tensor, torch.Tensor]] = {}
    for index, layer in enumerate(config["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        a = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "attention":
            y = differential_attention(a, w, p + "mix.", m, eps)
        elif layer["type"] == "attention_2":
            source = m.get("kv_from")
            lent[index] = lent[source] if source is not None else keys_and_values(a, w, p + "mix.", m)
            y = sink_attention(a, w, p + "mix.", m, *lent[index])
        else:
            raise ValueError(f"no mixer {layer['type']!r}")
        if layer.get("mlp") is not None:
            y = y + experts_ff(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    z = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    cap = config.get("logit_softcap")
    return z if cap is None else soft_cap(z, cap)
