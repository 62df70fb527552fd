"""A plain, slow implementation of the Biropel decoder: whole sequences, no cache, no batching, one
function per mechanism, torch on the CPU in float64 (or the dtype asked for).

It shares no code with the package: it reads the model folder with its own safetensors reader.
Notation: T tokens, W the model width, H query heads, G key/value heads, d the query/key size of a head,
e the value size, R the number of residual streams.  Weights are stored [out, in].

The embedding row passes a norm and becomes every one of R residual streams X [R, T, W].  A sublayer f reads one
mixture of them and writes to all of them:
    u = sum_r a[r] X[r];   y = f(norm(u));   X[t] <- sum_r B[r, t] X[r] + c[t] y
and the streams are added up at the end.
"""
from __future__ import annotations

import json
import math
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


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def read_streams(streams: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    """[R, T, W] -> [T, W]: the mixture a sublayer reads."""
    return torch.einsum("r,rtw->tw", w[p + "in"], streams)


def write_streams(streams: torch.Tensor, y: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    """Every new stream is a mixture of the old ones plus its share of the sublayer's result."""
    return torch.einsum("rs,rtw->stw", w[p + "mix"], streams) + w[p + "out"][:, None, None] * y[None]


# ------------------------------------------------------------------------------------------ positions
def frequencies(rot: dict) -> tuple[list[float], float]:
    """(radians per position of every pair, the factor on cosine and sine).  With ``scaling``, pairs that turn often within the original
    length keep their frequency, pairs that turn rarely are slowed down by ``factor``, with a ramp between the two."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if scaling is None:
        return plain, 1.0

    def pair_that_turns(times: float) -> float:
        return dims * math.log(scaling["original"] / (2 * math.pi * times)) / (2 * math.log(base))

    low = max(math.floor(pair_that_turns(scaling["fast"])), 0)
    high = min(math.ceil(pair_that_turns(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x: torch.Tensor, rot: dict | None) -> torch.Tensor:
    """[T, heads, d]: entry i of a head's first ``dims`` entries turns together with entry i + dims / 2 by position times frequency."""
    if rot is None:
        return x
    half = rot["dims"] // 2
    f, factor = frequencies(rot)
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
    c, s = ((t * factor).to(x.dtype)[:, None, :] for t in (torch.cos(angle), torch.sin(angle)))
    first, second = x[..., :half], x[..., half : 2 * half]
    return torch.cat([first * c - second * s, second * c + first * s, x[..., 2 * half :]], dim=-1)


def temperature(T: int, temp: dict | None, dtype) -> torch.Tensor:
    """What queries are multiplied by, per position: it grows by steps of ``every`` positions."""
    if temp is None:
        return torch.ones(T, dtype=dtype)
    return torch.tensor([1.0 + temp["coef"] * math.log((p + 1) // temp["every"] + 1) for p in range(T)], dtype=torch.float64).to(dtype)


# ------------------------------------------------------------------------------------------ attention
def sees(T: int, window: int | None) -> torch.Tensor:
    """[T, T] bool: whether position i sees position j: itself and the ``window`` - 1 positions before it (None: all of them)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (torch.ones(T, T, dtype=torch.bool) if window is None else i - j < window)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor, cap: float | None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; query head h reads key/value head h // (H / G)."""
    rep = q.shape[1] // k.shape[1]
    scores = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(rep, dim=1)) * scale
    if cap is not None:
        scores = soft_cap(scores, cap)
    weights = torch.softmax(scores.masked_fill(~seen[None], float("-inf")), dim=-1)
    return torch.einsum("hij,jhe->ihe", weights, v.repeat_interleave(rep, dim=1))


def project(h: torch.Tensor, w: dict, name: str, heads: int, bias: bool) -> torch.Tensor:
    z = h @ w[name].T
    if bias:
        z = z + w[name + ".b"]
    return z.reshape(h.shape[0], heads, -1)


def keys_and_values(h: torch.Tensor, w: dict, p: str, m: dict, bias: bool, unit: bool, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    k = project(h, w, p + "k", m["kv_heads"], bias)
    if unit:
        k = unit_rms(k, eps)
    return rotate(k, m.get("rot")), project(h, w, p + "v", m["kv_heads"], bias)


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, k: torch.Tensor, v: torch.Tensor, bias: bool = False, unit: bool = False,
              gate: bool = False) -> torch.Tensor:
    """Grouped-query attention over keys and values that are given (they may be another layer's)."""
    T = h.shape[0]
    q = project(h, w, p + "q", m["heads"], bias)
    if unit:
        q = unit_rms(q, eps)
    q = rotate(q, m.get("rot")) * temperature(T, m.get("q_temp"), h.dtype)[:, None, None]
    mask = m.get("mask")
    o = attend(q, k, v, m["scale"], sees(T, None if mask is None else mask["size"]), m.get("softcap")).reshape(T, -1)
    if gate:
        o = o * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ------------------------------------------------------------------------------------------ recurrences
def causal_convolution(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """x [T, C], weight [C, taps] (the last column multiplies the current token), zeros before the start."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return bias + sum(weight[:, j] * padded[j : j + x.shape[0]] for j in range(taps))


def state_space(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """Mamba-2, token by token."""
    T, H, e, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = torch.split(silu(causal_convolution(xbc, w[p + "conv"], w[p + "conv.b"])), [inner, G * N, G * N], dim=-1)
    x = x.reshape(T, H, e)
    B, C = (t.reshape(T, G, N).repeat_interleave(H // G, dim=1) for t in (B, C))
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=1e9)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    S = torch.zeros(H, N, e, dtype=h.dtype)
    rows = []
    for t in range(T):
        S = decay[t][:, None, None] * S + torch.einsum("h,hn,he->hne", dt[t], B[t], x[t])
        rows.append(torch.einsum("hne,hn->he", S, C[t]) + w[p + "D"][:, None] * x[t])
    y = torch.stack(rows).reshape(T, inner) * silu(z)
    y = unit_rms(y.reshape(T, m["norm_groups"], -1), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def matrix_memory_gates(h: torch.Tensor, w: dict, p: str, cap: float) -> tuple[torch.Tensor, torch.Tensor]:
    """[T, H] each: the logarithms of the input gate and of the forget gate."""
    i = soft_cap(h @ w[p + "i"].T + w[p + "i.b"], cap)
    f = torch.nn.functional.logsigmoid(soft_cap(h @ w[p + "f"].T + w[p + "f.b"], cap))
    return i, f


def matrix_memory(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """The matrix memory of xLSTM, token by token, with its running maximum."""
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).reshape(T, H, d), (h @ w[p + "v"].T).reshape(T, H, e)
    i, f = matrix_memory_gates(h, w, p, m["gate_cap"])
    S, n, top = torch.zeros(H, d, e, dtype=h.dtype), torch.zeros(H, d, dtype=h.dtype), torch.zeros(H, dtype=h.dtype)
    rows = []
    for t in range(T):
        new = torch.maximum(f[t] + top, i[t])
        keep, take = torch.exp(f[t] + top - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + take[:, None, None] * torch.einsum("hd,he->hde", k[t], v[t])
        n = keep[:, None] * n + take[:, None] * k[t]
        top = new
        below = torch.maximum((n * q[t]).sum(dim=-1).abs(), torch.exp(-top)) + 1e-6
        rows.append(torch.einsum("hde,hd->he", S, q[t]) / below[:, None])
    o = unit_rms(torch.stack(rows), eps).reshape(T, H * e) * w[p + "norm"]
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------ feed-forward, two mixers side by side
def feed_forward(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return torch.relu(h @ w[p + "up"].T).pow(2) @ w[p + "down"].T


def side_by_side(left: torch.Tensor, right: torch.Tensor, w: dict, p: str, eps: float) -> torch.Tensor:
    return 0.5 * (rms_norm(left, w[p + "left.out"], eps) + rms_norm(right, w[p + "right.out"], eps))


# ------------------------------------------------------------------------------------------ the model
def forward(config: dict, weights: dict[str, torch.Tensor], token_ids, dtype=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the sum of the streams after every layer."""
    w = {name: (t.to(dtype) if t.is_floating_point() else t) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    ids = torch.as_tensor(token_ids, dtype=torch.long)
    streams = rms_norm(w["embed"][ids], w["embed.norm"], eps)[None].repeat(config["streams"], 1, 1)
    lent: dict[int, tuple[torch.Tensor, torch.Tensor]] = {}
    for index, layer in enumerate(config["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        h = rms_norm(read_streams(streams, w, p + "hc1."), w[p + "norm1"], eps)
        if layer["type"] == "attention":
            source = m.get("kv_from")
            lent[index] = lent[source] if source is not None else keys_and_values(h, w, p + "mix.", m, True, False, eps)
            y = attention(h, w, p + "mix.", m, eps, *lent[index], bias=True, gate=True)
        elif layer["type"] in ("parallel", "parallel_2"):
            unit = layer["type"] == "parallel_2"
            k, v = keys_and_values(h, w, p + "mix.left.", m["left"], False, unit, eps)
            left = attention(h, w, p + "mix.left.", m["left"], eps, k, v, unit=unit)
            right = (matrix_memory if unit else state_space)(h, w, p + "mix.right.", m["right"], eps)
            y = side_by_side(left, right, w, p + "mix.", eps)
        else:
            raise ValueError(f"no mixer {layer['type']!r}")
        streams = write_streams(streams, y, w, p + "hc1.")
        if layer.get("mlp") is not None:
            y = feed_forward(rms_norm(read_streams(streams, w, p + "hc2."), w[p + "norm2"], eps), w, p + "mlp.")
            streams = write_streams(streams, y, w, p + "hc2.")
        if layers_out is not None:
            layers_out.append(streams.sum(dim=0))
    return rms_norm(streams.sum(dim=0), w["final.norm"], eps) @ w["head"].T
