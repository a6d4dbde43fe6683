"""A plain, slow Ludelorn: whole sequences, no cache, explicit loops, one function per mechanism.

The oracle of the Ludelorn tests.  It shares no code with the package: it reads a model folder with its own
safetensors reader and computes every position from all tokens before it.  ``dtype`` is the arithmetic (float64 in
most tests).

Notation: T tokens, H query heads, G key/value heads, d key size, e value size, W window, P tokens per pooled block.
"""

from __future__ import annotations

import json
import math
import os
import struct

import numpy as np
import torch


def read_folder(path):
    """(config dictionary, name -> float64 tensor) of a model folder."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    with open(os.path.join(path, "model.safetensors"), "rb") as f:
        blob = f.read()
    (n,) = struct.unpack("<Q", blob[:8])
    header = json.loads(blob[8:8 + n])
    tensors = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        raw = blob[8 + n + a:8 + n + b]
        if info["dtype"] == "BF16":
            arr = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif info["dtype"] == "F32":
            arr = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        else:
            raise ValueError(f"{name}: dtype {info['dtype']}")
        tensors[name] = torch.from_numpy(arr.reshape(info["shape"]).copy())
    return config, tensors


# ---- norms -----------------------------------------------------------------------------------------------------

def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def stream_norm(x, g, eps):
    """The norm of the stream: one learned number for all coordinates."""
    return rms(x, eps) * g


# ---- positions -------------------------------------------------------------------------------------------------

def plain_frequencies(dims, base):
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn(dims, base, factor, original, fast, slow):
    """(frequencies, factor on cosine and sine): pairs that turn more than ``fast`` times within ``original``
    positions keep their frequency, those that turn less than ``slow`` times are slowed by ``factor``, a linear ramp
    over the pair's index between."""
    def index_of(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    freq = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        freq.append(f / factor * r + f * (1 - r))
    return freq, 0.1 * math.log(factor) + 1.0


def turn(x, positions, dims, freq, magnitude, interleaved):
    """x [T, heads, d]: pair i of the first ``dims`` sizes turns by position * freq[i] and grows by ``magnitude``;
    pair i is (2i, 2i + 1) when interleaved, else (i, i + dims/2).  The other sizes stay."""
    out = x.clone()
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        angle = positions.to(x.dtype) * freq[i]
        c, s = (magnitude * torch.cos(angle))[:, None], (magnitude * torch.sin(angle))[:, None]
        out[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
        out[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return out


def rotate(x, positions, rot, interleaved):
    sc = rot.get("scaling")
    if sc is None:
        freq, magnitude = plain_frequencies(rot["dims"], rot["base"]), 1.0
    else:
        freq, magnitude = yarn(rot["dims"], rot["base"], sc["factor"], sc["original"], sc["fast"], sc["slow"])
    return turn(x, positions, rot["dims"], freq, magnitude, interleaved)


def distance_bucket(n, B, D):
    """Which of B learned numbers a distance n takes: one each up to B/2, then logarithmically wider steps up to D.
    Decided with whole numbers: floor(m ln(n/h) / ln(D/h)) >= k exactly when (n/h)^m >= (D/h)^k, m = B - h."""
    h = B // 2
    if n < h:
        return n
    m, k = B - h, 0
    while h + k < B - 1 and n ** m * h ** (k + 1) >= D ** (k + 1) * h ** m:
        k += 1
    return h + k


# ---- attention core --------------------------------------------------------------------------------------------

def window_of(i, W):
    return range(max(0, i - W + 1), i + 1)


def blocks_before(i, W, P):
    """The blocks of P positions that lie wholly before the window of position i."""
    return [b for b in range(i // P + 1) if b * P + P - 1 <= i - W]


def attend(q, k, v, scale, W, pool=None, sink=None, rel=None, bias_max=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e].  ``sink`` [H]: exp(sink_h) joins the denominator.  ``rel``
    [B, H]: a number per distance bucket and head is added to the scaled score.  ``pool`` P: beside the window, one
    mean key and mean value for every block before it."""
    T, H, _ = q.shape
    G = k.shape[1]
    if pool is not None:
        whole = T // pool * pool
        pk = k[:whole].reshape(-1, pool, G, k.shape[-1]).mean(dim=1)
        pv = v[:whole].reshape(-1, pool, G, v.shape[-1]).mean(dim=1)
    out = torch.zeros((T, H, v.shape[-1]), dtype=q.dtype)
    group = torch.tensor([h // (H // G) for h in range(H)])
    for i in range(T):
        js = list(window_of(i, W))
        keys, values = k[js], v[js]
        if pool is not None:
            bs = blocks_before(i, W, pool)
            keys, values = torch.cat([pk[bs], keys]), torch.cat([pv[bs], values])
        s = torch.einsum("jhd,hd->hj", keys[:, group], q[i]) * scale
        if rel is not None:
            s = s + torch.stack([rel[distance_bucket(i - j, rel.shape[0], bias_max)] for j in js]).T
        m = s.max(dim=1).values
        if sink is not None:
            m = torch.maximum(m, sink)
        e = torch.exp(s - m[:, None])
        denom = e.sum(dim=1)
        if sink is not None:
            denom = denom + torch.exp(sink - m)
        out[i] = torch.einsum("hj,jhe->he", e / denom[:, None], values[:, group])
    return out


def element_gate(o, h, w):
    return o * torch.sigmoid(h @ w.T)


# ---- the mixers ------------------------------------------------------------------------------------------------

def windowed_heads(h, t, p, m, eps, positions):
    """Heads normed one by one, half-split rotation (YaRN), window, a gate per element."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ t[p + "q"].T).reshape(T, H, d), eps) * t[p + "q.norm"]
    k = rms((h @ t[p + "k"].T).reshape(T, G, d), eps) * t[p + "k.norm"]
    v = (h @ t[p + "v"].T).reshape(T, G, e)
    q, k = rotate(q, positions, m["rot"], False), rotate(k, positions, m["rot"], False)
    o = attend(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, -1)
    return element_gate(o, h, t[p + "g"]) @ t[p + "o"].T


def short_convolution(x, w, b):
    """y_t = silu(b + sum_j w[., K-1-j] x_(t-j)) per channel, x before the start is zero."""
    K = w.shape[1]
    y = torch.zeros_like(x) + b
    for j in range(min(K, x.shape[0])):
        y[j:] += x[:x.shape[0] - j] * w[:, K - 1 - j]
    return y * torch.sigmoid(y)


def state_space(h, t, p, m, eps, states=None):
    """S_t = exp(-exp(A) dt) S_(t-1) + dt B_t x_t^T, y_t = S_t^T C_t + D x_t per head; y silu(z), normed in equal
    parts, output matrix.  ``states``: a list that receives the state after every token."""
    T, H, e, N, G, parts = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"]
    inner = H * e
    u = h @ t[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = short_convolution(xbc, t[p + "conv"], t[p + "conv.b"])
    x = xbc[:, :inner].reshape(T, H, e)
    B, C = xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    dt = torch.nn.functional.softplus(dt + t[p + "dt_bias"], threshold=1e9)
    y = torch.zeros_like(x)
    S = torch.zeros((H, N, e), dtype=h.dtype)
    group = torch.tensor([i // (H // G) for i in range(H)])
    for i in range(T):
        decay = torch.exp(-torch.exp(t[p + "A_log"]) * dt[i])
        S = decay[:, None, None] * S + dt[i][:, None, None] * B[i][group][:, :, None] * x[i][:, None, :]
        y[i] = torch.einsum("hne,hn->he", S, C[i][group]) + t[p + "D"][:, None] * x[i]
        if states is not None:
            states.append(S.clone())
    y = y.reshape(T, inner) * (z * torch.sigmoid(z))
    y = rms(y.reshape(T, parts, -1), eps).reshape(T, inner) * t[p + "norm"]
    return y @ t[p + "o"].T


def side_by_side(h, t, p, m, eps, positions):
    left = windowed_heads(h, t, p + "left.", m["left"], eps, positions)
    right = state_space(h, t, p + "right.", m["right"], eps)
    return 0.5 * (rms(left, eps) * t[p + "left.out"] + rms(right, eps) * t[p + "right.out"])


def pooled_attention(h, t, p, m, eps, positions):
    """q and k normed over all heads at once, interleaved rotation, window beside pooled blocks, a gate per element."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ t[p + "q"].T, eps) * t[p + "q.norm"]).reshape(T, H, d)
    k = (rms(h @ t[p + "k"].T, eps) * t[p + "k.norm"]).reshape(T, G, d)
    v = (h @ t[p + "v"].T).reshape(T, G, e)
    q, k = rotate(q, positions, m["rot"], True), rotate(k, positions, m["rot"], True)
    o = attend(q, k, v, m["scale"], m["mask"]["size"], pool=m["mask"]["pool"]).reshape(T, -1)
    return element_gate(o, h, t[p + "g"]) @ t[p + "o"].T


def biased_attention(h, t, p, m, eps):
    """Values are the raw keys; heads brought to unit root mean square, no rotation, a learned bias per distance, a
    sink, a gate per head."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    raw = (h @ t[p + "k"].T).reshape(T, G, d)
    q, k = rms((h @ t[p + "q"].T).reshape(T, H, d), eps), rms(raw, eps)
    o = attend(q, k, raw, m["scale"], m["mask"]["size"], sink=t[p + "sink"], rel=t[p + "rel"], bias_max=m["bias_max"])
    o = o * torch.sigmoid(h @ t[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ t[p + "o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------

def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_ff(h, t, p):
    return gelu_tanh(h @ t[p + "up"].T + t[p + "up.b"]) @ t[p + "down"].T + t[p + "down.b"]


# ---- the model ---------------------------------------------------------------------------------------------------

def forward(config, tensors, tokens, dtype=torch.float64, taps=None):
    """Logits [T, vocab] of one sequence.  ``taps``: a list that receives the stream after every layer."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    positions = torch.arange(len(tokens))
    x = t["embed"][torch.tensor(tokens)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        h = stream_norm(x, t[p + "norm1"], eps)
        if kind == "parallel":
            y = side_by_side(h, t, p + "mix.", m, eps, positions)
        elif kind == "attention":
            y = pooled_attention(h, t, p + "mix.", m, eps, positions)
        else:
            y = biased_attention(h, t, p + "mix.", m, eps)
        x = x + y * t[p + "ls1"]
        if layer.get("mlp") is not None:
            x = x + dense_ff(stream_norm(x, t[p + "norm2"], eps), t, p + "mlp.") * t[p + "ls2"]
        if taps is not None:
            taps.append(x.clone())
    return stream_norm(x, t["final.norm"], eps) @ t["head"].T


def greedy(config, tensors, prompt, n_new, dtype=torch.float64):
    """The prompt's continuation by ``n_new`` tokens, each the arg-max of the logits at the last position."""
    tokens, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(torch.argmax(forward(config, tensors, tokens, dtype)[-1]))
        tokens.append(nxt)
        out.append(nxt)
    return out
