"""A plain, slow Lagulorn: whole sequences, no cache, explicit loops, one function per mechanism.

The oracle of the Lagulorn tests.  It shares no code with the package: it reads a model folder with its own
safetensors reader and computes every position from all tokens before it.  ``dtype`` is the arithmetic
(float64 in most tests).

Notation: T tokens, H query heads, G key heads, d query/key size of one map, e value size, S copies of the stream,
E experts, I identity experts.
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
        kind = info["dtype"]
        if kind == "BF16":
            bits = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            arr = bits.view(np.float32).astype(np.float64)
        elif kind == "F32":
            arr = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif kind == "I32":
            arr = np.frombuffer(raw, dtype="<i4").astype(np.int64)
        else:
            raise ValueError(f"{name}: dtype {kind}")
        tensors[name] = torch.from_numpy(arr.reshape(info["shape"]).copy())
    return config, tensors


# ---- small pieces ---------------------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def unit_rms(x, eps):
    """x divided by its root mean square, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    """The stream's norm: its weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


# ---- lightning attention --------------------------------------------------------------------------

def decaying_state(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, e], decay: a number per head.  S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.
    Returns (o [T, H, e], the last state [H, d, e]); ``state`` is S before the first token (zeros)."""
    T, H, d = q.shape
    e = v.shape[-1]
    out = torch.zeros((T, H, e), dtype=q.dtype)
    last = torch.zeros((H, d, e), dtype=q.dtype)
    for h in range(H):
        S = torch.zeros((d, e), dtype=q.dtype) if state is None else state[h].clone()
        for i in range(T):
            S = decay[h] * S + torch.outer(k[i, h], v[i, h])
            out[i, h] = S.T @ q[i, h]
        last[h] = S
    return out, last


def lightning_mixer(h, t, prefix, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ t[prefix + "q"].T).reshape(T, H, d)
    k = silu(h @ t[prefix + "k"].T).reshape(T, H, d)
    v = silu(h @ t[prefix + "v"].T).reshape(T, H, e)
    o, _ = decaying_state(q, k, v, m["decay"])
    y = unit_rms(o.reshape(T, H * e), eps) * t[prefix + "norm"]              # all heads in one norm
    return (y * sigmoid(h @ t[prefix + "g"].T)) @ t[prefix + "o"].T


# ---- differential attention -----------------------------------------------------------------------

def windowed_attention(q, k, v, scale, window):
    """One map: q [T, H, d], k [T, G, d], v [T, G, e]; query head h reads key head h // (H / G); position i sees the
    keys j with 0 <= i - j < window (None: all up to itself)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros((T, H, v.shape[-1]), dtype=q.dtype)
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            s = (k[lo:i + 1, h // per] @ q[i, h]) * scale
            w = torch.exp(s - s.max())
            out[i, h] = (w @ v[lo:i + 1, h // per]) / w.sum()
    return out


def map_balance(t, prefix, diff):
    """lambda, the weight of the second map: one number for the layer."""
    return (math.exp(float((t[prefix + "lq1"] * t[prefix + "lk1"]).sum()))
            - math.exp(float((t[prefix + "lq2"] * t[prefix + "lk2"]).sum())) + diff)


def difference_of_maps(a1, a2, balance, diff, eps):
    """(a1 - lambda a2), every head divided by its root mean square, times 1 - diff."""
    return unit_rms(a1 - balance * a2, eps) * (1.0 - diff)


def attention_mixer(h, t, prefix, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ t[prefix + "q"].T).reshape(T, H, 2, d), eps) * t[prefix + "q.norm"]
    k = unit_rms((h @ t[prefix + "k"].T).reshape(T, G, 2, d), eps) * t[prefix + "k.norm"]
    v = (h @ t[prefix + "v"].T).reshape(T, G, e)
    window = m["mask"]["size"] if m.get("mask") else None
    a1 = windowed_attention(q[:, :, 0], k[:, :, 0], v, m["scale"], window)
    a2 = windowed_attention(q[:, :, 1], k[:, :, 1], v, m["scale"], window)
    o = difference_of_maps(a1, a2, map_balance(t, prefix, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * e) @ t[prefix + "o"].T


# ---- feed-forward ---------------------------------------------------------------------------------

def dense(h, t, prefix):
    return gelu_erf(h @ t[prefix + "up"].T) @ t[prefix + "down"].T


def clamped_unit(g, u, limit):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(h, t, prefix, limit):
    return clamped_unit(h @ t[prefix + "gate"].T, h @ t[prefix + "up"].T, limit) @ t[prefix + "down"].T


def routing(h, router_weight, correction, top, groups):
    """(chosen [T, top], weights [T, top]): softmax scores over all outputs; choice scores are scores + correction;
    only members of the ``keep`` groups with the largest choice scores can be chosen; the weights are the scores."""
    z = h @ router_weight.T
    z = torch.exp(z - z.max(dim=-1, keepdim=True).values)
    s = z / z.sum(dim=-1, keepdim=True)
    chosen, weights = [], []
    for i in range(h.shape[0]):
        c = (s[i] + correction).tolist()
        allowed = range(len(c))
        if groups is not None:
            size = len(c) // groups["count"]
            best = [max(c[g * size:(g + 1) * size]) for g in range(groups["count"])]
            kept = sorted(range(groups["count"]), key=lambda g: (-best[g], g))[:groups["keep"]]
            allowed = [e for g in kept for e in range(g * size, (g + 1) * size)]
        picked = sorted(allowed, key=lambda e: (-c[e], e))[:top]
        chosen.append(picked)
        weights.append(s[i][picked])
    return torch.tensor(chosen), torch.stack(weights)


def mixture_of_experts(h, t, prefix, mlp):
    r = mlp["router"]
    chosen, weights = routing(h, t[prefix + "router"], t[prefix + "correction"], r["top"], r.get("groups"))
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        for e, w in zip(chosen[i].tolist(), weights[i]):
            y = h[i] if e >= r["experts"] else expert(h[i:i + 1], t, f"{prefix}e{e}.", mlp["expert"]["limit"])[0]
            out[i] += w * y
    return out


def feed_forward(h, t, prefix, mlp):
    return dense(h, t, prefix) if mlp["kind"] == "dense" else mixture_of_experts(h, t, prefix, mlp)


# ---- the layer arrangement ------------------------------------------------------------------------

def read_copies(streams, weights):
    """u = sum_s weights[s] x_s of the copies [S, T, width]."""
    return torch.einsum("s,stw->tw", weights, streams)


def write_copies(streams, mix, out, y):
    """All copies at once from the old ones: x_t <- sum_s mix[s, t] x_s + out[t] y."""
    return torch.einsum("sr,stw->rtw", mix, streams) + out[:, None, None] * y[None]


def sublayer(streams, t, layer_prefix, q, eps, factor, run):
    """One sub-layer (q = 1: mixer, 2: feed-forward) between the copies of the stream [S, T, width]."""
    hc = f"{layer_prefix}hc{q}."
    if hc + "in" not in t:                          # a stream of one copy: the plain residual sum
        return streams + factor * run(layer_norm(streams[0], t[f"{layer_prefix}norm{q}"], eps))[None]
    h = layer_norm(read_copies(streams, t[hc + "in"]), t[f"{layer_prefix}norm{q}"], eps)
    return write_copies(streams, t[hc + "mix"], factor * t[hc + "out"], run(h))


def owner_of(config, i):
    """The layer whose tensors layer ``i`` uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def forward(config, t, tokens, dtype=torch.float64, taps=None):
    """Logits [T, vocab] of a whole sequence.  ``taps``, a list, receives the sum of the streams after every layer."""
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in t.items()}
    eps, factor = config["norm"]["eps"], config["residual_mult"]
    x = t["embed"][torch.tensor(list(tokens))] * config["embedding"]["scale"]
    streams = x[None].repeat(config.get("streams") or 1, 1, 1)
    for i, layer in enumerate(config["layers"]):
        lp, m = f"l{owner_of(config, i)}.", layer["mixer"]
        mixer = lightning_mixer if layer["type"] == "lightning" else attention_mixer
        streams = sublayer(streams, t, lp, 1, eps, factor, lambda h: mixer(h, t, lp + "mix.", m, eps))
        if layer.get("mlp") is not None:
            streams = sublayer(streams, t, lp, 2, eps, factor, lambda h: feed_forward(h, t, lp + "mlp.", layer["mlp"]))
        if taps is not None:
            taps.append(streams.sum(dim=0))
    return layer_norm(streams.sum(dim=0), t["final.norm"], eps) @ t["head"].T


def greedy(config, t, prompt, n_new, dtype=torch.float64):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(config, t, tokens, dtype)[-1].argmax()))
    return tokens[len(prompt):]
