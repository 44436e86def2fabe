"""Plain, slow implementation of the Deginex decoder for the tests.

Whole sequences, no cache, one function per mechanism, torch on the CPU in 64-bit.  It shares
no code with the package under test: it reads config.json and the safetensors file with its
own few lines and computes every layer with dense masks and loops over tokens and experts.

The design in this file's notation (rows are tokens, h: the normed input of a sublayer):

    norm       N(x; w, b) = (x - mean x) / sqrt(mean (x - mean x)^2 + eps) * w + b
    streams    X = (x_1 .. x_s), every one the embedding row at the start; a sublayer f with its
               norm N and its tensors a [s], M [s, s], c [s]:
                   y = f(N(sum_r a_r x_r));   x_t <- sum_r M_rt x_r + c_t y   for all t at once
               (every layer: the mixer, then the feed-forward if there is one; the model's output
               reads sum_r x_r)
    loop       the layers start .. stop - 1 run `times` times in a row, then the rest follow
    attention  q, k, v = W h; every head of q and of k divided by sqrt(its mean square + eps);
               s_ij = q_i . k_j * scale, then softcap * tanh(s_ij / softcap), for the j <= i with
               i // size == j // size;  softmax;  query head a reads key/value head a // (heads /
               kv_heads);  the heads side by side times sigmoid(W_g h), column by column;  then W_o
    dense      W_down (silu(W_gate h) * (W_up h))
    experts    z = W_r h + b_r;  the `top` largest are chosen;  their weights are the softmax of z
               over the chosen alone;  each expert is a small dense feed-forward
    output     logits = E N(sum_r x_r; w_final, b_final) with the embedding table E
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import numpy as np
import torch

F64 = torch.float64


# ----------------------------------------------------------------------------- loading
def read_tensors(path):
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        b, e = meta["data_offsets"]
        chunk = raw[8 + n + b:8 + n + e]
        if meta["dtype"] == "BF16":
            bits = np.frombuffer(chunk, dtype="<u2").astype(np.uint32) << 16
            t = torch.from_numpy(bits.view(np.float32).copy())
        elif meta["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(chunk, dtype="<f4").copy())
        else:
            raise ValueError(meta["dtype"])
        out[name] = t.reshape(meta["shape"]).to(F64)
    return out


def load(model_dir):
    model_dir = Path(model_dir)
    config = json.loads((model_dir / "config.json").read_text())
    return config, read_tensors(model_dir / "model.safetensors")


# -------------------------------------------------------------------------- mechanisms
def layer_norm(x, w, b, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w + b


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def gather_streams(streams, a):
    """streams: list of [n, width]; a [s] -> sum_r a_r x_r."""
    u = torch.zeros_like(streams[0])
    for r, x in enumerate(streams):
        u = u + a[r] * x
    return u


def spread_streams(streams, mix, c, y):
    """x_t <- sum_r mix[r, t] x_r + c_t y, every new stream from the old ones."""
    out = []
    for t in range(len(streams)):
        x = c[t] * y
        for r, old in enumerate(streams):
            x = x + mix[r, t] * old
        out.append(x)
    return out


def chunk_mask(n, size):
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


def capped_scores(q, k, scale, softcap):
    """q [n, dim], k [m, dim] -> [n, m]."""
    return softcap * torch.tanh((q @ k.T) * scale / softcap)


def capped_attention(q, k, v, mask, scale, softcap):
    """q [n, heads, dim], k [n, kv_heads, dim], v [n, kv_heads, vdim] -> [n, heads, vdim]."""
    n, heads, _ = q.shape
    group = heads // k.shape[1]
    out = torch.zeros(n, heads, v.shape[-1], dtype=F64)
    for a in range(heads):
        s = capped_scores(q[:, a], k[:, a // group], scale, softcap)
        out[:, a] = torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1) @ v[:, a // group]
    return out


def attention(h, w, prefix, m, eps):
    n = h.shape[0]
    q = unit_rms((h @ w[prefix + "q"].T).view(n, m["heads"], m["dim"]), eps)
    k = unit_rms((h @ w[prefix + "k"].T).view(n, m["kv_heads"], m["dim"]), eps)
    v = (h @ w[prefix + "v"].T).view(n, m["kv_heads"], m["vdim"])
    out = capped_attention(q, k, v, chunk_mask(n, int(m["mask"]["size"])), float(m["scale"]), float(m["softcap"]))
    out = out.reshape(n, -1) * torch.sigmoid(h @ w[prefix + "g"].T)
    return out @ w[prefix + "o"].T


def dense(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def route(h, w, prefix, top):
    """(ids [n, top], weights [n, top])."""
    z = h @ w[prefix + "router"].T + w[prefix + "router.b"]
    chosen, ids = torch.topk(z, top, dim=-1)
    return ids, torch.softmax(chosen, dim=-1)


def experts(h, w, prefix, mlp):
    ids, weights = route(h, w, prefix, int(mlp["router"]["top"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(ids[t].tolist(), weights[t]):
            out[t] += g * dense(h[t:t + 1], w, f"{prefix}e{e}.")[0]
    return out


def feed_forward(h, w, prefix, mlp):
    return dense(h, w, prefix) if mlp["kind"] == "dense" else experts(h, w, prefix, mlp)


# ------------------------------------------------------------------------------- model
def run_order(config):
    count, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(count))
    start, stop = int(loop["start"]), int(loop["stop"])
    return list(range(start)) + list(range(start, stop)) * int(loop["times"]) + list(range(stop, count))


def sublayer(streams, w, prefix, q, eps, f):
    u = gather_streams(streams, w[f"{prefix}hc{q}.in"])
    y = f(layer_norm(u, w[f"{prefix}norm{q}"], w[f"{prefix}norm{q}.b"], eps))
    return spread_streams(streams, w[f"{prefix}hc{q}.mix"], w[f"{prefix}hc{q}.out"], y)


def forward(config, w, ids, layer_outputs=None):
    """Logits [len(ids), vocab] in 64-bit.  `layer_outputs`: a list that receives the sum of the
    streams after every layer run."""
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.tensor(ids)]
    streams = [x.clone() for _ in range(int(config["streams"]))]
    for index in run_order(config):
        layer, p = config["layers"][index], f"l{index}."
        if layer["type"] != "attention":
            raise ValueError(layer["type"])
        streams = sublayer(streams, w, p, 1, eps, lambda h: attention(h, w, p + "mix.", layer["mixer"], eps))
        if layer.get("mlp") is not None:
            streams = sublayer(streams, w, p, 2, eps, lambda h: feed_forward(h, w, p + "mlp.", layer["mlp"]))
        if layer_outputs is not None:
            layer_outputs.append(sum(streams))
    return layer_norm(sum(streams), w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T


def logits_for(model_dir, ids):
    config, w = load(model_dir)
    return forward(config, w, list(ids)).numpy()
