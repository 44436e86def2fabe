"""Plain, slow implementation of the Lanilorn decoder for the tests.

Whole sequences, no cache, one function per mechanism, torch on the CPU in 64-bit.  It shares
no code with the package under test: it reads config.json and the safetensors file with its
own few lines and computes every layer with dense masks and loops over tokens.

The design in this file's notation (rows are tokens, h: the normed input of a sublayer, p: a position):

    norm       N(x; w) = x / sqrt(mean x^2 + eps) * w
    streams    X = (x_1 .. x_s), every one the scaled embedding row at the start; a sublayer f with its
               norm N, its column scale l and its tensors a [s], M [s, s], c [s]:
                   y = l * f(N(sum_r a_r x_r));   x_t <- sum_r M_rt x_r + c_t y   for all t at once
               (every layer: the mixer, then the feed-forward if there is one; the model's output
               reads sum_r x_r)
    attention  q = W_q h, k = W_k h, v = k;  then q <- N(q; w_q) and k <- N(k; w_k), each over all its
               heads at once;  the first `dims` columns of every head turn by YaRN angles, pairs half a
               rotation apart;  s_ij = q_i . k_j * scale for 0 <= i - j < size;  the weights are
               e^s / (sum e^s + e^sink) with one sink per query head;  head a reads key/value head
               a // (heads / kv_heads);  times sigmoid(W_g h)[a];  then W_o
    difference every query head a has two queries and every key/value head two keys (`dim` wide, side by
    attention  side), one value;  q_m <- q_m (1 + coef ln(floor((p + 1) / every) + 1));  softmax over all
               j <= i of q_m . k_m * scale, m = 1, 2, gives o_1 and o_2;  o = o_1 - lam o_2 with
               lam = exp(lq1 . lk1) - exp(lq2 . lk2) + diff;  o <- o / sqrt(mean o^2 + eps) (1 - diff);
               times sigmoid(W_g h)[a];  then W_o
    gated      per head: q = W_q h dim^-1/2, k = W_k h, v = W_v h;  a = sigmoid(W_a2 W_a1 h + b)^(1/tau)
    linear     per key row;  S <- diag(a) S + k v^T;  o = S^T q;  o <- N(o; w) per head;  times
    attention  silu(W_g h);  then W_o
    dense      W_down relu(W_up h)^2
    output     logits = E N(sum_r x_r; w_final) * logit_scale with the embedding table E
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
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


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


def yarn_frequencies(rot):
    """(frequencies [dims / 2], factor on cos and sin)."""
    dims, base, scaling = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freq, 1.0

    def dim_at(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(dim_at(scaling["fast"])), 0)
    hi = min(math.ceil(dim_at(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, rot, positions=None):
    """x [n, heads, dim]; row i sits at position i unless `positions` says where."""
    if not rot or not rot["dims"]:
        return x
    half = int(rot["dims"]) // 2
    freq, magnitude = yarn_frequencies(rot)
    out = x.clone()
    for row in range(x.shape[0]):
        p = row if positions is None else positions[row]
        for i, f in enumerate(freq):
            c, s = magnitude * math.cos(p * f), magnitude * math.sin(p * f)
            u, v = x[row, :, i], x[row, :, i + half]
            out[row, :, i] = u * c - v * s
            out[row, :, i + half] = v * c + u * s
    return out


def causal_mask(n):
    i = torch.arange(n)
    return i[None, :] <= i[:, None]


def window_mask(n, size):
    back = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    return (back >= 0) & (back < size)


def sink_attention(q, k, v, mask, scale, sink):
    """q [n, heads, dim], k [n, kv_heads, dim], v [n, kv_heads, vdim], sink [heads] or None."""
    n, heads, _ = q.shape
    group = heads // k.shape[1]
    out = torch.zeros(n, heads, v.shape[-1], dtype=F64)
    for a in range(heads):
        s = ((q[:, a] @ k[:, a // group].T) * scale).masked_fill(~mask, -math.inf)
        if sink is not None:            # one more column that has no key and no value
            s = torch.cat([s, sink[a].expand(n, 1)], dim=1)
        weights = torch.softmax(s, dim=-1)[:, :mask.shape[1]]
        out[:, a] = weights @ v[:, a // group]
    return out


def head_gate(out, h, w_gate):
    """out [n, heads, vdim] times one sigmoid per token and head."""
    return out * torch.sigmoid(h @ w_gate.T)[:, :, None]


def attention(h, w, prefix, m, eps):
    n = h.shape[0]
    heads, kv_heads, dim = m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w[prefix + "q"].T, h @ w[prefix + "k"].T
    v = k.view(n, kv_heads, dim)
    q = rms_norm(q, w[prefix + "q.norm"], eps).view(n, heads, dim)
    k = rms_norm(k, w[prefix + "k.norm"], eps).view(n, kv_heads, dim)
    q, k = rotate(q, m.get("rot")), rotate(k, m.get("rot"))
    mask = window_mask(n, int(m["mask"]["size"])) if m.get("mask") else causal_mask(n)
    out = sink_attention(q, k, v, mask, float(m["scale"]), w[prefix + "sink"])
    return head_gate(out, h, w[prefix + "g"]).reshape(n, -1) @ w[prefix + "o"].T


def query_temperature(n, temperature):
    """[n]: the factor on the query at every position."""
    if not temperature:
        return torch.ones(n, dtype=F64)
    return torch.tensor([1 + temperature["coef"] * math.log(math.floor((p + 1) / temperature["every"]) + 1)
                         for p in range(n)], dtype=F64)


def difference(o1, o2, lam, diff, eps):
    """o1, o2 [n, heads, vdim]."""
    return unit_rms(o1 - lam * o2, eps) * (1 - diff)


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return math.exp(float(lq1 @ lk1)) - math.exp(float(lq2 @ lk2)) + diff


def difference_attention(h, w, prefix, m, eps):
    n = h.shape[0]
    heads, kv_heads, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[prefix + "q"].T).view(n, heads, 2, dim) * query_temperature(n, m.get("q_temp"))[:, None, None, None]
    k = (h @ w[prefix + "k"].T).view(n, kv_heads, 2, dim)
    v = (h @ w[prefix + "v"].T).view(n, kv_heads, vdim)
    o = [sink_attention(q[:, :, i], k[:, :, i], v, causal_mask(n), float(m["scale"]), None) for i in range(2)]
    lam = difference_weight(w[prefix + "lq1"], w[prefix + "lk1"], w[prefix + "lq2"], w[prefix + "lk2"],
                            float(m["diff"]))
    out = difference(o[0], o[1], lam, float(m["diff"]), eps)
    return head_gate(out, h, w[prefix + "g"]).reshape(n, -1) @ w[prefix + "o"].T


def key_decays(h, w, prefix, tau):
    z = (h @ w[prefix + "a1"].T) @ w[prefix + "a2"].T + w[prefix + "a2.b"]
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def decayed_recurrence(q, k, v, a, state=None):
    """q, k, a [n, heads, dim], v [n, heads, vdim] -> o [n, heads, vdim]; token by token."""
    n, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[-1], dtype=F64) if state is None else state
    out = torch.zeros(n, heads, v.shape[-1], dtype=F64)
    for t in range(n):
        s = a[t][:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (s * q[t][:, :, None]).sum(1)
    return out


def gated_linear_attention(h, w, prefix, m, eps):
    n = h.shape[0]
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[prefix + "q"].T).view(n, heads, dim) * dim ** -0.5
    k = (h @ w[prefix + "k"].T).view(n, heads, dim)
    v = (h @ w[prefix + "v"].T).view(n, heads, vdim)
    a = key_decays(h, w, prefix, float(m["tau"])).view(n, heads, dim)
    o = rms_norm(decayed_recurrence(q, k, v, a), w[prefix + "norm"], eps).reshape(n, -1)
    return (o * torch.nn.functional.silu(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def dense(h, w, prefix):
    return torch.relu(h @ w[prefix + "up"].T) ** 2 @ w[prefix + "down"].T


MIXERS = {"attention": attention, "attention_2": difference_attention, "gla": gated_linear_attention}


# ------------------------------------------------------------------------------- model
def sublayer(streams, w, prefix, q, eps, f):
    u = gather_streams(streams, w[f"{prefix}hc{q}.in"])
    y = f(rms_norm(u, w[f"{prefix}norm{q}"], eps)) * w[f"{prefix}ls{q}"]
    return spread_streams(streams, w[f"{prefix}hc{q}.mix"], w[f"{prefix}hc{q}.out"], y)


def forward(config, w, ids, layer_outputs=None):
    """Logits [len(ids), vocab] in 64-bit.  `layer_outputs`: a list that receives the sum of the
    streams after every layer."""
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.tensor(ids)] * float(config["embedding"]["scale"])
    streams = [x.clone() for _ in range(int(config["streams"]))]
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}."
        mixer = MIXERS[layer["type"]]
        streams = sublayer(streams, w, p, 1, eps, lambda h: mixer(h, w, p + "mix.", layer["mixer"], eps))
        if layer.get("mlp") is not None:
            streams = sublayer(streams, w, p, 2, eps, lambda h: dense(h, w, p + "mlp."))
        if layer_outputs is not None:
            layer_outputs.append(sum(streams))
    return rms_norm(sum(streams), w["final.norm"], eps) @ w["embed"].T * float(config["logit_scale"])


def logits_for(model_dir, ids):
    config, w = load(model_dir)
    return forward(config, w, list(ids)).numpy()
