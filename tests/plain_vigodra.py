"""A plain, slow implementation of the Vigodra decoder, one function per mechanism, written from the design's equations
and sharing no code with the package.  Everything is torch on the CPU in the dtype it is asked for (float64 for an
oracle); attention is a full score matrix and a latent attention is written out with its keys and values per head.

The design.  X_0 = embed[tok] * s.  Layer i reads the stream x itself and norms the sum (post-norm):
    x <- n1(alpha x + mixer(x));   x <- n2(alpha x + ff(x))      n(z) = (z - mean) / sqrt(var + eps) * w + b
(no second line when the layer has no feed-forward); that result is X_(i+1), and what goes on is the depth average
    x <- sum_(j <= i + 1) a_i[j] X_j.
Mixers:
  attention         q, k, v = projections with biases, each channel through a short causal filter over time; q and k
                    RMS-normed over the WHOLE projection; score q.k * scale + rel[bucket(i - j), h] for keys inside a
                    window or among the first kept positions; softmax with exp(sink_h) in the denominator; Wo + bias.
  latent_attention  keys and values are projections of one small normed latent per token plus one rotated key part
                    shared by the heads; queries are [plain | rotated] per head, rotation in halves; window; softmax;
                    the joined heads times sigmoid(Wg h), one gate per value; Wo.  A layer may use the latent and the
                    rotated key part of an earlier layer instead of making its own.
Feed-forward: g = min(Wg h, L), u = clamp(Wu h, -L, L), y = Wd (g sigmoid(1.702 g) (u + 1)).
Output: the model's norm, then the head matrix."""
from __future__ import annotations

import json
import math
import os

import torch


def no_quant(x):
    return x


def bf16_quant(x):
    """Rounds to bfloat16 and back: what the engine's bfloat16 path does to an activation it stores."""
    return x.to(torch.bfloat16).to(x.dtype)


def load_config(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def load_weights(model_dir):
    """Reads model.safetensors with this file's own reader: 8 bytes of length, a JSON header, raw little-endian data."""
    import numpy as np
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        n = int.from_bytes(f.read(8), "little")
        header = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw = bytes(data[lo:hi])
        if info["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(raw, dtype="<f4").copy())
        elif info["dtype"] == "BF16":
            t = (torch.from_numpy(np.frombuffer(raw, dtype="<u2").astype(np.int32).copy()) << 16).view(torch.float32)
        else:
            raise ValueError(info["dtype"])
        out[name] = t.reshape(info["shape"])
    return out


# ---------------------------------------------------------------------------------------------- small pieces

def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def depth_average(stages, a):
    """What goes on after a layer: the weighted sum of the embedding output and every layer's result so far."""
    return sum(a[j] * s for j, s in enumerate(stages))


def short_conv(x, taps):
    """y[t, c] = sum_j taps[c, j] x[t - (n - 1) + j, c], zeros before the start."""
    n = taps.shape[1]
    pad = torch.cat([x.new_zeros(n - 1, x.shape[1]), x], dim=0)
    return sum(pad[j: j + x.shape[0]] * taps[:, j] for j in range(n))


def distance_bucket(n, buckets, far):
    """Bucket of the distance n >= 0: one each below buckets / 2, logarithmic from there to `far`, the last beyond."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (buckets - half)))


def distance_bias(rel, t, far):
    """[H, T, T]: rel[bucket(i - j), h] for j <= i (0 elsewhere)."""
    rows = torch.tensor([distance_bucket(n, rel.shape[0], far) for n in range(t)], dtype=torch.long)
    d = (torch.arange(t)[:, None] - torch.arange(t)[None, :]).clamp(min=0)
    return rel[rows[d]].permute(2, 0, 1)


def visible(t, window=None, keep_first=0):
    i, j = torch.arange(t)[:, None], torch.arange(t)[None, :]
    seen = j <= i
    if window is not None:
        seen = seen & ((i - j < window) | (j < keep_first))
    return seen


def masked_softmax_attention(scores, v, seen, sink=None):
    """scores [H, T, T] (query, key), v [H, T, vd], seen [T, T]; with `sink` [H] the denominator also holds exp(sink_h)."""
    scores = scores.masked_fill(~seen, float("-inf"))
    top = scores.amax(dim=-1, keepdim=True)
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(scores - top)
    den = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - top)
    return torch.einsum("hij,hjd->ihd", e / den, v)


def rotate_halves(x, positions, dims, base):
    """x [T, heads, d]: the first `dims` values of every head turn, value i with i + dims / 2."""
    f = float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    half = dims // 2
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def clamped_glu(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


# ---------------------------------------------------------------------------------------------- mixers

def attention(m, w, p, h, eps, quant):
    heads, kvh, kd, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    t = h.shape[0]

    def part(name):
        return short_conv(quant(h @ w[p + name].T) + w[p + name + ".b"], w[p + name + ".conv"])
    q, k, v = part("q"), part("k"), quant(part("v"))
    q = quant(rms_unit(q, eps) * w[p + "q.norm"]).view(t, heads, kd)
    k = quant(rms_unit(k, eps) * w[p + "k.norm"]).view(t, kvh, kd)
    per = heads // kvh
    k, v = k.repeat_interleave(per, dim=1), v.view(t, kvh, vd).repeat_interleave(per, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] + distance_bias(w[p + "rel"], t, m["bias_max"])
    mask = m.get("mask") or {}
    o = masked_softmax_attention(scores, v.transpose(0, 1), visible(t, mask.get("size"), mask.get("keep_first", 0)), w[p + "sink"])
    return quant(o.reshape(t, heads * vd)) @ w[p + "o"].T + w[p + "o.b"]


def latent_parts(m, w, p, h, positions, eps, quant):
    """What a latent attention caches per token: the normed latent and the rotated key part."""
    rank = m["kv_rank"]
    dkv = quant(h @ w[p + "dkv"].T)
    c = quant(rms_unit(dkv[:, :rank], eps) * w[p + "dkv.norm"])
    kr = quant(rotate_halves(dkv[:, None, rank:], positions, m["rot"]["dims"], m["rot"]["base"])[:, 0])
    return c, kr


def latent_attention(m, w, p, h, positions, eps, quant, shared=None):
    heads, nd, rd, vd = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    t = h.shape[0]
    c, kr = shared if shared is not None else latent_parts(m, w, p, h, positions, eps, quant)
    q = quant(h @ w[p + "q"].T).view(t, heads, nd + rd)
    q_rot = quant(rotate_halves(q[..., nd:], positions, m["rot"]["dims"], m["rot"]["base"]))
    k_plain = (c @ w[p + "uk"].T).view(t, heads, nd)
    v = (c @ w[p + "uv"].T).view(t, heads, vd)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :nd], k_plain) + torch.einsum("ihd,jd->hij", q_rot, kr)) * m["scale"]
    o = masked_softmax_attention(scores, v.transpose(0, 1), visible(t, (m.get("mask") or {}).get("size")))
    gate = torch.sigmoid(quant(h @ w[p + "g"].T))
    return quant(o.reshape(t, heads * vd) * gate) @ w[p + "o"].T, (c, kr)


def feed_forward(mlp, w, p, h, quant):
    y = clamped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, mlp["limit"])
    return quant(y) @ w[p + "down"].T


# ---------------------------------------------------------------------------------------------- the model

def forward(cfg, weights, tokens, dtype=torch.float64, quant=no_quant, streams=None):
    """Logits [T, vocab] of one sequence.  `streams`: a list that receives the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    tok = torch.as_tensor(list(tokens), dtype=torch.long)
    positions = torch.arange(len(tok))
    x = w["embed"][tok] * cfg["embedding"]["scale"]
    stages, kept = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        m, l = layer["mixer"], f"l{i}."
        if layer["type"] == "attention":
            y = attention(m, w, l + "mix.", quant(x), eps, quant)
        elif layer["type"] == "latent_attention":
            y, kept[i] = latent_attention(m, w, l + "mix.", quant(x), positions, eps, quant,
                                          shared=kept[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            raise ValueError(layer["type"])
        x = layer_norm(alpha * x + y, w[l + "norm1"], w[l + "norm1.b"], eps)
        if layer.get("mlp") is not None:
            x = layer_norm(alpha * x + feed_forward(layer["mlp"], w, l + "mlp.", quant(x), quant),
                           w[l + "norm2"], w[l + "norm2.b"], eps)
        stages.append(x)
        x = depth_average(stages, w[l + "dwa"])
        if streams is not None:
            streams.append(x.clone())
    return quant(layer_norm(x, w["final.norm"], w["final.norm.b"], eps)) @ w["head"].T
