"""A plain, slow implementation of the Lovapel decoder, one function per mechanism, written from the design's
equations and sharing no code with the package.  Everything is torch on the CPU in the dtype of the weights it is
handed (float64 for an oracle).

The design.  x = E[token].  A layer norms both sides of each branch,
    x += n1b(attn(n1(x)));  x += n2b(ff(n2(x)))          n(y) = (y - mean) / sqrt(mean((y - mean)^2) + eps) * w
(no second line when the layer has no feed-forward), and a span of the layers is run several times with the same
weights, each pass with keys and values of its own.
  attention   grouped heads without biases; all query rows of a token are divided by ONE root mean square and multiplied
              by a weight per row, and so are all its key rows; then the first `dims` values of every query and key head
              turn, value i with value i + dims / 2, by p * base^(-2i / dims); scores times a constant; a key is seen while
              0 <= i - j < size; the softmax's denominator also holds exp(sink_h); Wo.
  dense       Wd (gelu(Wg h) * (Wu h)), gelu(z) = z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))).
  experts     s = softmax(Wr h) over experts and identity experts (the last ones, whose output is h); c = s + correction;
              equal groups of neighbours, a group is worth its largest c, only the best groups' members stand for choice;
              the `top` largest c are taken with weights s / (sum of the taken s + 1e-20); an expert is
              Wd (silu(Wg h) * (Wu h)), and a shared one of the same form is added for every token.
Logits: z = logit_scale * E n(x), then cap * tanh(z / cap)."""
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
        elif info["dtype"] == "I32":
            t = torch.from_numpy(np.frombuffer(raw, dtype="<i4").copy())
        else:
            raise ValueError(info["dtype"])
        out[name] = t.reshape(info["shape"])
    return out


# ---------------------------------------------------------------------------------------------- small pieces

def layer_norm(x, w, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x * x * x)))


def rotate_halves(x, pos, dims, base):
    """x [T, heads, D]: value i with value i + dims / 2, i < dims / 2, by pos * base^(-2i / dims); the angle is taken in
    x's own precision (in 32-bit, at position 300, it is off by some hundred-thousandths of a radian)."""
    if not dims:
        return x
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    f = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / dims)
    a = pos.to(x.dtype)[:, None, None] * f.to(x.dtype)
    c, s = torch.cos(a), torch.sin(a)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def window_sink_attention(q, k, v, pos_q, pos_k, scale, sink, window=None):
    """q [Tq, heads, D], k [Tk, kv, D], v [Tk, kv, Dv]; head h reads key/value head h // (heads / kv); a key at j is seen
    from i iff 0 <= i - j (< window).  exp(sink_h) joins the denominator.  Returns [Tq, heads, Dv]."""
    tq, heads, _ = q.shape
    group = heads // k.shape[1]
    out = torch.zeros(tq, heads, v.shape[-1], dtype=q.dtype)
    d = pos_q[:, None] - pos_k[None, :]
    seen = (d >= 0) if window is None else (d >= 0) & (d < window)
    for h in range(heads):
        s = (q[:, h] @ k[:, h // group].T) * scale
        s = torch.where(seen, s, torch.full_like(s, -float("inf")))
        m = torch.maximum(s.max(dim=-1, keepdim=True).values, sink[h].to(q.dtype).reshape(1, 1))
        e = torch.exp(s - m)
        out[:, h] = (e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[h].to(q.dtype) - m))) @ v[:, h // group]
    return out


def route(z, correction, top, groups=1, keep=1):
    """Indices and weights of the chosen experts, largest choice score first (ties: the lower index).  `groups` equal
    groups of neighbours, of which `keep` stay."""
    s = torch.softmax(z, dim=-1)
    c = s + correction
    size = z.shape[-1] // groups
    ids, weights = [], []
    for row_s, row_c in zip(s, c):
        worth = [float(row_c[g * size:(g + 1) * size].max()) for g in range(groups)]
        best = sorted(range(groups), key=lambda g: (-worth[g], g))[:keep]
        open_ = [e for e in range(z.shape[-1]) if e // size in best]
        taken = sorted(open_, key=lambda e: (-float(row_c[e]), e))[:top]
        ids.append(taken)
        weights.append(row_s[taken] / (row_s[taken].sum() + 1e-20))
    return torch.tensor(ids), torch.stack(weights)


# ---------------------------------------------------------------------------------------------- branches

def attention_mixer(h, w, p, m, eps, pos, quant=no_quant):
    t = h.shape[0]
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(quant(h @ w(p + "q").T), w(p + "q.norm"), eps).view(t, heads, dim)
    k = rms_norm(quant(h @ w(p + "k").T), w(p + "k.norm"), eps).view(t, kv, dim)
    v = quant(h @ w(p + "v").T).view(t, kv, vdim)
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    q = quant(rotate_halves(q, pos, rot["dims"], rot["base"]))
    k = quant(rotate_halves(k, pos, rot["dims"], rot["base"]))
    o = window_sink_attention(q, k, v, pos, pos, m["scale"], w(p + "sink"), (m.get("mask") or {}).get("size"))
    return quant(o.reshape(t, heads * vdim)) @ w(p + "o").T


def gated_ff(h, w, p, act, quant=no_quant):
    return quant(act(h @ w(p + "gate").T) * (h @ w(p + "up").T)) @ w(p + "down").T


def expert_ff(h, w, p, mlp, quant=no_quant):
    r = mlp["router"]
    n, identity = r["experts"], r.get("identity") or 0
    g = r.get("groups") or {"count": 1, "keep": 1}
    ids, weights = route(h @ w(p + "router").T, w(p + "correction"), r["top"], g["count"], g["keep"])
    out = torch.zeros_like(h)
    for e in range(n + identity):
        y = h if e >= n else gated_ff(h, w, p + f"e{e}.", silu, quant)
        out = out + ((ids == e) * weights).sum(dim=-1, keepdim=True) * y
    if mlp.get("shared"):
        out = out + gated_ff(h, w, p + "shared.", silu, quant)
    return out


# ---------------------------------------------------------------------------------------------- the model

def layer_order(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + loop["times"] * list(range(loop["start"], loop["stop"])) + list(range(loop["stop"], n))


def forward(cfg, weights, tokens, dtype=torch.float64, quant=no_quant, layers_out=None):
    """Logits [T, vocab] of one whole sequence; `layers_out` (a list) receives the stream after every layer run."""
    def w(name):
        return weights[name].to(dtype)
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    pos = torch.arange(tokens.numel())
    x = w("embed")[tokens]
    for i in layer_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        h = quant(layer_norm(x, w(p + "norm1"), eps))
        x = x + layer_norm(attention_mixer(h, w, p + "mix.", layer["mixer"], eps, pos, quant), w(p + "norm1b"), eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = quant(layer_norm(x, w(p + "norm2"), eps))
            y = gated_ff(h, w, p + "mlp.", gelu_tanh, quant) if mlp["kind"] == "dense" else expert_ff(h, w, p + "mlp.", mlp, quant)
            x = x + layer_norm(y, w(p + "norm2b"), eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    z = quant(layer_norm(x, w("final.norm"), eps)) @ w("embed").T * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
