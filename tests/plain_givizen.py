"""A plain, slow restatement of the Givizen decoder, one function per mechanism.

Written from the design's equations for the tests only; it shares no code with the package. Everything runs in the
dtype of the tensors it is given (float64 in the tests). Notation: x is the residual stream [T, C]; sublayers read x
itself; positions count from 0.

  rms         r(x) = x / sqrt(mean(x^2) + eps)
  embedding   x = scale * E[token]
  layer       x <- x + r(mixer(x)) * (1 + w1);  x <- x + r(ff(x)) * (1 + w2)
  output      z = W_head (r(x) * (1 + w_final));  logits = c * tanh(z / c)

Attention, both kinds: no rotation and no biases; q and k divided by their root mean square per head ("attention":
times a weight of the head's size), q times a temperature that grows with its position; the score may be capped
("attention_2"), then slope_h * distance is taken off; the query sees the last ``size`` positions, itself among them;
"attention" has one more learned term per head in the softmax's denominator, "attention_2" a sigmoid per head on its
output. Feed-forward: routed experts with clamped inputs, a token's weight for an expert multiplying the expert's
input, beside a shared expert.
"""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch


def read_folder(folder, dtype=torch.float64):
    from safetensors import safe_open

    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    w = {}
    for shard in sorted(folder.glob("*.safetensors")):
        with safe_open(str(shard), framework="pt", device="cpu") as f:
            for name in f.keys():
                t = f.get_tensor(name)
                w[name] = t.to(dtype) if t.dtype.is_floating_point else t
    return cfg, w


# ---------------------------------------------------------------------------
# small pieces
# ---------------------------------------------------------------------------

def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def cap(z, limit):
    return z if limit is None else limit * torch.tanh(z / limit)


def temperature(position, coef, every):
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1.0)


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


# ---------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------

def queries_and_keys(h, w, p, m, eps):
    """q [T, H, D] and k [T, G, D], normed per head, q times its temperature."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rms((h @ w[p + "q"].T).view(T, H, D), eps)
    k = rms((h @ w[p + "k"].T).view(T, G, D), eps)
    if p + "q.norm" in w:
        q, k = q * w[p + "q.norm"], k * w[p + "k.norm"]
    t = m.get("q_temp")
    if t is not None:
        factor = [temperature(i, t["coef"], t["every"]) for i in range(T)]
        q = q * torch.tensor(factor, dtype=torch.float64).to(q.dtype)[:, None, None]
    return q, k


def biased_window_softmax(q, k, v, scale, window, softcap=None, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, P] -> [T, H, P], one query and head after the other."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = q.new_zeros(T, H, v.shape[-1])
    for hd, slope in enumerate(slopes(H)):
        keys, values = k[:, hd // group], v[:, hd // group]
        for i in range(T):
            lo = 0 if window is None else max(0, i - window + 1)
            s = cap(keys[lo:i + 1] @ q[i, hd] * scale, softcap)
            s = s - slope * (i - torch.arange(lo, i + 1)).to(s.dtype)
            top = s.max() if sink is None else torch.maximum(s.max(), sink[hd])
            e = torch.exp(s - top)
            total = e.sum() + (0.0 if sink is None else torch.exp(sink[hd] - top))
            out[i, hd] = (e / total) @ values[lo:i + 1]
    return out


def attention(kind, h, w, p, m, eps):
    T, H, G, P = h.shape[0], m["heads"], m["kv_heads"], m["vdim"]
    q, k = queries_and_keys(h, w, p, m, eps)
    v = (h @ w[p + "v"].T).view(T, G, P)
    window = m["mask"]["size"] if m.get("mask") is not None else None
    if kind == "attention":
        o = biased_window_softmax(q, k, v, m["scale"], window, sink=w[p + "sink"])
    else:
        o = biased_window_softmax(q, k, v, m["scale"], window, softcap=m["softcap"])
        o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * P) @ w[p + "o"].T


# ---------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------

def expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def choose(z, top):
    """z [n] logits of one token -> (chosen indices, their weights)."""
    s = torch.sigmoid(z)
    idx = torch.topk(s, top).indices
    return idx.tolist(), s[idx]


def routed_ff(h, w, p, mlp):
    z = h @ w[p + "router"].T
    rows = []
    for t in range(h.shape[0]):
        acc = torch.zeros_like(h[t])
        for e, a in zip(*choose(z[t], mlp["router"]["top"])):
            acc = acc + expert(a * h[t], w, f"{p}e{e}.", mlp["expert"]["limit"])
        rows.append(acc)
    out = torch.stack(rows)
    if mlp.get("shared") is not None:
        out = out + expert(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def forward(cfg, w, ids, keep_layers=False):
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids)] * cfg["embedding"]["scale"]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + norm(attention(layer["type"], x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + norm(routed_ff(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], eps)
        after.append(x)
    logits = cap(norm(x, w["final.norm"], eps) @ w["head"].T, cfg.get("logit_softcap"))
    return (logits, torch.stack(after)) if keep_layers else logits
