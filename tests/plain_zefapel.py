"""A plain, slow restatement of the Zefapel decoder, one function per mechanism.

Written from the design's equations for the tests only; it shares no code with the package. Everything runs in the
dtype of the tensors it is given (float64 in the tests). Notation: x is the residual stream [T, C]; h a sublayer's
squashed input; positions count from 0.

  squash      y = tanh(a x) * g + b                                 (no mean, no variance)
  embedding   x = scale * E[token]
  layer       x <- x + ls1 * mixer(squash1(x));  x <- x + ls2 * ff(squash2(x))
  output      logits = W_head . squash_final(x)

Mixers: ``mlstm`` (matrix memory with exponential input gates and a running maximum), ``gla`` (linear attention with a
decay per key channel), ``latent_attention`` (keys and values from one low-rank row per token beside one rotated key
part that all heads share; a layer may read an earlier layer's rows).
Feed-forward: a gated dense layer, or routed experts within groups, some of which return their input, beside a shared
expert behind a sigmoid.
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

def squash(x, w, name):
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def log_sigmoid(z):
    return -(torch.log1p(torch.exp(-z.abs())) + torch.clamp(-z, min=0.0))


# ---------------------------------------------------------------------------
# recurrent mixers: one token after the other
# ---------------------------------------------------------------------------

def mlstm_gates(h, w, p, cap):
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    return i, f


def mlstm_scan(q, k, v, i, f, state=None):
    """q, k [T, H, N], v [T, H, P], i, f [T, H] (log gates) -> o [T, H, P] and the final (S, n, m)."""
    T, H, N = q.shape
    P = v.shape[-1]
    if state is None:
        state = (q.new_zeros(H, N, P), q.new_zeros(H, N), q.new_zeros(H))
    S, n, m = state
    out = q.new_zeros(T, H, P)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hnp,hn->hp", S, q[t]) / den[:, None]
    return out, (S, n, m)


def mlstm(h, w, p, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, N) * N ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, N)
    v = (h @ w[p + "v"].T).view(T, H, P)
    i, f = mlstm_gates(h, w, p, m["gate_cap"])
    o, _ = mlstm_scan(q, k, v, i, f)
    o = rms(o, eps).reshape(T, H * P) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def gla_log_decay(h, w, p, tau):
    return log_sigmoid((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]) / tau


def gla_scan(q, k, v, alpha, S=None):
    """q, k, alpha [T, H, N], v [T, H, P] -> o [T, H, P] and the final S."""
    T, H, N = q.shape
    if S is None:
        S = q.new_zeros(H, N, v.shape[-1])
    out = q.new_zeros(T, H, v.shape[-1])
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hnp,hn->hp", S, q[t])
    return out, S


def gla(h, w, p, m, eps):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, N) * N ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, N)
    v = (h @ w[p + "v"].T).view(T, H, P)
    alpha = torch.exp(gla_log_decay(h, w, p, m["tau"])).view(T, H, N)
    o, _ = gla_scan(q, k, v, alpha)
    o = (rms(o, eps) * w[p + "norm"]).reshape(T, H * P) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------

def rotation(rot):
    """Frequencies (a list of floats) and the factor of cosine and sine."""
    dims, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s is None:
        return freq, 1.0
    where = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(where(s["fast"])), 0)
    hi = min(math.ceil(where(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, positions, rot):
    """x [T, heads, dims]: neighbours (2i, 2i + 1) turned by position * f_i, the result times the factor."""
    freq, factor = rotation(rot)
    a = positions.to(x.dtype)[:, None] * torch.tensor(freq, dtype=torch.float64).to(x.dtype)[None, :]
    c, s = (factor * torch.cos(a))[:, None, :], (factor * torch.sin(a))[:, None, :]
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * c - v * s
    out[..., 1::2] = v * c + u * s
    return out


def latent_rows(h, w, p, m, eps):
    """The row a token leaves in the cache: c [T, R] and the rotated key part [T, rot]."""
    R = m["kv_rank"]
    d = h @ w[p + "dkv"].T
    c = rms(d[:, :R], eps) * w[p + "dkv.norm"]
    return c, rotate_pairs(d[:, None, R:], torch.arange(h.shape[0]), m["rot"])[:, 0]


def softmax_mix(q, k, v, scale):
    """q, k [T, H, D], v [T, H, P] -> [T, H, P], causal, one query after the other."""
    T, H, _ = q.shape
    out = q.new_zeros(T, H, v.shape[-1])
    for i in range(T):
        s = torch.einsum("jhd,hd->hj", k[:i + 1], q[i]) * scale
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhp->hp", e / e.sum(-1, keepdim=True), v[:i + 1])
    return out


def latent_attention(h, w, p, m, eps, rows):
    T, H, D, E, P = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = rows
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).view(T, H, D + E)
    q = torch.cat([q[..., :D], rotate_pairs(q[..., D:], torch.arange(T), m["rot"])], dim=-1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, D), kr[:, None, :].expand(T, H, E)], dim=-1)
    v = (c @ w[p + "uv"].T).view(T, H, P)
    o = softmax_mix(q, k, v, m["scale"]).reshape(T, H * P) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------

def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, p):
    return torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def choose(z, correction, top, groups):
    """z [n] logits of one token -> (chosen indices, their weights). ``groups`` None or {count, keep}."""
    s = torch.softmax(z, dim=-1)
    c = s + correction
    if groups is not None:
        size = z.shape[0] // groups["count"]
        best = c.view(groups["count"], size).max(dim=-1).values
        keep = torch.topk(best, groups["keep"]).indices.tolist()
        for g in range(groups["count"]):
            if g not in keep:
                c = c.clone()
                c[g * size:(g + 1) * size] = -math.inf
    idx = torch.topk(c, top).indices
    return idx.tolist(), s[idx]


def routed_ff(h, w, p, mlp):
    r = mlp["router"]
    E = r["experts"]
    z = h @ w[p + "router"].T
    rows = []
    for t in range(h.shape[0]):
        idx, weight = choose(z[t], w[p + "correction"], r["top"], r.get("groups"))
        acc = torch.zeros_like(h[t])
        for e, a in zip(idx, weight):
            acc = acc + a * (expert(h[t], w, f"{p}e{e}.") if e < E else h[t])
        rows.append(acc)
    out = torch.stack(rows)
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return out


# ---------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------

def forward(cfg, w, ids, keep_layers=False):
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids)] * cfg["embedding"]["scale"]
    left = {}  # layer -> the rows its cache holds
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = squash(x, w, p + "norm1")
        if layer["type"] == "mlstm":
            y = mlstm(h, w, p + "mix.", m, eps)
        elif layer["type"] == "gla":
            y = gla(h, w, p + "mix.", m, eps)
        elif layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                left[i] = latent_rows(h, w, p + "mix.", m, eps)
            y = latent_attention(h, w, p + "mix.", m, eps, left[i if src is None else src])
        else:
            raise ValueError(layer["type"])
        x = x + w[p + "ls1"] * y
        mlp = layer["mlp"]
        if mlp is not None:
            h = squash(x, w, p + "norm2")
            y = dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(h, w, p + "mlp.", mlp)
            x = x + w[p + "ls2"] * y
        after.append(x)
    logits = squash(x, w, "final.norm") @ w["head"].T
    return (logits, torch.stack(after)) if keep_layers else logits
