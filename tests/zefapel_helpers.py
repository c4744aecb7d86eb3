"""Shared by the Zefapel tests: small configurations, model folders, comparisons.

The configurations differ from one another in every size and constant, and no two sizes of a model coincide by accident:
key and value heads of different sizes, ranks below and above the heads' sizes, one head and several, layers that share
an earlier layer's rows (with other head counts and sizes than its own), experts with and without groups, identity
experts and a shared expert, layers without a feed-forward, frequencies with and without scaling (and a ramp of no
width), and one model with nothing a multiple of 4 or 8.

  za  width 64, vocab 211: gla 3 x (20, 12) rank 5 tau 7 + 5 experts and 3 identity top 3, 2 of 4 groups, shared 24
      | latent 3 x (16 + 8, 24) rank 32 q 40 + dense 72 | mlstm 2 x (24, 40) cap 4, no feed-forward
      | latent 5 x (12 + 8, 16) reads layer 1, q 24 + 6 experts top 2, no groups, no shared
      | mlstm 1 x (8, 72) cap 9 + dense 40
  zb  width 96, vocab 302 (sizes that tensor-core kernels take): mlstm 2 x (32, 48) cap 12 + dense 128
      | latent 2 x (48 + 16, 64) rank 80 q 56 | gla 2 x (48, 64) rank 12 tau 3 + 7 experts and 1 identity top 8, shared 40
      | latent 4 x (16 + 16, 32) reads layer 1 + dense 96 | latent 18 x (32 + 32, 16) rank 48 (one layer's rows of its own)
      | gla 1 x (128, 112) rank 3 tau 16, mlstm 1 x (144, 80)
  zc  width 50, vocab 97 (nothing a multiple of 4 or 8): latent 3 x (7 + 2, 5) rank 9 q 11 + 3 experts and 3 identity top 1
      | mlstm 3 x (5, 7) cap 2.5 + dense 23 | gla 1 x (9, 13) rank 3 tau 0.5 + 5 experts top 5 in 1 group, shared 11
"""

from __future__ import annotations

import torch

import plain_zefapel as plain


def _memory(kind, heads, dim, vdim, **k):
    return {"type": kind, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, **k}}


def _latent(heads, dim, rot, vdim, rank, q_rank, scale, base, scaling=None, kv_from=None):
    r = {"dims": rot, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale, "rot": r}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def _moe(experts, identity, top, ff, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _layers(*pairs):
    return [{**mixer, "mlp": mlp} for mixer, mlp in pairs]


_YARN_A, _YARN_B = (3.0, 40, 4.0, 1.0), (8.0, 512, 16.0, 2.0)
CONFIGS = {
    "za": {"architecture": "Zefapel", "vocab": 211, "width": 64, "norm": {"eps": 1e-4}, "embedding": {"scale": 2.0}, "layers": _layers(
        (_memory("gla", 3, 20, 12, tau=7.0), _moe(5, 3, 3, 40, (4, 2), 24)),
        (_latent(3, 16, 8, 24, 32, 40, 0.2, 100.0, _YARN_A), _dense(72)),
        (_memory("mlstm", 2, 24, 40, gate_cap=4.0), None),
        (_latent(5, 12, 8, 16, 32, 24, 0.3, 100.0, _YARN_A, kv_from=1), _moe(6, 0, 2, 16)),
        (_memory("mlstm", 1, 8, 72, gate_cap=9.0), _dense(40)))},
    "zb": {"architecture": "Zefapel", "vocab": 302, "width": 96, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "layers": _layers(
        (_memory("mlstm", 2, 32, 48, gate_cap=12.0), _dense(128)),
        (_latent(2, 48, 16, 64, 80, 56, 0.11, 5000.0, _YARN_B), None),
        (_memory("gla", 2, 48, 64, tau=3.0), _moe(7, 1, 8, 32, None, 40)),
        (_latent(4, 16, 16, 32, 80, 24, 0.25, 5000.0, _YARN_B, kv_from=1), _dense(96)),
        (_latent(18, 32, 32, 16, 48, 64, 0.15, 300.0), None),
        (_memory("gla", 1, 128, 112, tau=16.0), None),
        (_memory("mlstm", 1, 144, 80, gate_cap=15.0), _moe(4, 2, 2, 24, (3, 2))))},
    "zc": {"architecture": "Zefapel", "vocab": 97, "width": 50, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.7}, "layers": _layers(
        (_latent(3, 7, 2, 5, 9, 11, 0.4, 7.0, (2.0, 9, 1.0, 1.0)), _moe(3, 3, 1, 9)),
        (_memory("mlstm", 3, 5, 7, gate_cap=2.5), _dense(23)),
        (_memory("gla", 1, 9, 13, tau=0.5), _moe(5, 0, 5, 11, (1, 1), 11)))},
}
RANKS = {"za": {0: 5}, "zb": {2: 12, 5: 3}, "zc": {2: 3}}  # of the decays' small matrices
SEEDS = {"za": 21, "zb": 22, "zc": 23}


def config(name: str):
    from kernel_rush_kawk_b200 import ZefapelConfig

    cfg = ZefapelConfig.from_dict(CONFIGS[name])
    return cfg.with_tensor_shapes({f"l{i}.mix.a1": (rank,) for i, rank in RANKS[name].items()})


def write_folder(folder, name: str):
    """Random weights, shaped so that every mechanism carries weight in the logits: projections of std 0.08, queries and
    keys scaled up (a sharp softmax: a wrong key shows), gates, routers and decays with logits of order one, corrections
    that change choices and are negative as often as not."""
    from kernel_rush_kawk_b200 import write_model_folder
    from kernel_rush_kawk_b200.config.registry import get_architecture
    from kernel_rush_kawk_b200.engine.model import expected_tensors

    cfg = config(name)
    names = expected_tensors(get_architecture(cfg.architecture).plan(cfg))
    scale = {}
    for n in names:
        if n.endswith((".mix.q", ".mix.k", ".mix.uk", ".mix.uq", ".mix.dkv")):
            scale[n] = 2.5
        elif n.endswith((".mix.i", ".mix.f")):
            scale[n] = 2.0
        elif n.endswith((".mix.g", ".router", ".shared.sg", ".mix.a1", ".mix.a2")):
            scale[n] = 4.0
        elif n.endswith((".i.b", ".f.b", ".a2.b")):
            scale[n] = 12.0
        elif n.endswith(".mix.o"):
            scale[n] = 0.5
        elif n == "embed":
            scale[n] = 8.0
    return write_model_folder(folder, cfg, SEEDS[name], std=0.08, gain_std=0.1, scale=scale)


def prompts(name: str, lengths, seed=0):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist() for n in lengths]


_cache: dict = {}


def plain_logits(folder, ids) -> torch.Tensor:
    """float64 logits [T, vocab] of the plain implementation (cached per folder and sequence)."""
    key = (str(folder), tuple(ids))
    if key not in _cache:
        cfg, w = plain.read_folder(folder, torch.float64)
        _cache[key] = plain.forward(cfg, w, ids)
    return _cache[key]


def spread(got: torch.Tensor, ref: torch.Tensor) -> torch.Tensor:
    """Per row: root mean square of the difference with its mean taken off, over the reference's own spread."""
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    d = got - ref
    d = d - d.mean(dim=-1, keepdim=True)
    r = ref - ref.mean(dim=-1, keepdim=True)
    return d.pow(2).mean(dim=-1).sqrt() / r.pow(2).mean().sqrt()


TOL = {"float32": 5e-5, "bfloat16": 1e-1}


def assert_logits(got, ref, dtype: str, what: str) -> None:
    """32-bit: every row within the tolerance. bfloat16: a token whose best choice scores lie closer than the rounding of
    its input may take another expert than the 64-bit implementation does, and the rows after it feel that; so nineteen
    rows in twenty are held to the tolerance and the rest to five times it."""
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    s = spread(got, ref)
    worst = int(s.argmax())
    if dtype == "float32":
        assert s.max().item() <= TOL[dtype], f"{what}: row {worst} differs by {s.max().item():.3e} of the logits' spread (allowed {TOL[dtype]:.0e})"
        return
    over = int((s > TOL[dtype]).sum())
    assert over <= max(1, s.numel() // 20), f"{what}: {over} of {s.numel()} rows differ by more than {TOL[dtype]:.0e}; worst row {worst}: {s.max().item():.3e}"
    assert s.max().item() <= 5 * TOL[dtype], f"{what}: row {worst} differs by {s.max().item():.3e} of the logits' spread"
