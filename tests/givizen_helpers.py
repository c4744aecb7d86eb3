"""Shared by the Givizen tests: small configurations, model folders, comparisons.

The configurations differ from one another in every size and constant, and no two sizes of a model coincide by accident:
key and value heads of different sizes, one kv head and several, groups of one query head and of many, head counts that are
no power of two, windows below, at and above a page, one layer without a window, limits that differ between a layer's
experts and its shared expert, one and several experts a token, a layer without a shared expert, a layer without a
feed-forward, no temperature, no cap of the logits, and one model with nothing a multiple of 4 or 8.

  ga  width 64, vocab 211: attention 4/2 x (16, 24) window 20, temperature 0.7 every 8 + 6 experts of 40 top 2, shared 72
      | attention_2 3/1 x (24, 16) window 33 cap 5, temperature 0.4 every 24 + 3 experts of 16 top 1, shared 24
      | attention_2 2/2 x (40, 12) window 1 cap 2 + no feed-forward | attention 6/3 x (8, 8) window 64 + 4 experts top 4
  gb  width 96, vocab 302 (sizes that tensor-core kernels take): attention 8/2 x 32 window 65, every 64
      + 5 experts of 64 top 3, shared 128 | attention_2 5/5 x 48 window 130 cap 9, every 50 + 9 experts of 72 top 1, shared 64
      | attention 18/1 x 16 window 128 + 4 experts of 80 top 2, no shared | attention_2 2/1 x 64 all keys, cap 15 + none
  gc  width 50, vocab 97 (nothing a multiple of 4 or 8): attention 3/1 x (7, 5) window 11 + 3 experts of 9 top 3, shared 7
      | attention_2 2/1 x (9, 13) window 70 cap 3 + 5 experts of 11 top 2, no shared | attention 5/5 x (6, 7) all keys
"""

from __future__ import annotations

import torch

import plain_givizen as plain


def _layer(kind, heads, kv_heads, dim, vdim, scale, window, temp=None, softcap=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if softcap is not None:
        m["softcap"] = softcap
    return {"type": kind, "mixer": m, "mlp": mlp}


def _moe(experts, top, ff, limit, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


CONFIGS = {
    "ga": {"architecture": "Givizen", "vocab": 211, "width": 64, "norm": {"eps": 1e-4}, "embedding": {"scale": 2.0},
           "logit_softcap": 12.0, "layers": [
               _layer("attention", 4, 2, 16, 24, 0.6, 20, (0.7, 8), None, _moe(6, 2, 40, 1.0, (72, 2.5))),
               _layer("attention_2", 3, 1, 24, 16, 0.5, 33, (0.4, 24), 5.0, _moe(3, 1, 16, 0.7, (24, 0.4))),
               _layer("attention_2", 2, 2, 40, 12, 0.3, 1, None, 2.0, None),
               _layer("attention", 6, 3, 8, 8, 0.9, 64, (1.5, 1), None, _moe(4, 4, 24, 3.0, (16, 1.0)))]},
    "gb": {"architecture": "Givizen", "vocab": 302, "width": 96, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
           "logit_softcap": 20.0, "layers": [
               _layer("attention", 8, 2, 32, 32, 0.35, 65, (0.5, 64), None, _moe(5, 3, 64, 1.5, (128, 0.8))),
               _layer("attention_2", 5, 5, 48, 48, 0.3, 130, (0.3, 50), 9.0, _moe(9, 1, 72, 0.5, (64, 2.0))),
               _layer("attention", 18, 1, 16, 16, 0.5, 128, (0.2, 100), None, _moe(4, 2, 80, 7.0)),
               _layer("attention_2", 2, 1, 64, 64, 0.25, None, (0.6, 33), 15.0, None)]},
    "gc": {"architecture": "Givizen", "vocab": 97, "width": 50, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.7}, "layers": [
               _layer("attention", 3, 1, 7, 5, 0.8, 11, (0.9, 5), None, _moe(3, 3, 9, 0.6, (7, 0.9))),
               _layer("attention_2", 2, 1, 9, 13, 0.7, 70, (0.5, 7), 3.0, _moe(5, 2, 11, 1.2)),
               _layer("attention", 5, 5, 6, 7, 1.0, None, None, None, _moe(2, 1, 21, 2.0, (13, 0.3)))]},
}
SEEDS = {"ga": 31, "gb": 32, "gc": 33}


def config(name: str):
    from kernel_rush_kawk_b200 import GivizenConfig

    return GivizenConfig.from_dict(CONFIGS[name])


def write_folder(folder, name: str):
    """Random weights, shaped so that every mechanism carries weight in the logits: gates and routers with logits of order
    one, sinks of the size of the scores, experts' inputs that reach their limits, a head whose logits feel their cap."""
    from kernel_rush_kawk_b200 import write_model_folder
    from kernel_rush_kawk_b200.config.registry import get_architecture
    from kernel_rush_kawk_b200.engine.model import expected_tensors

    cfg = config(name)
    names = expected_tensors(get_architecture(cfg.architecture).plan(cfg))
    scale = {}
    for n in names:
        if n.endswith((".gate", ".up")):
            scale[n] = 2.0
        elif n.endswith(".shared.down"):
            scale[n] = 2.0
        elif n.endswith((".mix.g", ".router")):
            scale[n] = 3.0
        elif n.endswith(".sink"):
            scale[n] = 25.0
        elif n == "embed":
            scale[n] = 10.0
        elif n == "head":
            scale[n] = 6.0
        elif n.endswith((".norm1", ".norm2")) or n == "final.norm":
            scale[n] = 3.0
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
    """32-bit: every row within the tolerance. bfloat16: a token whose best router logits lie closer than the rounding of
    its input may take another expert than the 64-bit implementation does; its feed-forward's output, which the norm behind
    it brings to full size, is then another one, and the rows that see it feel that. So five rows in six are held to the
    tolerance and the rest to ten times it: a fault of a mechanism shows in nearly every row."""
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    s = spread(got, ref)
    worst = int(s.argmax())
    if dtype == "float32":
        assert s.max().item() <= TOL[dtype], f"{what}: row {worst} differs by {s.max().item():.3e} of the logits' spread (allowed {TOL[dtype]:.0e})"
        return
    over = int((s > TOL[dtype]).sum())
    assert over <= max(1, s.numel() // 6), f"{what}: {over} of {s.numel()} rows differ by more than {TOL[dtype]:.0e}; worst row {worst}: {s.max().item():.3e}"
    assert s.max().item() <= 10 * TOL[dtype], f"{what}: row {worst} differs by {s.max().item():.3e} of the logits' spread"
