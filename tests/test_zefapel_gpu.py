"""Zefapel on the GPU: every mechanism's kernels alone against the plain functions of tests/plain_zefapel.py, then the
model through the engine: whole prompts, portions, single tokens, unequal batches, reused slots and pages, keys far away,
long decoding, greedy generation and trace replay."""

import io
import json
from types import SimpleNamespace

import pytest
import torch

import plain_zefapel as plain
from zefapel_helpers import CONFIGS, assert_logits, plain_logits, prompts, write_folder

pytestmark = pytest.mark.gpu

DTYPES = (torch.float32, torch.bfloat16)
PART_TOL = {torch.float32: 3e-5, torch.bfloat16: 5e-2}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("zefapel_gpu")
    return {name: write_folder(root / name, name) for name in CONFIGS}


def runtime(dtype):
    from kernel_rush_kawk_b200.csrc import load_kernels
    from kernel_rush_kawk_b200.engine.model import Runtime

    return Runtime(torch.device("cuda:0"), dtype, load_kernels())


def rand(shape, seed, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return torch.randn(shape, generator=g) * scale


def context(rt, slots, starts, q_lens, cache):
    from kernel_rush_kawk_b200.engine.step import BatchMeta, StepContext

    meta = BatchMeta(sum(q_lens), len(slots), 0, rt.device)
    meta.fill(slots, starts, [[0] * n for n in q_lens], [])
    return StepContext(rt.ops, meta, cache)


def close(got, ref, dtype, what, loosen=1.0):
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    err = (got - ref).abs().max().item()
    tol = loosen * PART_TOL[dtype] * ref.abs().max().item()
    assert err <= tol, f"{what}: max |d| = {err:.3e} > {tol:.3e}; first bad row {int(((got - ref).abs() > tol).any(-1).nonzero()[0])}"


def as_path(w, dtype):
    """The tensors as the path stores them, and the same values in float64 for the plain functions."""
    stored = {k: v.to(torch.bfloat16) for k, v in w.items()}  # checkpoints hold bfloat16
    return {k: v.to(dtype).cuda() for k, v in stored.items()}, {k: v.double() for k, v in stored.items()}


def run_part(part, rt, h, pieces, dtype, prior=(), reader=None):
    """One sequence through a mixer part, cut into ``pieces``; ``prior``: sequences that used (and gave back) the slot and
    its pages before. ``reader``: a second part that reads the first one's cache; its result is returned."""
    from kernel_rush_kawk_b200.cache import SequenceCache

    needs = [part.cache_need()] + ([("from", 0)] if reader is not None else [])
    cache = SequenceCache(needs, 2048, 1, 2048, rt.device, dtype)
    for seq, cuts in list(prior) + [(h, pieces)]:
        slot = cache.alloc()
        got, start = [], 0
        for n in cuts:
            cache.reserve(slot, start + n)
            cache.sync()
            ctx = context(rt, [slot], [start], [n], cache)
            rows = seq[start:start + n].to(dtype).cuda()
            out = part.forward(ctx, rows, cache.view(0))
            if reader is not None:
                out = reader.forward(ctx, rows, cache.view(1))
            got.append(out)
            cache.advance(slot, n)
            start += n
        cache.free(slot)
    rt.ops.check()
    return torch.cat(got)


def run_batch(part, rt, seqs, splits, dtype):
    """Unequal sequences side by side: a prompt each, then single tokens while the shorter ones end."""
    from kernel_rush_kawk_b200.cache import SequenceCache

    cache = SequenceCache([part.cache_need()], 8192, len(seqs), 2048, rt.device, dtype)
    slots = [cache.alloc() for _ in seqs]
    got = [[] for _ in seqs]

    def step(which, counts):
        starts = [cache.length[slots[i]] for i in which]
        for i, n in zip(which, counts):
            cache.reserve(slots[i], cache.length[slots[i]] + n)
        cache.sync()
        ctx = context(rt, [slots[i] for i in which], starts, counts, cache)
        out = part.forward(ctx, torch.cat([seqs[i][a:a + n] for i, a, n in zip(which, starts, counts)]).to(dtype).cuda(), cache.view(0))
        row = 0
        for i, n in zip(which, counts):
            got[i].append(out[row:row + n])
            cache.advance(slots[i], n)
            row += n

    step(list(range(len(seqs))), splits)
    while True:
        live = [i for i in range(len(seqs)) if cache.length[slots[i]] < len(seqs[i])]
        if not live:
            break
        step(live, [1] * len(live))
    rt.ops.check()
    return [torch.cat(g) for g in got]


# ----------------------------------------------------------------------------------------------
# each mechanism alone
# ----------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [64, 50, 33, 1536])
def test_tanh_norm_folds_a_scaled_output(dtype, size):
    """The first norm only reads; the second folds the sublayer's output times the first one's vector; the last one
    (without a vector) leaves none on the stream."""
    from kernel_rush_kawk_b200.parts import Stream, TanhNorm

    rt = runtime(dtype)
    ctx = SimpleNamespace(ops=rt.ops)
    x, y = rand((7, size), 1, 3.0), rand((7, size), 2, 2.0).to(dtype)
    norms, ws = [], []
    for q in range(3):
        w = {"weight": 1 + 0.3 * rand((size,), 10 + q), "alpha": torch.tensor(0.4 + 0.3 * q), "b": rand((size,), 20 + q, 0.5)}
        if q < 2:
            w["scale"] = 1 + 0.7 * rand((size,), 30 + q)
        part = TanhNorm({"size": size, "branch_scale": q < 2})
        assert {k: tuple(s.shape) for k, s in part.tensor_specs().items()} == {k: tuple(v.shape) for k, v in w.items()}
        dev, ref = as_path(w, dtype)
        part.bind(dev, rt)
        norms.append(part)
        ws.append(ref)
    want = lambda s, w: plain.squash(s, {"n": w["weight"], "n.alpha": w["alpha"], "n.b": w["b"]}, "n")
    stream = Stream(x.cuda())
    s = x.double()
    for q in range(3):
        close(norms[q].forward(ctx, stream).tensor(), want(s, ws[q]), dtype, f"norm {q}")
        assert stream.branch is None and (stream.fold is None) == (q == 2)
        assert (stream.x.double().cpu() - s).abs().max() < 1e-5  # 32-bit whatever the path
        if q < 2:
            stream.branch = y.cuda()
            s = s + ws[q]["scale"] * y.double()


MEMORY_SHAPES = [  # hidden, heads, dim, vdim
    (64, 3, 20, 12), (48, 2, 32, 80), (50, 1, 9, 13), (96, 2, 48, 64), (64, 1, 130, 24), (32, 4, 16, 144), (40, 1, 128, 128),
    (32, 2, 64, 256),
]


def gla_part(shape, dtype, rt, rank=5, tau=7.0, decay_scale=3.0, seed=100):
    from kernel_rush_kawk_b200.parts import GatedLinearAttention

    C, H, N, P = shape
    part = GatedLinearAttention({"hidden": C, "heads": H, "dim": N, "vdim": P, "rank": rank, "tau": tau, "eps": 1e-5})
    w = {k: rand((H * n, C), seed + i, C ** -0.5) for i, (k, n) in enumerate((("q", N), ("k", N), ("v", P), ("g", P)))}
    w.update({"o": rand((C, H * P), seed + 5, (H * P) ** -0.5), "a1": rand((rank, C), seed + 6, C ** -0.5),
              "a2": rand((H * N, rank), seed + 7, decay_scale), "a2.b": rand((H * N,), seed + 8, 2.0),
              "norm": 1 + 0.3 * rand((P,), seed + 9)})
    assert {k: tuple(s.shape) for k, s in part.tensor_specs().items()} == {k: tuple(v.shape) for k, v in w.items()}
    dev, ref = as_path(w, dtype)
    part.bind(dev, rt)
    return part, ref, {"heads": H, "dim": N, "vdim": P, "tau": tau}


def mlstm_part(shape, dtype, rt, cap=6.0, gate_scale=3.0, bias=(0.0, 0.0), seed=200):
    from kernel_rush_kawk_b200.parts import MatrixLSTM

    C, H, N, P = shape
    part = MatrixLSTM({"hidden": C, "heads": H, "dim": N, "vdim": P, "gate_cap": cap, "eps": 1e-5})
    w = {k: rand((H * n, C), seed + i, C ** -0.5) for i, (k, n) in enumerate((("q", N), ("k", N), ("v", P), ("g", P)))}
    w.update({"o": rand((C, H * P), seed + 5, (H * P) ** -0.5), "i": rand((H, C), seed + 6, gate_scale * C ** -0.5),
              "f": rand((H, C), seed + 7, gate_scale * C ** -0.5), "i.b": rand((H,), seed + 8) + bias[0],
              "f.b": rand((H,), seed + 9) + bias[1], "norm": 1 + 0.3 * rand((H * P,), seed + 10)})
    assert {k: tuple(s.shape) for k, s in part.tensor_specs().items()} == {k: tuple(v.shape) for k, v in w.items()}
    dev, ref = as_path(w, dtype)
    part.bind(dev, rt)
    return part, ref, {"heads": H, "dim": N, "vdim": P, "gate_cap": cap}


def memory_from_projections(kind, part, rt, ref, m, h, dtype, eps=1e-5):
    """The mechanism in 64-bit behind the projections as the path computes them (rounded to its dtype). A sum S^T q that
    nearly cancels is divided by its own size afterwards, so what the projections' rounding does to such a row says nothing
    about the scan; everything behind them is held to the tolerance."""
    proj = rt.ops.linear(h.to(dtype).cuda(), part._w_in).double().cpu()
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v, g, rest = torch.split(proj, [H * N, H * N, H * P, H * P, proj.shape[1] - 2 * H * (N + P)], dim=1)
    q, k, v = q.reshape(T, H, N) * N ** -0.5, k.reshape(T, H, N), v.reshape(T, H, P)
    if kind == "gla":
        z = rest[:, :ref["a1"].shape[0]] @ ref["a2"].T + ref["a2.b"]
        o, _ = plain.gla_scan(q, k, v, torch.exp(plain.log_sigmoid(z) / m["tau"]).view(T, H, N))
        o = (plain.rms(o, eps) * ref["norm"]).reshape(T, H * P) * plain.silu(g)
    else:
        cap = m["gate_cap"]
        z = cap * torch.tanh((rest[:, :2 * H] + torch.cat([ref["i.b"], ref["f.b"]])) / cap)
        o, _ = plain.mlstm_scan(q, k, v, z[:, :H], plain.log_sigmoid(z[:, H:]))
        o = plain.rms(o, eps).reshape(T, H * P) * ref["norm"] * torch.sigmoid(g)
    return o @ ref["o"].T


PIECES = ([230], [100, 2, 3, 64, 61], [180] + [1] * 50, [64, 64, 64, 38], [2] * 115)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MEMORY_SHAPES)
def test_gated_linear_attention_alone(dtype, shape):
    rt = runtime(dtype)
    part, ref, m = gla_part(shape, dtype, rt, rank=200 if shape[0] == 96 else 5, decay_scale=0.5 if shape[0] == 96 else 3.0)
    h = rand((230, shape[0]), 1, 1.5)
    want = memory_from_projections("gla", part, rt, ref, m, h, dtype)
    for pieces in PIECES:
        close(run_part(part, rt, h, pieces, dtype, prior=[(rand((90, shape[0]), 2), [90])]), want, dtype, f"gla {shape}, pieces {pieces[:4]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MEMORY_SHAPES)
def test_matrix_lstm_alone(dtype, shape):
    rt = runtime(dtype)
    part, ref, m = mlstm_part(shape, dtype, rt)
    h = rand((230, shape[0]), 1, 1.5)
    want = memory_from_projections("mlstm", part, rt, ref, m, h, dtype)
    for pieces in PIECES:
        close(run_part(part, rt, h, pieces, dtype, prior=[(rand((90, shape[0]), 2), [90])]), want, dtype, f"mlstm {shape}, pieces {pieces[:4]}",
              loosen=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tau, decay_scale", [(1.0, 40.0), (0.3, 10.0), (16.0, 0.2), (1000.0, 1.0)])
def test_decays_from_nothing_kept_to_everything_kept(dtype, tau, decay_scale):
    """Decays down to e^-100 a token (what is forgotten must not come back as an overflow's NaN) and up to nearly 1 (what
    is kept over hundreds of tokens must still be there)."""
    rt = runtime(dtype)
    shape = (64, 3, 48, 16)
    part, ref, m = gla_part(shape, dtype, rt, tau=tau, decay_scale=decay_scale)
    h = rand((400, shape[0]), 1, 1.5)
    want = memory_from_projections("gla", part, rt, ref, m, h, dtype)
    for pieces in ([400], [330] + [1] * 70):
        close(run_part(part, rt, h, pieces, dtype), want, dtype, f"tau {tau}, pieces {pieces[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap, bias", [(15.0, (0.0, 12.0)), (15.0, (-25.0, 0.0)), (15.0, (20.0, -10.0)), (30.0, (0.0, 20.0)), (1.0, (0.0, 0.0))])
def test_gates_at_their_ends(dtype, cap, bias):
    """Forget gates that keep everything, input gates that admit next to nothing (the maximum stays at its start and then
    falls), input gates near the cap with a fast decay, a wide cap and a narrow one."""
    rt = runtime(dtype)
    shape = (64, 2, 32, 48)
    part, ref, m = mlstm_part(shape, dtype, rt, cap=cap, bias=bias)
    h = rand((300, shape[0]), 1, 1.5)
    want = memory_from_projections("mlstm", part, rt, ref, m, h, dtype)
    for pieces in ([300], [64] * 4 + [44], [260] + [1] * 40):
        close(run_part(part, rt, h, pieces, dtype), want, dtype, f"cap {cap} bias {bias}, pieces {pieces[:3]}", loosen=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_early_token_still_shows_hundreds_of_tokens_later(dtype):
    """A token whose key is written loudly into a state that decays slowly: the last queries ask for it."""
    rt = runtime(dtype)
    shape = (64, 1, 32, 32)
    for make, kind in ((lambda: gla_part(shape, dtype, rt, tau=200.0, decay_scale=0.5), plain.gla),
                       (lambda: mlstm_part(shape, dtype, rt, cap=15.0, gate_scale=1.0, bias=(0.0, 14.0)), plain.mlstm)):
        part, ref, m = make()
        name = "gla" if kind is plain.gla else "mlstm"
        for place in (0, 63, 64, 127, 128, 255):
            h = rand((600, shape[0]), 3, 0.3)
            h[place] = rand((shape[0],), 4, 6.0)
            h[-3:] = h[place] * 0.5
            want = memory_from_projections(name, part, rt, ref, m, h, dtype)
            if dtype == torch.float32:
                close(want, kind(h.double(), ref, "", m, 1e-5), dtype, "the mechanism behind the path's projections", loosen=2.0)
            for pieces in ([600], [590] + [1] * 10):
                close(run_part(part, rt, h, pieces, dtype), want, dtype, f"token {place}, pieces {pieces[:2]}", loosen=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gla", "mlstm", "latent"])
def test_unequal_batches_against_each_alone(dtype, kind):
    rt = runtime(dtype)
    if kind == "latent":
        part, ref, m = latent_part(LATENT_SHAPES[1], dtype, rt)
        C = LATENT_SHAPES[1][0]
    else:
        part, ref, m = (gla_part if kind == "gla" else mlstm_part)((96, 2, 48, 64), dtype, rt)
        C = 96
    lengths = [150, 1, 64, 200, 65, 3]
    seqs = [rand((n, C), 40 + i, 1.2) for i, n in enumerate(lengths)]
    got = run_batch(part, rt, seqs, [140, 1, 63, 130, 64, 1], dtype)
    for i, s in enumerate(seqs):
        h = s.to(dtype).double()
        if kind == "latent":
            want = plain.latent_attention(h, ref, "", m, 1e-5, plain.latent_rows(h, ref, "", m, 1e-5))
        else:
            want = memory_from_projections(kind, part, rt, ref, m, s, dtype)
        close(got[i], want, dtype, f"{kind}, sequence {i} of the batch", loosen=2.0)


LATENT_SHAPES = [  # hidden, heads, dim, rot, vdim, kv rank, q rank
    (64, 3, 16, 8, 24, 32, 40), (96, 2, 48, 16, 64, 80, 56), (50, 3, 7, 2, 5, 9, 11), (64, 5, 12, 8, 16, 32, 24),
    (96, 18, 32, 32, 16, 48, 64), (64, 1, 64, 64, 128, 112, 32), (128, 16, 128, 64, 128, 512, 96), (64, 33, 16, 16, 32, 64, 16),
    (64, 2, 16, 8, 16, 600, 24),  # a latent wider than the tensor-core kernels take
]
ROT = {"base": 500.0, "scaling": {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 1.0}}


def latent_part(shape, dtype, rt, own=True, like=None, seed=300, loud=1.0, scaled=True):
    """``like``: another part's plain tensors, whose rows a part without rows of its own reads."""
    from kernel_rush_kawk_b200.parts import RotatedLatentAttention

    C, H, D, E, P, R, Q = shape
    scale = (D + E) ** -0.5
    part = RotatedLatentAttention({"hidden": C, "heads": H, "dim": D, "rot_dim": E, "vdim": P, "kv_rank": R, "q_rank": Q,
                                   "scale": scale, "rot_base": ROT["base"], "rot_scaling": ROT["scaling"] if scaled else None,
                                   "own_cache": own, "eps": 1e-5})
    w = {"dq": rand((Q, C), seed, C ** -0.5), "dq.norm": 1 + 0.3 * rand((Q,), seed + 1),
         "uq": rand((H * (D + E), Q), seed + 2, 1.6 * loud * Q ** -0.5), "uk": rand((H * D, R), seed + 3, 1.6 * R ** -0.5),
         "uv": rand((H * P, R), seed + 4, R ** -0.5), "g": rand((H * P, C), seed + 5, C ** -0.5),
         "o": rand((C, H * P), seed + 6, (H * P) ** -0.5)}
    if own:
        w.update({"dkv": rand((R + E, C), seed + 7, 1.3 * C ** -0.5), "dkv.norm": 1 + 0.3 * rand((R,), seed + 8)})
    assert {k: tuple(s.shape) for k, s in part.tensor_specs().items()} == {k: tuple(v.shape) for k, v in w.items()}
    dev, ref = as_path(w, dtype)
    part.bind(dev, rt)
    m = {"heads": H, "dim": D, "rot_dim": E, "vdim": P, "kv_rank": R, "q_rank": Q, "scale": scale,
         "rot": {"dims": E, "base": ROT["base"], "scaling": ROT["scaling"] if scaled else None}}
    return part, ref, m


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", LATENT_SHAPES)
def test_latent_attention_alone(dtype, shape):
    rt = runtime(dtype)
    part, ref, m = latent_part(shape, dtype, rt)
    T = 150
    h = rand((T, shape[0]), 1, 1.2)
    hd = h.to(dtype).double()
    want = plain.latent_attention(hd, ref, "", m, 1e-5, plain.latent_rows(hd, ref, "", m, 1e-5))
    for pieces in ([T], [63, 1, 2, 66, 18], [130] + [1] * 20, [2] * 75):
        close(run_part(part, rt, h, pieces, dtype, prior=[(rand((200, shape[0]), 2), [200])]), want, dtype, f"latent {shape}, pieces {pieces[:4]}")


@pytest.mark.parametrize("heads, rank, rot", [(16, 512, 64), (5, 64, 16), (33, 128, 32), (20, 272, 16), (3, 96, 32)])
@pytest.mark.parametrize("lengths", [[1, 64, 65, 500], [129], [2000] + [3] * 11])
def test_single_tokens_over_latent_rows_on_the_tensor_cores(heads, rank, rot, lengths):
    """The kernel against the general one (bfloat16, same rows): pages shared by more blocks than there are pages, sequences of
    very different length side by side, heads that do not fill a tile."""
    from kernel_rush_kawk_b200.cache import SequenceCache
    from kernel_rush_kawk_b200.parts import KVNeed

    rt = runtime(torch.bfloat16)
    W = rank + rot
    cache = SequenceCache([KVNeed(1, W, None, values=False)], 64 * 80, len(lengths), 4096, rt.device, torch.bfloat16)
    slots = [cache.alloc() for _ in lengths]
    for s, n in zip(slots, lengths):
        cache.reserve(s, n)
        cache.advance(s, n - 1)
    cache.sync()
    view = cache.view(0)
    view.k.copy_(rand(tuple(view.k.shape), 1).to(torch.bfloat16))
    batch = context(rt, slots, [n - 1 for n in lengths], [1] * len(lengths), cache).batch
    q = rand((len(lengths), heads * W), 2, 3.0 * W ** -0.5).to(torch.bfloat16).cuda()
    got, want = (torch.zeros((len(lengths), heads * rank), dtype=torch.bfloat16, device="cuda") for _ in range(2))
    assert rt.ops._latent_decode(q, heads, rank, W, 0.7, batch, view, got)
    rt.ops.sink_attention(q, 0, heads, W, rank, None, 0.7, None, batch, view, want, 0, 1.0)
    close(got, want, torch.bfloat16, f"{heads} heads, rank {rank}, lengths {lengths[:4]}", loosen=0.3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_over_another_layers_rows(dtype):
    """The reader has head counts, sizes and weights of its own; the rows are the other part's."""
    rt = runtime(dtype)
    for a, b in ((LATENT_SHAPES[0], (64, 5, 12, 8, 16, 32, 24)), (LATENT_SHAPES[1], (96, 4, 16, 16, 32, 80, 24))):
        owner, wa, ma = latent_part(a, dtype, rt)
        reader, wb, mb = latent_part(b, dtype, rt, own=False, seed=400)
        h = rand((140, a[0]), 1, 1.2)
        hd = h.to(dtype).double()
        want = plain.latent_attention(hd, wb, "", mb, 1e-5, plain.latent_rows(hd, wa, "", ma, 1e-5))
        for pieces in ([140], [64, 2, 74], [120] + [1] * 20):
            close(run_part(owner, rt, h, pieces, dtype, reader=reader), want, dtype, f"reader {b}, pieces {pieces[:3]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scaled", [True, False])
def test_latent_attention_finds_one_loud_key_wherever_it_sits(dtype, scaled):
    """One token's row points where the last queries look, so that one score stands out among hundreds: at the start, at
    page borders, just before the query; in a prompt and in single tokens (whose last key is the token itself)."""
    rt = runtime(dtype)
    shape = (64, 2, 32, 16, 32, 48, 32)
    part, ref, m = latent_part(shape, dtype, rt, loud=4.0, scaled=scaled)
    T = 700
    for place in (0, 1, 62, 63, 64, 65, 127, 128, 383, 384, 639, 698, 699):
        h = rand((T, shape[0]), 5, 0.2)
        loud = rand((shape[0],), 6, 3.0)
        h[place] = loud
        h[-2:] = loud
        hd = h.to(dtype).double()
        want = plain.latent_attention(hd, ref, "", m, 1e-5, plain.latent_rows(hd, ref, "", m, 1e-5))
        for pieces in ([T], [T - 5] + [1] * 5):
            close(run_part(part, rt, h, pieces, dtype), want, dtype, f"loud key {place}, pieces {pieces[:2]}")


MOE_SHAPES = [  # hidden, experts, identity, top, ff, (groups, keep), shared ff
    (64, 5, 3, 3, 40, (4, 2), 24), (96, 7, 1, 8, 32, (1, 1), 40), (50, 3, 3, 1, 9, (1, 1), None), (50, 5, 0, 5, 11, (1, 1), 11),
    (64, 11, 3, 2, 48, (2, 1), 64), (32, 4, 2, 2, 24, (3, 2), None), (32, 9, 0, 8, 1800, (3, 3), 8), (64, 2, 30, 4, 16, (8, 3), 16),
    # rows ordered by expert and multiplied in one launch: experts with more than a tile of rows and with none
    (96, 7, 1, 3, 72, (2, 1), 40), (192, 10, 5, 2, 80, (3, 1), 104), (136, 40, 8, 4, 264, (4, 2), None), (64, 70, 2, 2, 64, (6, 2), 8),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MOE_SHAPES)
@pytest.mark.parametrize("rows", [1, 5, 200, 777])
def test_routed_experts_with_identity_experts_alone(dtype, shape, rows):
    from kernel_rush_kawk_b200.parts import RoutedExperts

    rt = runtime(dtype)
    C, E, I, top, F, (count, keep), Fs = shape
    part = RoutedExperts({"hidden": C, "experts": E, "identity": I, "top": top, "intermediate": F, "activation": "relu2",
                          "gated": False, "scoring": "softmax_groups", "groups": count, "keep_groups": keep,
                          "shared_intermediate": Fs, "shared_gate": Fs is not None})
    w = {"router": rand((E + I, C), 1, 0.5), "correction": rand((E + I,), 2, 0.3)}
    for e in range(E):
        w.update({f"e{e}.up": rand((F, C), 11 + 2 * e, 0.3), f"e{e}.down": rand((C, F), 12 + 2 * e, 0.3)})
    if Fs is not None:
        w.update({"shared.up": rand((Fs, C), 4, 0.3), "shared.down": rand((C, Fs), 5, 0.3), "shared.sg": rand((1, C), 6, 0.5)})
    assert {k: tuple(s.shape) for k, s in part.tensor_specs().items()} == {k: tuple(v.shape) for k, v in w.items()}
    dev, ref = as_path(w, dtype)
    part.bind(dev, rt)
    h = rand((rows, C), 7, 1.5).to(dtype)
    mlp = {"router": {"experts": E, "top": top, "groups": {"count": count, "keep": keep}}, "shared": None if Fs is None else {"ff": Fs}}
    want = plain.routed_ff(h.double(), ref, "", mlp)
    for decode in (False, True):
        ctx = SimpleNamespace(ops=rt.ops, batch=SimpleNamespace(is_decode=decode))
        close(part.forward(ctx, h.cuda()), want, dtype, f"experts {shape}, {rows} rows, single-token step {decode}")


def test_grouped_products_where_experts_have_few_rows_many_or_none():
    rt = runtime(torch.bfloat16)
    for E, N, K, counts in ((5, 200, 72, [0, 300, 1, 0, 128]), (3, 64, 128, [129, 0, 0]), (40, 320, 96, [7 * (e % 3) for e in range(40)])):
        offsets = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
        rows = int(offsets[-1])
        a, w = rand((rows + 5, K), 1).to(torch.bfloat16), rand((E, N, K), 2, K ** -0.5).to(torch.bfloat16)
        for act in (-1, 5):
            out = torch.full((rows + 5, N), 7.0, dtype=torch.bfloat16, device="cuda")
            a_d, w_d, o_d = a.cuda(), w.cuda(), offsets.cuda()
            rt.ops._ok(rt.ops.moe.krk_grouped_gemm(out.data_ptr(), a_d.data_ptr(), w_d.data_ptr(), o_d.data_ptr(), rows + 5, E, N, K,
                                                   act, 0, 0, None, 0.0, 0.0, rt.ops.error.data_ptr(), rt.ops._stream()), "grouped product")
            want = torch.full((rows + 5, N), 7.0, dtype=torch.float64)
            for e in range(E):
                lo, hi = int(offsets[e]), int(offsets[e + 1])
                y = a[lo:hi].double() @ w[e].double().t()
                want[lo:hi] = torch.clamp(y, min=0.0) ** 2 if act == 5 else y
            close(out, want, torch.bfloat16, f"{E} experts, act {act}")  # rows beyond the last expert's stay as they were
    rt.ops.check()


def test_experts_are_ordered_stably():
    rt = runtime(torch.float32)
    g = torch.Generator().manual_seed(3)
    for rows, top, E in ((1, 2, 3), (700, 3, 11), (2048, 6, 64), (33, 1, 300)):
        experts = torch.randint(-1, E, (rows, top), generator=g, dtype=torch.int32)
        offsets = torch.empty(E + 1, dtype=torch.int32, device="cuda")
        place = torch.full((rows * top,), -5, dtype=torch.int32, device="cuda")
        d = experts.cuda()
        rt.ops._ok(rt.ops.moe.krk_moe_sort(offsets.data_ptr(), place.data_ptr(), d.data_ptr(), rows, top, E, rt.ops._stream()), "ordering")
        flat = experts.flatten()
        counts = torch.bincount(flat[flat >= 0].long(), minlength=E)
        assert offsets.tolist() == [0] + counts.cumsum(0).tolist()
        order = sorted((i for i in range(flat.numel()) if flat[i] >= 0), key=lambda i: (int(flat[i]), i))
        want = torch.full((flat.numel(),), -5, dtype=torch.int32)
        want[torch.tensor(order, dtype=torch.long)] = torch.arange(len(order), dtype=torch.int32)
        assert torch.equal(place.cpu(), want)


def test_routing_within_groups_by_hand():
    """Group scores are the largest choice score (not a sum), struck-out scores stay out although all are negative, weights
    are the softmax over every output, identity choices are handed through, ties take the lower index."""
    rt = runtime(torch.float32)
    z = torch.tensor([[2.0, -1.0, 1.2, 1.1, 0.3, 0.3], [0.0, 0.0, 0.0, 0.0, 0.0, 0.0]], device="cuda")
    corr = torch.tensor([-3.0, -3.0, -3.0, -3.0, -3.0, -3.0], device="cuda")
    experts, weights, _, passed = rt.ops.moe_route_softmax_groups(torch.eye(2, device="cuda"), z.t().contiguous(), corr, 2, 3, 1, 2)
    s = torch.softmax(z, dim=-1)
    assert experts.tolist() == [[0, 1], [0, 1]]  # the first group holds the largest score although the second has the larger sum
    assert torch.allclose(weights, s[:, :2], atol=1e-6) and torch.all(passed == 0)
    corr[4:] = 0.0
    experts, weights, _, passed = rt.ops.moe_route_softmax_groups(torch.eye(2, device="cuda"), z.t().contiguous(), corr, 2, 3, 1, 2)
    assert experts.tolist() == [[-1, -1], [-1, -1]] and torch.all(weights == 0)
    assert torch.allclose(passed, s[:, 4] + s[:, 5], atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
def test_squared_relu_without_a_gate(dtype):
    rt = runtime(dtype)
    z = rand((9, 200), 2, 1.5).to(dtype)
    close(rt.ops.act_rows(z.cuda(), "relu2"), torch.clamp(z.double(), min=0.0) ** 2, dtype, "squared relu")
    for rows, K, N in ((1, 64, 40), (8, 96, 4000), (13, 256, 24), (40, 64, 48), (3, 50, 21)):  # few rows: in the product's epilogue
        h, w = rand((rows, K), 3).to(dtype), rand((N, K), 4, K ** -0.5).to(dtype)
        want = torch.clamp(h.double() @ w.double().t(), min=0.0) ** 2
        close(rt.ops.up_act(h.cuda(), w.cuda(), "relu2"), want, dtype, f"squared relu of a product of {rows} rows")


# ----------------------------------------------------------------------------------------------
# the model through the engine
# ----------------------------------------------------------------------------------------------

def engine(folder, dtype, **kw):
    from kernel_rush_kawk_b200 import Engine

    args = dict(dtype=dtype, max_tokens=4096, max_slots=6, max_context=1024)
    args.update(kw)
    return Engine(folder, **args)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_portions_and_single_tokens_through_the_engine(folders, name, dtype):
    from kernel_rush_kawk_b200 import StepEntry

    eng = engine(folders[name], dtype, max_step_rows=170)  # longer steps are cut into passes
    ids = prompts(name, [260])[0]
    ref = plain_logits(folders[name], ids)
    for pieces in ([260], [130, 2, 3, 64, 61], [210] + [1] * 50):
        slot = eng.cache.alloc()
        got, start = [], 0
        for n in pieces:
            got.append(eng.step([StepEntry(slot, ids[start:start + n], list(range(n)))]).clone())
            start += n
        eng.cache.free(slot)
        assert_logits(torch.cat(got), ref, dtype, f"{name} {dtype}, pieces {pieces[:4]}")
    eng.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["za", "zb"])
def test_unequal_batches_reused_slots_and_long_decoding(folders, name, dtype):
    """Requests of unequal length start together and are decoded together while the shorter ones end; their slots and
    pages are then used again by others. Every row against the sequence run alone in the plain implementation."""
    from kernel_rush_kawk_b200 import StepEntry

    eng = engine(folders[name], dtype, max_slots=5)
    for round_ in range(2):
        lengths = [90, 1, 200, 37, 64] if round_ == 0 else [65, 130, 2]
        tails = [70, 0, 100, 20, 1] if round_ == 0 else [30, 60, 1]
        seqs = prompts(name, lengths, seed=5 + round_)
        slots = [eng.cache.alloc() for _ in seqs]
        heads = [len(ids) - t for ids, t in zip(seqs, tails)]
        first = eng.step([StepEntry(s, ids[:n], [n - 1]) for s, ids, n in zip(slots, seqs, heads)]).clone()
        for i, (ids, n) in enumerate(zip(seqs, heads)):
            assert_logits(first[i:i + 1], plain_logits(folders[name], ids)[n - 1:n], dtype, f"round {round_}, prompt {i}")
        got = {i: [] for i in range(len(seqs))}
        for t in range(max(tails)):
            live = [i for i in range(len(seqs)) if t < tails[i]]
            out = eng.step([StepEntry(slots[i], [seqs[i][heads[i] + t]], [0]) for i in live])
            for row, i in enumerate(live):
                got[i].append(out[row].clone())
            for i in range(len(seqs)):
                if t + 1 == tails[i]:
                    eng.cache.free(slots[i])
        for i, ids in enumerate(seqs):
            if tails[i] == 0:
                eng.cache.free(slots[i])
                continue
            assert_logits(torch.stack(got[i]), plain_logits(folders[name], ids)[heads[i]:], dtype, f"round {round_}, decoded sequence {i}")
        eng.cache.check()
        assert eng.cache.live == 0


def test_greedy_generation_through_the_engines_own_entry(folders):
    """Engine.generate (scheduler, captured single-token steps, selection kernel) against greedy decoding with the plain
    implementation; prompts of unequal length, one of a single token."""
    name = "za"
    eng = engine(folders[name], "float32", max_tokens=None)
    seqs = prompts(name, [33, 1, 80], seed=9)
    steps = list(eng.generate(seqs, 12))
    assert len(steps) == 12
    cfg, w = plain.read_folder(folders[name], torch.float64)
    for i, ids in enumerate(seqs):
        ids = list(ids)
        for t in range(12):
            logits = plain.forward(cfg, w, ids)[-1]
            best = torch.topk(logits, 2).values
            if best[0] - best[1] < 1e-4:  # too close to call in 32-bit: stop comparing this sequence
                break
            assert steps[t][i] == int(logits.argmax()), f"sequence {i}, new token {t}"
            ids.append(steps[t][i])


def test_trace_replay_serves_the_design(folders, tmp_path):
    """bin/trace_run's program on a small schedule: a batch of prompts, single tokens, a request that ends."""
    from kernel_rush_kawk_b200 import replay

    name = "zc"
    a, b = prompts(name, [70, 9], seed=4)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": a[:60], "want": [0, 59]}, {"id": "b", "tokens": b[:8], "want": [7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[60]], "want": [0]}, {"id": "b", "tokens": [b[8]], "want": []}], "end": ["b"]}]
    lines += [{"step": 2 + t, "entries": [{"id": "a", "tokens": [a[61 + t]], "want": [0]}], "end": ["a"] if t == 8 else []} for t in range(9)]
    out = io.StringIO()
    args = replay.build_parser().parse_args(["--model", str(folders[name]), "--dtype", "float32", "--out", str(tmp_path / "o"),
                                             "--max-tokens", "256"])
    assert replay.run(args, stdin=io.StringIO("\n".join(json.dumps(l) for l in lines) + "\n"), stdout=out) == 0
    assert out.getvalue().split() == [w for t in range(11) for w in ("done", str(t))]
    import numpy as np
    ref_a, ref_b = plain_logits(folders[name], a), plain_logits(folders[name], b)
    first = torch.from_numpy(np.fromfile(tmp_path / "o" / "0.f32", dtype="<f4").reshape(3, -1))
    assert_logits(first, torch.stack([ref_a[0], ref_a[59], ref_b[7]]), "float32", "replayed prompts")
    for t in range(10):
        row = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{1 + t}.f32", dtype="<f4").reshape(1, -1))
        assert_logits(row, ref_a[60 + t:61 + t], "float32", f"replayed token {t}")


def test_command_line_writes_a_random_model_and_generates_from_it(tmp_path, capsys):
    """`write-random`, then `generate` from that folder and straight from the preset's name: the same weights, so the same
    greedy tokens."""
    from kernel_rush_kawk_b200 import cli

    assert cli.main(["write-random", "--preset", "zefapel_tiny", "--seed", "3", "--out", str(tmp_path / "m")]) == 0
    capsys.readouterr()
    common = ["--prompt-ids", "5,6,7,8,9", "--prompt-ids", "11", "--max-new-tokens", "6", "--max-context", "256"]
    assert cli.main(["generate", "--model", str(tmp_path / "m")] + common) == 0
    from_folder = [json.loads(line) for line in capsys.readouterr().out.strip().splitlines()]
    assert cli.main(["generate", "--random", "zefapel_tiny", "--weights-seed", "3"] + common) == 0
    from_preset = [json.loads(line) for line in capsys.readouterr().out.strip().splitlines()]
    assert from_folder == from_preset and [len(r["tokens"]) for r in from_folder] == [6, 6]
