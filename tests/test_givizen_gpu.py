"""Givizen on the GPU: every mechanism's kernels alone against the plain functions of tests/plain_givizen.py, then the
model through the engine: whole prompts, portions, single tokens, unequal batches, reused slots and pages, keys at the
edges of windows and far away, long decoding, greedy generation and trace replay."""

import io
import json
from types import SimpleNamespace

import pytest
import torch

import plain_givizen as plain
from givizen_helpers import CONFIGS, assert_logits, plain_logits, prompts, write_folder

pytestmark = pytest.mark.gpu

DTYPES = (torch.float32, torch.bfloat16)
PART_TOL = {torch.float32: 3e-5, torch.bfloat16: 5e-2}
EPS = 1e-5


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("givizen_gpu")
    return {name: write_folder(root / name, name) for name in CONFIGS}


def runtime(dtype):
    from kernel_rush_kawk_b200.csrc import load_kernels
    from kernel_rush_kawk_b200.engine.model import Runtime

    # with the per-head-size attention libraries of these sizes loaded, bfloat16 steps of many tokens whose key and
    # value heads have one of them take the tensor-core kernel; all others the general one
    return Runtime(torch.device("cuda:0"), dtype, load_kernels((16, 32, 48, 64, 128)))


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


def run_part(part, rt, h, pieces, dtype, prior=(), step_tokens=1024):
    """One sequence through a mixer part, cut into ``pieces``; ``prior``: sequences that used (and gave back) the slot and
    its pages before."""
    from kernel_rush_kawk_b200.cache import SequenceCache

    cache = SequenceCache([part.cache_need()], 2048, 1, 2048, rt.device, dtype, step_tokens=step_tokens)
    for seq, cuts in list(prior) + [(h, pieces)]:
        slot = cache.alloc()
        got, start = [], 0
        for n in cuts:
            assert n <= step_tokens
            cache.reserve(slot, start + n)
            cache.sync()
            ctx = context(rt, [slot], [start], [n], cache)
            got.append(part.forward(ctx, seq[start:start + n].to(dtype).cuda(), cache.view(0)))
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
@pytest.mark.parametrize("size", [64, 50, 33, 320, 1536, 2560, 17000])
def test_norms_of_outputs_on_their_way_into_the_stream(dtype, size):
    """x <- x + r(y) (1 + w), twice over; the rounded rows go along; a last norm reads the stream. The stream stays 32-bit
    whatever the path, and a small x beside a large y (and the other way round) loses nothing."""
    from kernel_rush_kawk_b200.parts import Stream, WideRMSNorm

    rt = runtime(dtype)
    ctx = SimpleNamespace(ops=rt.ops)
    for x_scale, y_scale in ((3.0, 2.0), (1e-3, 500.0), (200.0, 1e-3)):
        x = rand((7, size), 1, x_scale)
        stream, s = Stream(x.cuda()), x.double()
        norms = []
        for q in range(3):
            w = (0.3 * rand((size,), 10 + q)).to(torch.bfloat16)
            part = WideRMSNorm({"size": size, "eps": EPS, "gain_offset": 1.0})
            part.bind({"weight": w.to(dtype).cuda()}, rt)
            norms.append((part, w.double()))
        close(norms[0][0].read_stream(ctx, stream), s, dtype, "the stream as a sublayer reads it")
        for q in range(2):
            y = rand((7, size), 20 + q, y_scale).to(dtype)
            norms[q][0].fold_output(ctx, stream, y.cuda())
            s = s + plain.norm(y.double(), norms[q][1], EPS)
            assert stream.x.dtype == torch.float32 and (stream.x.double().cpu() - s).abs().max() < 2e-6 * s.abs().max()
            assert stream.rows.dtype == dtype and norms[q][0].read_stream(ctx, stream) is stream.rows
            assert torch.equal(stream.rows, stream.x.to(dtype))
        close(norms[2][0].forward(ctx, stream).tensor(), plain.norm(s, norms[2][1], EPS), dtype, "a norm of the stream")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [64, 50, 33, 1300])
def test_embedding_leaves_its_rows_in_both_types(dtype, size):
    from kernel_rush_kawk_b200.parts import ScaledEmbedding

    rt = runtime(dtype)
    table = rand((19, size), 1).to(torch.bfloat16)
    part = ScaledEmbedding({"vocab": 19, "hidden": size, "scale": 7.3, "rounded": True})
    part.bind({"table": table.to(dtype).cuda()}, rt)
    ids = torch.tensor([3, 18, 0, 3, 7], dtype=torch.int32)
    stream = part.forward(SimpleNamespace(ops=rt.ops, batch=SimpleNamespace(tokens=ids.cuda(), n_rows=5)))
    want = table.double()[ids.long()] * 7.3
    assert stream.x.dtype == torch.float32 and (stream.x.double().cpu() - want).abs().max() < 1e-5
    assert torch.equal(stream.rows, stream.x.to(dtype))
    plain_rows = ScaledEmbedding({"vocab": 19, "hidden": size, "scale": 7.3})
    plain_rows.bind({"table": table.to(dtype).cuda()}, rt)
    assert torch.equal(plain_rows.forward(SimpleNamespace(ops=rt.ops, batch=SimpleNamespace(tokens=ids.cuda(), n_rows=5))), stream.x)


def test_capped_logits():
    rt = runtime(torch.float32)
    for rows, vocab, cap in ((1, 7, 3.0), (3, 33, 30.0), (2, 1024, 0.5), (5, 50001, 12.0)):
        z = rand((rows, vocab), 1, 2.0 * cap)
        z[0, :4] = torch.tensor([1e6, -1e6, 0.0, 1e-4])
        got = rt.ops.tanh_cap_(z.cuda(), cap)
        want = plain.cap(z.double(), cap)
        assert (got.double().cpu() - want).abs().max() < 1e-6 * cap
        assert abs(got[0, 3].item() - want[0, 3].item()) < 1e-9  # small logits keep their relative precision


ROW_SHAPES = [(4, 2, 16, 24), (3, 1, 7, 5), (2, 2, 128, 64), (5, 5, 48, 48), (1, 1, 256, 4), (2, 1, 260, 12), (6, 3, 6, 10)]  # H, G, D, P


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", ROW_SHAPES)
@pytest.mark.parametrize("weights", [True, False])
@pytest.mark.parametrize("temp", [(0.5, 64), (1.3, 1), None])
def test_head_norms_temperature_and_cache_write(dtype, shape, weights, temp):
    """Queries in place, keys and values in their pages; positions across several steps of the temperature, at page borders
    and far into a sequence. A second call gives a bias, which takes the general kernel: the same but for the bias."""
    from kernel_rush_kawk_b200.cache import SequenceCache
    from kernel_rush_kawk_b200.parts import KVNeed

    rt = runtime(dtype)
    H, G, D, P = shape
    n = H * D + G * (D + P)
    proj = rand((140, n + 3), 1, 1.5).to(dtype)
    gain = (1 + 0.3 * rand((2 * D,), 2)) if weights else None
    bias = rand((n,), 3)
    for start in (0, 127, 5000):
        for b in (None, bias):
            cache = SequenceCache([KVNeed(G, D, None, None if P == D else P)], 8192, 2, 8192, rt.device, dtype)
            slot = cache.alloc()
            cache.reserve(slot, start + 140)
            cache.sync()
            view, batch = cache.view(0), context(rt, [slot], [start], [140], cache).batch
            rows = proj.cuda()
            rt.ops.bias_norm_rotate_write(rows, 0, H * D, (H + G) * D, H, G, D, P, None if b is None else b.cuda(),
                                          None if gain is None else gain.cuda(), EPS, torch.zeros(0, device="cuda"), 0, False,
                                          batch, view, unit=not weights, temperature=temp)
            x = proj[:, :n].double() + (0.0 if b is None else b.double())
            q, k = plain.rms(x[:, :H * D].view(140, H, D), EPS), plain.rms(x[:, H * D:(H + G) * D].reshape(140, G, D), EPS)
            if weights:
                q, k = q * gain[:D].double(), k * gain[D:].double()
            if temp is not None:
                q = q * torch.tensor([plain.temperature(start + i, *temp) for i in range(140)], dtype=torch.float64)[:, None, None]
            pos = torch.arange(start, start + 140)
            page = cache.view(0).table[slot].cpu().long()[pos // 64]
            tol = 1e-5 if dtype == torch.float32 else 5e-3
            err = lambda got, want: (got.double().cpu() - want).abs().max().item() / want.abs().max().item()
            assert err(rows[:, :H * D].reshape(140, H, D), q) < tol and err(view.k.cpu()[page, :, pos % 64], k) < tol
            assert err(view.v.cpu()[page, :, pos % 64], x[:, (H + G) * D:].reshape(140, G, P)) < tol
            assert torch.equal(rows[:, H * D:].cpu(), proj[:, H * D:])  # the rest of the rows is left alone


def attention_part(kind, C, H, G, D, P, window, dtype, rt, scale=None, softcap=4.0, temp=(0.6, 16), seed=100, sink=None):
    from kernel_rush_kawk_b200.parts import SinkWindowAttention

    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": P, "scale": scale or 1.6 * D ** -0.5}
    if window is not None:
        m["mask"] = {"size": window}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    params = {"hidden": C, "heads": H, "kv_heads": G, "dim": D, "vdim": P, "scale": m["scale"], "window": window, "q_temp": temp,
              "distance_bias": True, "eps": EPS}
    w = {"q": rand((H * D, C), seed, C ** -0.5), "k": rand((G * D, C), seed + 1, C ** -0.5), "v": rand((G * P, C), seed + 2, C ** -0.5),
         "o": rand((C, H * P), seed + 3, (H * P) ** -0.5)}
    if kind == "attention":
        params.update({"qk_norm": "head", "sink": True})
        w.update({"q.norm": 1 + 0.3 * rand((D,), seed + 4), "k.norm": 1 + 0.3 * rand((D,), seed + 5),
                  "sink": rand((H,), seed + 6, 2.0) if sink is None else torch.tensor(sink)})
    else:
        m["softcap"] = softcap
        params.update({"qk_norm": "head_rms", "softcap": softcap, "gate": "head"})
        w["g"] = rand((H, C), seed + 7, 2.0 * C ** -0.5)
    part = SinkWindowAttention(params)
    assert {k: tuple(s.shape) for k, s in part.tensor_specs().items()} == {k: tuple(v.shape) for k, v in w.items()}
    dev, ref = as_path(w, dtype)
    part.bind(dev, rt)
    return part, ref, m


ATTENTION_SHAPES = [  # hidden, heads, kv heads, dim, vdim, window
    (64, 4, 2, 16, 24, 20), (50, 3, 1, 7, 5, 11), (64, 8, 1, 64, 64, 64), (48, 5, 5, 48, 48, 65), (64, 6, 3, 32, 32, 130),
    (40, 18, 1, 16, 16, None), (64, 12, 1, 32, 32, 1), (32, 2, 1, 128, 128, 100), (32, 3, 3, 20, 144, 70), (32, 2, 2, 8, 260, 33),
    (32, 7, 1, 12, 12, 2), (32, 1, 1, 64, 96, 127),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("shape", ATTENTION_SHAPES)
def test_attention_alone(dtype, kind, shape):
    """Whole, in portions down to two tokens, token by token, in a slot whose pages another sequence used."""
    rt = runtime(dtype)
    part, ref, m = attention_part(kind, *shape, dtype, rt)
    T = 200
    h = rand((T, shape[0]), 1, 1.2)
    want = plain.attention(kind, h.to(dtype).double(), ref, "", m, EPS)
    for pieces in ([T], [63, 1, 2, 64, 70], [130] + [1] * 70, [2] * 100):
        close(run_part(part, rt, h, pieces, dtype, prior=[(rand((150, shape[0]), 2), [150])]), want, dtype, f"{kind} {shape}, pieces {pieces[:4]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [32, 24])
def test_the_sink_counts_once_and_is_neither_scaled_nor_biased(dtype, D):
    """Sinks that swallow nearly everything, about half, and nothing, at every distance of a long sequence."""
    rt = runtime(dtype)
    part, ref, m = attention_part("attention", 32, 4, 2, D, D, 90, dtype, rt, sink=[40.0, 2.0, -40.0, 3.0])
    h = rand((260, 32), 3, 1.0)
    part._w_out = torch.eye(4 * D, dtype=dtype, device="cuda")  # look at the heads themselves
    ref["o"] = torch.eye(4 * D, dtype=torch.float64)
    want = plain.attention("attention", h.to(dtype).double(), ref, "", m, EPS)
    for pieces in ([260], [200] + [1] * 60):
        got = run_part(part, rt, h, pieces, dtype)
        close(got, want, dtype, f"sinks, pieces {pieces[:2]}")
        assert got[:, :D].abs().max() < 1e-6 and got[:, 2 * D:3 * D].abs().max() > 0.1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scale, cap", [(6.0, 1.0), (20.0, 3.0), (0.05, 50.0), (2.0, 30.0)])
@pytest.mark.parametrize("D", [32, 20])
def test_scores_far_beyond_their_cap_and_far_below_it(dtype, scale, cap, D):
    """Where the cap levels the scores the bias still orders them (it comes after the cap); where scores are small the cap
    changes nothing. One kv head's keys are made alike, so that the bias alone decides."""
    rt = runtime(dtype)
    part, ref, m = attention_part("attention_2", 32, 3, 1, D, D, 150, dtype, rt, scale=scale, softcap=cap)
    h = rand((300, 32), 5, 1.0)
    want = plain.attention("attention_2", h.to(dtype).double(), ref, "", m, EPS)
    for pieces in ([300], [250] + [1] * 50):
        close(run_part(part, rt, h, pieces, dtype), want, dtype, f"scale {scale} cap {cap}, pieces {pieces[:2]}", loosen=2.0)


EDGES = [  # window, the loud token, total
    (10, 3, 40), (64, 0, 140), (65, 63, 200), (300, 5, 420), (1, 7, 20), (2, 63, 80), (63, 64, 160), (128, 127, 300), (257, 1, 300),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("D", [16, 12])
@pytest.mark.parametrize("window, loud, T", EDGES)
def test_one_loud_token_at_the_edges_of_what_a_query_sees(dtype, kind, D, window, loud, T):
    """One token's value dominates every output that sees it: a window that is one token off shows as a row that is loud or
    quiet at the wrong place. Whole, with the edge crossed token by token, and in pieces of two."""
    rt = runtime(dtype)
    C = 32
    part, ref, m = attention_part(kind, C, 2, 1, D, D, window, dtype, rt, scale=0.02, temp=(0.1, 50), seed=3, sink=[-2.0] * 2)
    h = rand((T, C), 21, 0.3)
    h[loud] *= 3000.0
    hd = h.to(dtype).double()
    want = plain.attention(kind, hd, ref, "", m, EPS)
    sees = (torch.arange(T) > loud) & (torch.arange(T) < loud + window)
    after = torch.arange(T) >= loud + window
    quiet = float(want[after].abs().max()) if after.any() else 0.0
    size = want.abs().max(dim=-1).values
    assert not sees.any() or size[sees].min() > 3 * quiet  # the case shows what it is meant to
    edge = min(T - 1, max(2, loud + window - 2))
    tol = PART_TOL[dtype]
    for pieces in ([T], [edge] + [1] * (T - edge), [2] * (T // 2)):
        got = run_part(part, rt, h, pieces, dtype).double().cpu()
        err = (got - want).abs().max(dim=-1).values / torch.clamp(size, min=max(quiet, 0.05))  # row by row: loud rows hide nothing
        assert err.max() <= tol, f"{kind} window {window} loud {loud}, pieces {pieces[:3]}: row {int(err.argmax())} off by {err.max():.3e}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("D", [32, 28])
def test_one_key_that_the_last_queries_look_for_wherever_it_sits(dtype, kind, D):
    """One token points where the last queries look, so that one score stands out among hundreds: at the start, at page
    borders, just before the query, just inside and just outside a wide window; slopes small enough to see that far (the last
    of sixteen heads). In a prompt and in single tokens."""
    rt = runtime(dtype)
    C, T, window = 48, 700, 600
    part, ref, m = attention_part(kind, C, 16, 2, D, D, window, dtype, rt, scale=1.2, softcap=60.0, seed=7, sink=[1.0] * 16)
    ref["k"] = ref["q"][-D:].repeat(2, 1)  # a token's key is what a like token's query of the last head looks for
    part.w["k"] = ref["k"].to(dtype).cuda()
    part.bind_standalone()
    for place in (0, 1, 63, 64, 65, 98, 99, 100, 101, 102, 128, 383, 639, 640, 698):
        h = rand((T, C), 5, 0.3)
        h[place] = rand((C,), 6, 3.0)
        h[-2:] = h[place] * 0.5
        want = plain.attention(kind, h.to(dtype).double(), ref, "", m, EPS)
        for pieces in ([T], [T - 5] + [1] * 5):
            close(run_part(part, rt, h, pieces, dtype), want, dtype, f"key {place}, pieces {pieces[:2]}", loosen=1.5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
@pytest.mark.parametrize("heads", [(4, 2, 32, 32, 70), (10, 1, 20, 12, 33)])
def test_unequal_batches_against_each_alone(dtype, kind, heads):
    rt = runtime(dtype)
    part, ref, m = attention_part(kind, 48, *heads, dtype, rt)
    lengths = [150, 1, 64, 200, 65, 3]
    seqs = [rand((n, 48), 40 + i, 1.2) for i, n in enumerate(lengths)]
    got = run_batch(part, rt, seqs, [140, 1, 63, 130, 64, 1], dtype)
    for i, s in enumerate(seqs):
        close(got[i], plain.attention(kind, s.to(dtype).double(), ref, "", m, EPS), dtype, f"{kind}, sequence {i} of the batch")


@pytest.mark.parametrize("n_seqs", [1, 3, 9, 20, 60])
def test_single_tokens_with_keys_split_over_more_or_fewer_blocks(n_seqs):
    """The number of blocks that share a sequence's keys falls with the batch: every sequence against the general kernel."""
    from kernel_rush_kawk_b200.cache import SequenceCache
    from kernel_rush_kawk_b200.parts import KVNeed

    for dtype in DTYPES:
        rt = runtime(dtype)
        H, G, D = 8, 2, 64
        cache = SequenceCache([KVNeed(G, D, None)], 64 * (n_seqs * 8), n_seqs, 2048, rt.device, dtype)
        lengths = [1 + (97 * i) % 450 for i in range(n_seqs)]
        slots = [cache.alloc() for _ in lengths]
        for s, n in zip(slots, lengths):
            cache.reserve(s, n)
            cache.advance(s, n - 1)
        cache.sync()
        view = cache.view(0)
        view.k.copy_(rand(tuple(view.k.shape), 1))
        view.v.copy_(rand(tuple(view.v.shape), 2))
        batch = context(rt, slots, [n - 1 for n in lengths], [1] * n_seqs, cache).batch
        proj = rand((n_seqs, H * D + 8), 3, 0.4).to(dtype).cuda()
        slopes = torch.tensor(plain.slopes(H)).float().cuda()
        sink = torch.linspace(-2, 2, H).cuda()
        got, want = (torch.zeros((n_seqs, H * D), dtype=dtype, device="cuda") for _ in range(2))
        args = (proj, 0, H, D, D, sink, 0.7, 300, batch, view)
        rt.ops.sink_attention(*args, got, 0, 0.5, gate=(H * D, "head"), slopes=slopes, softcap=6.0)
        batch.is_decode = False  # the step as one of unequal tokens: the kernels for many tokens
        rt.ops.sink_attention(*args, want, 0, 0.5, gate=(H * D, "head"), slopes=slopes, softcap=6.0)
        close(got, want, dtype, f"{n_seqs} sequences", loosen=0.3)


MOE_SHAPES = [  # hidden, experts, top, ff, limit, (shared ff, limit)
    (64, 5, 2, 40, 1.0, (24, 0.5)), (96, 8, 1, 48, 0.3, None), (50, 3, 3, 11, 2.0, (7, 1.0)), (64, 16, 4, 32, 0.7, (64, 3.0)),
    (32, 2, 2, 16, 7.0, (8, 7.0)), (32, 9, 8, 1800, 0.2, None), (192, 10, 2, 80, 1.0, (104, 0.4)), (136, 40, 4, 264, 0.6, None),
    (64, 70, 2, 64, 1.5, (8, 0.1)), (256, 2, 1, 72, 0.8, (40, 2.0)),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", MOE_SHAPES)
@pytest.mark.parametrize("rows", [1, 5, 200, 777])
def test_routed_experts_with_weighted_inputs_alone(dtype, shape, rows):
    """Few rows (every pair reads its expert) and many (rows ordered by expert), with inputs beyond the limits on both sides;
    the shared expert has a limit of its own."""
    from kernel_rush_kawk_b200.parts import RoutedExperts

    rt = runtime(dtype)
    C, E, top, F, limit, shared = shape
    part = RoutedExperts({"hidden": C, "experts": E, "top": top, "intermediate": F, "activation": "swish_clamped", "limit": limit,
                          "scoring": "sigmoid", "weigh_input": True, "shared_intermediate": shared and shared[0],
                          "shared_limit": shared and shared[1]})
    w = {"router": rand((E, C), 1, 2.0 * C ** -0.5)}
    for e in range(E):
        w.update({f"e{e}.gate": rand((F, C), 11 + 3 * e, 2.0 * C ** -0.5), f"e{e}.up": rand((F, C), 12 + 3 * e, 2.0 * C ** -0.5),
                  f"e{e}.down": rand((C, F), 13 + 3 * e, F ** -0.5)})
    if shared is not None:
        w.update({"shared.gate": rand((shared[0], C), 4, 2.0 * C ** -0.5), "shared.up": rand((shared[0], C), 5, 2.0 * C ** -0.5),
                  "shared.down": rand((C, shared[0]), 6, shared[0] ** -0.5)})
    assert {k: tuple(s.shape) for k, s in part.tensor_specs().items()} == {k: tuple(v.shape) for k, v in w.items()}
    dev, ref = as_path(w, dtype)
    part.bind(dev, rt)
    h = rand((rows, C), 7, 1.5).to(dtype)
    mlp = {"router": {"experts": E, "top": top}, "expert": {"ff": F, "limit": limit},
           "shared": None if shared is None else {"ff": shared[0], "limit": shared[1]}}
    want = plain.routed_ff(h.double(), ref, "", mlp)
    for decode in (False, True):
        ctx = SimpleNamespace(ops=rt.ops, batch=SimpleNamespace(is_decode=decode))
        close(part.forward(ctx, h.cuda()), want, dtype, f"experts {shape}, {rows} rows, single-token step {decode}")
    rt.ops.check()


@pytest.mark.parametrize("tall", [0, 1])
@pytest.mark.parametrize("act, weighted", [(3, True), (3, False), (0, False)])
def test_grouped_gated_products_where_experts_have_few_rows_many_or_none(tall, act, weighted):
    rt = runtime(torch.bfloat16)
    for E, N, K, counts in ((5, 200, 72, [0, 300, 1, 0, 128]), (3, 64, 128, [129, 0, 0]), (3, 136, 64, [256, 257, 511]),
                            (40, 320, 96, [7 * (e % 3) for e in range(40)])):
        offsets = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
        rows = int(offsets[-1])
        a, w = rand((rows + 5, K), 1, 2.0).to(torch.bfloat16), rand((E, 2 * N, K), 2, K ** -0.5).to(torch.bfloat16)
        weights = torch.rand(rows + 5, generator=torch.Generator().manual_seed(4))
        out = torch.full((rows + 5, N), 7.0, dtype=torch.bfloat16, device="cuda")
        a_d, w_d, o_d, r_d = a.cuda(), w.cuda(), offsets.cuda(), weights.cuda()
        rt.ops._ok(rt.ops.moe.krk_grouped_gemm(out.data_ptr(), a_d.data_ptr(), w_d.data_ptr(), o_d.data_ptr(), rows + 5, E, N, K,
                                               act, 1, tall, r_d.data_ptr() if weighted else None, 1.3, 1.702,
                                               rt.ops.error.data_ptr(), rt.ops._stream()), "grouped product")
        want = torch.full((rows + 5, N), 7.0, dtype=torch.float64)
        for e in range(E):
            lo, hi = int(offsets[e]), int(offsets[e + 1])
            y = a[lo:hi].double() @ w[e].double().t()
            if weighted:
                y = y * weights[lo:hi, None].double()
            g, u = y[:, :N], y[:, N:]
            if act == 3:
                g, u = torch.clamp(g, max=1.3), torch.clamp(u, min=-1.3, max=1.3)
                want[lo:hi] = g * torch.sigmoid(1.702 * g) * (u + 1.0)
            else:
                want[lo:hi] = g * torch.sigmoid(g) * u
        close(out, want, torch.bfloat16, f"{E} experts")  # rows beyond the last expert's stay as they were
    rt.ops.check()


@pytest.mark.parametrize("tall", [0, 1])
def test_grouped_products_without_a_gate_in_tall_tiles(tall):
    rt = runtime(torch.bfloat16)
    for E, N, K, counts in ((3, 200, 72, [0, 300, 129]), (3, 264, 64, [256, 257, 511]), (2, 512, 128, [128, 1])):
        offsets = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
        rows = int(offsets[-1])
        a, w = rand((rows, K), 1).to(torch.bfloat16), rand((E, N, K), 2, K ** -0.5).to(torch.bfloat16)
        out = torch.full((rows, N), 7.0, dtype=torch.bfloat16, device="cuda")
        a_d, w_d, o_d = a.cuda(), w.cuda(), offsets.cuda()
        rt.ops._ok(rt.ops.moe.krk_grouped_gemm(out.data_ptr(), a_d.data_ptr(), w_d.data_ptr(), o_d.data_ptr(), rows, E, N, K, -1, 0,
                                               tall, None, 0.0, 0.0, rt.ops.error.data_ptr(), rt.ops._stream()), "grouped product")
        want = torch.cat([a[int(offsets[e]):int(offsets[e + 1])].double() @ w[e].double().t() for e in range(E)])
        close(out, want, torch.bfloat16, f"{E} experts")
    rt.ops.check()


def test_routing_by_sigmoid_by_hand():
    """The largest logits, weighted by their own sigmoids; equal logits: the lower index; negative and saturated ones."""
    rt = runtime(torch.float32)
    z = torch.tensor([[2.0, -1.0, 3.0, 0.5], [0.0, 0.0, 0.0, 0.0], [-9.0, -7.0, -8.0, -30.0], [30.0, 40.0, 20.0, 50.0]], device="cuda")
    experts, weights, gate = rt.ops.moe_route(torch.eye(4, device="cuda"), z.t().contiguous(), None, 2, sigmoid=True)
    assert gate is None and experts.tolist() == [[2, 0], [0, 1], [1, 2], [3, 1]]
    assert torch.allclose(weights, torch.sigmoid(z).gather(1, experts.long()), rtol=1e-5, atol=0)


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
@pytest.mark.parametrize("name", ["ga", "gb"])
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
    name = "ga"
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

    name = "gc"
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

    assert cli.main(["write-random", "--preset", "givizen_tiny", "--seed", "3", "--out", str(tmp_path / "m")]) == 0
    capsys.readouterr()
    common = ["--prompt-ids", "5,6,7,8,9", "--prompt-ids", "11", "--max-new-tokens", "6", "--max-context", "256"]
    assert cli.main(["generate", "--model", str(tmp_path / "m")] + common) == 0
    from_folder = [json.loads(line) for line in capsys.readouterr().out.strip().splitlines()]
    assert cli.main(["generate", "--random", "givizen_tiny", "--weights-seed", "3"] + common) == 0
    from_preset = [json.loads(line) for line in capsys.readouterr().out.strip().splitlines()]
    assert from_folder == from_preset and [len(r["tokens"]) for r in from_folder] == [6, 6]
