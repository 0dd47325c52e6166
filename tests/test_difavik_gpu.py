"""The Difavik design on the GPU against the plain implementation (tests/plain_difavik.py).

Mechanisms alone (the boundary kernel that norms what joins the stream, with unsummed splits, experts' rows
and branches; the post-pass with joint norms; attention with linear penalties, kept first keys and head gates;
the fixed-decay recurrence token by token and in chunks; biased clamped feed-forwards; experts weighted by a plain
softmax; the pair embedding's rounding), then whole models of three small configurations: whole prompts,
prefill against token-by-token decoding, portions down to two tokens, unequal requests in one batch against
each alone, pages and slots used again, the first tokens of a sequence, long decoding past every window, and
greedy generation through `Engine` (scheduler, CUDA graphs, asynchronous scheduling, preemption).

Where random inputs would hide a fault, the inputs are made so that it shows: one key that stands out among the
kept ones, just inside and just outside the window, at page borders and at the borders of the pieces that kernels
cut long contexts into; one key whose trace in a slowly decaying state is asked for hundreds of tokens later.

Exactness is tested in float32 (differences of rounding order only); bfloat16 serving is compared with the
float32 oracle with a bound on the error of rounding.
"""
import math

import pytest
import torch

import plain_difavik as plain
import tiny_difavik as tiny
from gpu_util import Harness
from vosti_b200 import Engine, ops
from vosti_b200.config import ConfigError
from vosti_b200.config.difavik import _feed_forward, _lightning, _mixer, _retention, _sloped_attention
from vosti_b200.engine.batch import StepEntry
from vosti_b200.engine.runner import ModelRunner
from vosti_b200.parts import PagedCacheSpec, build_feed_forward, build_mixer
from vosti_b200.parts.feed_forward import interleave_gate_up

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32 = dict(atol=3e-4, rtol=3e-4)
EPS = 2e-6
LOG2E = 1.4426950408889634


def rounded(*shape, gen, std=1.0, mean=0.0):
    """Random values that bfloat16 holds exactly, as float32 on the CPU."""
    return (mean + std * torch.randn(tuple(shape), generator=gen)).to(torch.bfloat16).float()


def give(part, W, dtype):
    """Hand a part its tensors (keys of `weight_specs`) on the device in the serving layout."""
    assert set(W) == set(part.weight_specs()), (sorted(W), sorted(part.weight_specs()))
    part.load({k: v.to(DEV, dtype).contiguous() for k, v in W.items()}, dtype)
    part.setup(torch.device(DEV), dtype)


def weights_of(part, gen, prefix="l0.mix."):
    return {key: tiny.draw(prefix + key, w, gen).to(torch.bfloat16).float() for key, w in part.weight_specs().items()}


def double(W):
    return {k: v.double() for k, v in W.items()}


def close(got, want, dtype, what=None):
    assert torch.isfinite(got).all(), what
    if dtype == torch.float32:
        assert torch.allclose(got, want, **F32), (what, float((got - want).abs().max()))
    else:
        assert float((got - want).abs().mean() / want.abs().mean()) < 0.04, (what, float((got - want).abs().mean() / want.abs().mean()))


def run_mixer(mixer, harness, x, sizes, dtype, rid="r"):
    """The mixer over x in portions."""
    outs, at = [], 0
    for size in sizes:
        ctx = harness.context([StepEntry(rid, [0] * size)])
        out = mixer.forward(ctx, x[at:at + size].to(DEV, dtype).contiguous(), harness.cache.layer_caches[0])
        outs.append(ops.materialize(out).float().cpu())
        harness.cache.trim(rid)
        at += size
    assert at == x.shape[0] and int(harness.status.item()) == 0
    return torch.cat(outs)


CUTS = lambda T: ((T,), (T - 33,) + (1,) * 33, (2, 5, 1, 1, 17, 2, 3, T - 31), (T - 6, 2, 4))


def partial_of(x, splits, gen, scratch):
    """x as the unsummed K splits of a product."""
    parts = torch.randn((splits, *x.shape), generator=gen)
    parts[-1] = x - parts[:-1].sum(0)
    return ops.PartialSum(parts.to(DEV), splits, x.shape[0], x.shape[1], torch.float32, status_word(), scratch)


def status_word():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------- the boundary between sublayers
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,rows", [(200, 9), (67, 5), (1, 3), (4, 2), (1028, 70), (4099, 3), (4100, 2), (25600, 1), (25604, 1)])
def test_boundary_norms_what_joins_the_stream(dtype, width, rows):
    gen = torch.Generator().manual_seed(width)
    x, y, z = (torch.randn(rows, width, generator=gen) for _ in range(3))
    w, scale, bias, wa, wb = (rounded(width, gen=gen, std=0.4, mean=m) for m in (0.0, 0.8, 0.0, 1.2, 1.1))
    store = torch.bfloat16 if dtype == torch.bfloat16 else torch.float32
    status = status_word()
    dev = lambda t: t.to(DEV, store)

    def check(source, out, with_scale=True, with_bias=False):
        out = out.double() + (bias.double() if with_bias else 0.0)
        want = x.double() + (scale.double() if with_scale else 1.0) * plain.offset_norm(out, w.double(), EPS)
        stream = x.to(DEV).clone()
        pair = ops.out_norm_stream(ops.StreamPair(stream, stream), source, dev(w), EPS, dtype, status, offset=1.0,
                                   scale=dev(scale) if with_scale else None, bias=bias.to(DEV) if with_bias else None)
        assert pair.stream.data_ptr() == stream.data_ptr() and pair.rounded.dtype == dtype
        assert torch.allclose(stream.cpu(), want.float(), atol=4e-5, rtol=4e-5)
        assert torch.equal(pair.rounded.cpu(), stream.to(dtype).cpu())

    check(y.to(DEV), y)
    check(y.to(DEV), y, with_scale=False, with_bias=True)
    low = y.to(torch.bfloat16)
    check(low.to(DEV), low.float())
    for splits in (2, 3, 12):
        check(partial_of(y, splits, gen, "split_k"), y, with_bias=True)
    # the mean of two branches, each as a tensor or as splits
    mean = 0.5 * (plain.unit_rms(y.double(), EPS) * wa.double() + plain.unit_rms(z.double(), EPS) * wb.double())
    for a, b in ((y.to(DEV), z.to(DEV)), (partial_of(y, 3, gen, "split_k_branch0"), partial_of(z, 5, gen, "split_k_branch1")),
                 (partial_of(y, 9, gen, "split_k_branch0"), z.to(DEV))):
        branches = ops.BranchMean((a, b), (dev(wa), dev(wb)), EPS)
        assert torch.allclose(branches.materialize().cpu(), mean.float(), atol=1e-4, rtol=1e-4)
        check(branches, mean)
    assert int(status.item()) == 0


@pytest.mark.parametrize("width", [48, 37])
def test_boundary_adds_a_tokens_experts_with_their_weights(width):
    gen = torch.Generator().manual_seed(width)
    rows, picks = 6, 3
    y, x = torch.randn(rows * picks, width, generator=gen), torch.randn(rows, width, generator=gen)
    where = torch.randperm(rows * picks, generator=gen).view(rows, picks).to(torch.int32)
    weights = torch.rand(rows, picks, generator=gen)
    w = rounded(width, gen=gen, std=0.3)
    for splits in (1, 5):
        source = y.to(DEV) if splits == 1 else partial_of(y, splits, gen, "split_k")
        for own in (True, False):
            by = weights if own else torch.full_like(weights, 0.25)
            total = (y.double()[where.long()] * by.double()[..., None]).sum(1)
            picked = ops.PickedSum(source, where.to(DEV), 0.25, weights.to(DEV) if own else None)
            assert torch.allclose(picked.materialize().cpu(), total.float(), atol=1e-5)
            stream = x.to(DEV).clone()
            ops.out_norm_stream(ops.StreamPair(stream, stream), picked, w.to(DEV), EPS, torch.float32, status_word(), offset=1.0)
            want = x.double() + plain.offset_norm(total, w.double(), EPS)
            assert torch.allclose(stream.cpu(), want.float(), atol=1e-5, rtol=1e-5)


def test_two_unsummed_branches_need_a_scratch_each():
    gen = torch.Generator().manual_seed(1)
    a, b = (partial_of(torch.randn(2, 8, generator=gen), 2, gen, "split_k") for _ in range(2))
    with pytest.raises(ops.KernelError, match="scratch"):
        ops.BranchMean((a, b), (torch.ones(8, device=DEV),) * 2, EPS)


# ---------------------------------------------------------------- the pair embedding's rounding
@pytest.mark.parametrize("width", [64, 37])
def test_pair_embedding_writes_the_stream_and_its_rounding(width):
    gen = torch.Generator().manual_seed(width)
    table, pairs = rounded(50, width, gen=gen), rounded(12, width, gen=gen)
    from vosti_b200.parts import StateSpec
    harness = Harness([None], [StateSpec((1,), torch.int32)], torch.bfloat16, max_requests=2)
    tokens = torch.randint(0, 50, (23,), generator=gen).tolist()
    want = table[tokens] + pairs[plain.pair_rows(tokens, 11, 7, 3)]
    at, got = 0, []
    for size in (1, 1, 2, 9, 1, 9):
        ctx = harness.context([StepEntry("r", tokens[at:at + size])])
        pair, ids = ops.pair_embedding(ctx.tokens, table.to(DEV, torch.bfloat16), pairs.to(DEV, torch.bfloat16),
                                       harness.cache.layer_caches[0].state.view(-1), ctx, buckets=11, mul_prev=7, mul_cur=3, rounded=True)
        assert torch.equal(pair.rounded, pair.stream.to(torch.bfloat16)) and ids.cpu().tolist() == tokens[at:at + size]
        got.append(pair.stream.cpu())
        at += size
    assert torch.equal(torch.cat(got), want)


# ---------------------------------------------------------------- joint norms
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nq,nkv,dk,extra", [(6, 3, 14, 6), (8, 2, 64, 8), (1, 1, 1, 1), (5, 5, 7, 0), (32, 4, 128, 32)])
def test_joint_norms_and_values_that_are_keys(dtype, nq, nkv, dk, extra):
    gen = torch.Generator().manual_seed(nq * dk)
    T, page = 21, 8
    width = (nq + nkv) * dk
    proj, bias = 2.0 * torch.randn(T, width + extra, generator=gen), torch.randn(width, generator=gen)
    qn, kn = rounded(nq * dk, gen=gen, std=0.3, mean=1.0), rounded(nkv * dk, gen=gen, std=0.3, mean=1.0)
    row = proj[:, :width].double() + bias.double()
    q_want = (plain.unit_rms(row[:, : nq * dk], EPS) * qn.double()).float()
    k_want = (plain.unit_rms(row[:, nq * dk:], EPS) * kn.double()).float().view(T, nkv, dk)
    v_want = row[:, nq * dk:].float().view(T, nkv, dk)
    tol = dict(atol=2e-5, rtol=2e-5) if dtype == torch.float32 else dict(atol=1e-2, rtol=1e-2)
    for splits in (1, 4):
        harness = Harness([PagedCacheSpec(entries=2, heads=nkv, width=dk)], [None], dtype, num_pages=4, page_size=page)
        ctx = harness.context([StepEntry("r", [0] * T)])
        cache, group = harness.cache.layer_caches[0], ctx.group(0)
        source = proj.to(DEV) if splits == 1 else partial_of(proj, splits, gen, "split_k")
        q, gate = ops.qk_joint(source, cache.k, cache.v, nq=nq, nkv=nkv, dk=dk, page_size=page, slot_mapping=group.slot_mapping,
                               out_dtype=dtype, status=ctx.status, q_norm=qn.to(DEV), k_norm=kn.to(DEV), eps=EPS, bias=bias.to(DEV),
                               extra_width=extra)
        slots = group.slot_mapping.cpu().long()
        k = cache.k.cpu().float()[slots // page, :, slots % page]
        v = cache.v.cpu().float()[slots // page, :, slots % page]
        assert torch.allclose(q.float().cpu(), q_want, **tol) and torch.allclose(k, k_want, **tol) and torch.allclose(v, v_want, **tol)
        assert (gate is None) == (extra == 0)
        if extra:
            assert torch.allclose(gate.cpu(), proj[:, width:], atol=2e-5, rtol=2e-5)
        assert int(harness.status.item()) == 0


# ---------------------------------------------------------------- attention with penalties, kept keys and gates
ATTENTION_SIZES = [
    # heads, kv heads, dim, window, kept, page
    (6, 3, 14, 13, 11, 8), (4, 1, 10, 37, 3, 8), (1, 1, 1, 1, 0, 4), (3, 3, 40, 20, 33, 16), (8, 2, 48, 130, 20, 16), (2, 1, 96, 5, 1, 4),
    # sizes the tensor-core kernels take in bfloat16
    (8, 2, 64, 50, 20, 16), (4, 4, 128, 70, 17, 16), (16, 1, 64, 33, 64, 32), (2, 2, 64, 1, 1, 16), (4, 2, 128, 300, 40, 64), (6, 2, 64, 16, 0, 16),
    (8, 1, 128, 90, 130, 16)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv,dim,window,keep,page", ATTENTION_SIZES)
def test_sloped_attention_mixer_against_plain(dtype, heads, kv, dim, window, keep, page):
    gen = torch.Generator().manual_seed(heads * 100 + dim)
    width, T = 72, 190
    block = tiny.left(heads, kv, dim, 2.5 / math.sqrt(dim), window, keep)
    mixer = build_mixer(_sloped_attention(block, EPS, "left"), width, None)
    assert set(mixer.weight_specs()) == {"q", "q.b", "k", "k.b", "q.norm", "k.norm", "g", "o"}
    assert (mixer.cache_spec().window, mixer.cache_spec().keep_first) == (window, keep)
    W = weights_of(mixer, gen)
    give(mixer, W, dtype)
    x = rounded(T, width, gen=gen)
    want = plain.sloped_attention(x.double(), double(W), block, EPS).float()
    for sizes in CUTS(T):
        harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
        close(run_mixer(mixer, harness, x, sizes, dtype), want, dtype, sizes)


def test_attention_without_a_window_and_every_decode_kernel():
    """No mask at all (penalties alone), and the split-key decode kernels one by one: the one with a CTA per item,
    the persistent one, and a pinned segment length that a short context needs several of."""
    gen = torch.Generator().manual_seed(5)
    width, T, dtype = 96, 700, torch.bfloat16
    for window, keep in ((0, 0), (260, 50), (100, 0)):
        block = tiny.left(8, 2, 64, 0.3, max(window, 1), keep)
        block["mask"] = dict(size=window, keep_first=keep) if window else None
        mixer = build_mixer(_sloped_attention(block, EPS, "left"), width, None)
        W = weights_of(mixer, gen)
        give(mixer, W, dtype)
        x = rounded(T, width, gen=gen)
        want = plain.sloped_attention(x.double(), double(W), dict(block, mask=dict(size=window or T, keep_first=keep)), EPS).float()
        for once, segment in ((True, 0), (False, 0), (True, 64), (False, 128)):
            ops.set_decode_once(once)
            ops.library().vosti_set_decode_segment(segment)
            try:
                harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=45, page_size=16)
                got = run_mixer(mixer, harness, x, (T - 40,) + (1,) * 38 + (2,), dtype)
            finally:
                ops.set_decode_once(True)
                ops.library().vosti_set_decode_segment(0)
            close(got, want, dtype, (window, once, segment))
            close(got[-40:], want[-40:], dtype, (window, once, segment, "decoded"))


@pytest.mark.parametrize("dtype,dim,window,keep", [(torch.float32, 24, 40, 21), (torch.bfloat16, 24, 300, 37), (torch.bfloat16, 64, 70, 19),
                                                   (torch.bfloat16, 128, 300, 33), (torch.float32, 64, 290, 260), (torch.bfloat16, 64, 130, 70)])
def test_one_key_stands_out_at_the_edges_of_the_window_and_of_the_kept_keys(dtype, dim, window, keep):
    """The caches are written directly: all keys are small but the target's, which one query element looks for.
    A target that is visible must weigh as the plain softmax says (its penalty included), one that is not must not
    be seen at all. In prompts and in decoding."""
    heads, page = 4, 16
    gen = torch.Generator().manual_seed(dim + window)
    T = keep + 2 * window + 53
    oldest = T - window
    slopes = torch.tensor(plain.slopes(heads), dtype=torch.float64)
    borders = {b + d for p in (page, 32, 64, ops.SINK_SEGMENT) for b in range(0, T, p) for d in (-1, 0) if b in (0, p, keep // p * p, oldest // p * p, (oldest // p + 1) * p)}
    interesting = {0, 1, keep - 1, keep, keep + 1, oldest - 1, oldest - 2, oldest, oldest + 1, T - 2, T - 1} | borders
    base_k, v = rounded(T, dim, gen=gen, std=0.3), rounded(T, dim, gen=gen)
    base_k[:, 0] = 0.0
    q = rounded(T, heads, dim, gen=gen, std=0.3)
    q[T - 1, :, 0] = 8.0
    mask = plain.window_keeping_first(T, window, keep)
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).double()

    def oracle(k):
        scores = torch.einsum("ihd,jd->hij", q.double(), k.double()) * 0.25 - slopes[:, None, None] * back
        return (torch.softmax(scores.masked_fill(~mask, float("-inf")), dim=-1) @ v.double()).permute(1, 0, 2)

    for target in sorted(t for t in interesting if 0 <= t < T):
        k = base_k.clone()
        k[target, 0] = 8.0                      # a score of 16 before the penalty
        want = oracle(k)
        visible = target >= oldest or target < keep
        moved = float((want[T - 1] - oracle(base_k)[T - 1]).abs().max())
        assert (moved > 0.05) if visible else moved == 0.0, target
        for sizes in ((T,), (T - 1, 1), (T - 2, 2), (T - 7, 7), (oldest - 1, T - oldest + 1)):
            spec = PagedCacheSpec(entries=2, heads=1, width=dim, window=window, keep_first=keep)
            harness = Harness([spec], [None], dtype, num_pages=-(-T // page) + 1, page_size=page)
            at = 0
            for size in sizes:
                ctx = harness.context([StepEntry("r", [0] * size)])
                cache, group = harness.cache.layer_caches[0], ctx.group(0)
                slots = group.slot_mapping.long()
                cache.k[slots // page, 0, slots % page] = k[at:at + size].to(DEV, dtype)
                cache.v[slots // page, 0, slots % page] = v[at:at + size].to(DEV, dtype)
                out = ops.attention_sink(ctx, q[at:at + size].reshape(size, -1).to(DEV, dtype).contiguous(), cache.k, cache.v, group, nq=heads,
                                         nkv=1, dk=dim, dv=dim, scale=0.25, window=window, bias=None, sink=None,
                                         slopes=(slopes * LOG2E).float().to(DEV), keep=keep)
                harness.cache.trim("r")
                at += size
            assert int(harness.status.item()) == 0
            got, expected = out[-1].float().cpu().view(heads, dim), want[T - 1].float()
            tol = 2e-4 if dtype == torch.float32 else 0.02 * float(expected.abs().max())
            assert torch.allclose(got, expected, atol=tol, rtol=0), (target, sizes, float((got - expected).abs().max()))


def test_attention_of_unequal_requests_in_one_step_on_the_tensor_cores():
    """A long request decoding one token, a portion in the middle of another and a whole short prompt in one step."""
    gen = torch.Generator().manual_seed(12)
    width, dtype = 96, torch.bfloat16
    for window, keep in ((24, 5), (200, 40)):
        block = tiny.left(4, 2, 64, 0.3, window, keep)
        mixer = build_mixer(_sloped_attention(block, EPS, "left"), width, None)
        W = weights_of(mixer, gen)
        give(mixer, W, dtype)
        xs = {r: rounded(n, width, gen=gen) for r, n in (("a", 420), ("b", 77), ("c", 3))}
        want = {r: plain.sloped_attention(x.double(), double(W), block, EPS).float() for r, x in xs.items()}
        harness = Harness([mixer.cache_spec()], [None], dtype, num_pages=40, page_size=16)
        cache = harness.cache.layer_caches[0]
        run = lambda ctx, rows: ops.materialize(mixer.forward(ctx, torch.cat(rows).to(DEV, dtype), cache)).float().cpu()
        got = {r: [] for r in xs}
        got["a"].append(run(harness.context([StepEntry("a", [0] * 419)]), [xs["a"][:419]]))
        got["b"].append(run(harness.context([StepEntry("b", [0] * 20)]), [xs["b"][:20]]))
        rows = run(harness.context([StepEntry("a", [0]), StepEntry("b", [0] * 37), StepEntry("c", [0] * 3)]),
                   [xs["a"][419:], xs["b"][20:57], xs["c"]])
        got["a"].append(rows[:1]); got["b"].append(rows[1:38]); got["c"].append(rows[38:])
        got["b"].append(run(harness.context([StepEntry("b", [0] * 20)]), [xs["b"][57:]]))
        assert int(harness.status.item()) == 0
        for r in xs:
            close(torch.cat(got[r]), want[r], dtype, (window, r))


# ---------------------------------------------------------------- the fixed-decay recurrence
RECURRENT = [(3, 10, 7), (1, 1, 1), (2, 64, 64), (1, 128, 128), (3, 33, 50), (2, 128, 200), (2, 200, 24), (4, 16, 66), (1, 256, 5), (2, 8, 3)]
RECURRENT_CUTS = ((300,), (128, 128, 44), (127, 129, 44), (1,) * 20 + (280,), (17, 16, 267), (256, 2, 1, 41), (260,) + (1,) * 40)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["retention", "lightning"])
@pytest.mark.parametrize("heads,dim,vdim", RECURRENT)
def test_recurrent_mixers_against_plain(dtype, kind, heads, dim, vdim):
    gen = torch.Generator().manual_seed(heads * 1000 + dim)
    width, T = 72, 300
    decay = [1.0, 0.999, 0.9, 0.6][:heads] if dim % 2 else [0.97, 0.5, 0.9995, 1.0][:heads]
    if kind == "retention":
        if dim < 2:
            pytest.skip("a rotation needs two elements")
        dims = dim - dim % 2 if dim < 100 else 16 * (dim // 32)
        block = tiny.right(heads, dim, vdim, 100.0, dims, decay)
        mixer, oracle = build_mixer(_retention(block, EPS, "right"), width, None), plain.retention
    else:
        block = tiny.lightning(heads, dim, vdim, decay, None)["mixer"]
        mixer, oracle = build_mixer(_lightning(block, EPS, "mixer"), width, None), plain.lightning
    W = weights_of(mixer, gen)
    give(mixer, W, dtype)
    x = rounded(T, width, gen=gen)
    want = oracle(x.double(), double(W), block, EPS).float()
    harness = Harness([None], [mixer.state_spec()], dtype, max_requests=1)         # one slot, used again by every cut
    for n, sizes in enumerate(RECURRENT_CUTS):
        close(run_mixer(mixer, harness, x, sizes, dtype, rid=f"r{n}"), want, dtype, sizes)
        harness.cache.finish(f"r{n}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dv", [(1, 1), (1, 4), (2, 8), (2, 24), (4, 66), (3, 5), (9, 20), (2, 200), (32, 128), (5, 300), (40, 128)])
def test_read_outs_normed_and_gated(dtype, heads, dv):
    gen = torch.Generator().manual_seed(heads + dv)
    width = heads * dv
    for rows in (1, 6, 70):
        o, w = torch.randn(rows, width, generator=gen), rounded(width, gen=gen, std=0.3, mean=1.0)
        for before in (4, 8, 3):                      # columns before the gates
            proj = 2.0 * torch.randn(rows, before + width + 4 - before % 4, generator=gen)
            low = proj.to(dtype).float()
            gates = low[:, before: before + width].double()
            for splits in (0, 1, 5):
                if splits == 0:
                    source = low.to(DEV, dtype)
                else:
                    source = partial_of(low, splits, gen, "split_k")
                    source.dtype = dtype
                for silu in (False, True):
                    g = torch.nn.functional.silu(gates) if silu else torch.sigmoid(gates)
                    tol = dict(atol=3e-5, rtol=3e-5) if dtype == torch.float32 else dict(atol=2e-2, rtol=2e-2)
                    y = ops.decay_out(o.to(DEV), source, before, heads=heads, dv=dv, eps=EPS, weight=w.to(DEV), gate_silu=silu, out_dtype=dtype)
                    assert torch.allclose(y.float().cpu(), (plain.unit_rms(o.double(), EPS) * w.double() * g).float(), **tol), (rows, before, splits, silu)
                    y = ops.decay_out(o.to(DEV), source, before, heads=heads, dv=dv, eps=EPS, weight=None, gate_silu=silu, out_dtype=dtype)
                    want = plain.unit_rms(o.double().view(rows, heads, dv), EPS).view(rows, width) * g
                    assert torch.allclose(y.float().cpu(), want.float(), **tol), (rows, before, splits, silu)


def test_portions_of_several_requests_share_a_step():
    """Requests of unequal length in one step: some go token by token, some in chunks; each equals itself alone."""
    gen = torch.Generator().manual_seed(3)
    width, dtype = 96, torch.bfloat16
    block = tiny.right(2, 64, 80, 500.0, 64, [0.98, 0.9999])
    mixer = build_mixer(_retention(block, EPS, "right"), width, None)
    W = weights_of(mixer, gen)
    give(mixer, W, dtype)
    xs = {r: rounded(n, width, gen=gen) for r, n in (("a", 420), ("b", 177), ("c", 3), ("d", 40))}
    want = {r: plain.retention(x.double(), double(W), block, EPS).float() for r, x in xs.items()}
    harness = Harness([None], [mixer.state_spec()], dtype, max_requests=4)
    at, got = {r: 0 for r in xs}, {r: [] for r in xs}
    for step in ([("a", 131), ("b", 1)], [("b", 150), ("c", 2), ("a", 1)], [("c", 1), ("d", 17), ("a", 257)], [("d", 23), ("b", 26), ("a", 31)]):
        ctx = harness.context([StepEntry(r, [0] * n) for r, n in step])
        rows = torch.cat([xs[r][at[r]:at[r] + n] for r, n in step]).to(DEV, dtype)
        out = ops.materialize(mixer.forward(ctx, rows, harness.cache.layer_caches[0])).float().cpu()
        row = 0
        for r, n in step:
            got[r].append(out[row:row + n])
            row += n
            at[r] += n
    assert all(at[r] == len(x) for r, x in xs.items())
    for r in xs:
        close(torch.cat(got[r]), want[r], dtype, r)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("silu", [False, True])
def test_a_far_key_is_read_out_of_the_state(dtype, silu):
    """One key far back with a large value: the read-out hundreds of tokens later must be decay^distance of it, whether
    the tokens between came in one portion, in several, or one by one. (The recurrence alone, a large signal on
    a small background: rounding does not hide it.)"""
    heads, dk, dv, T = 2, 32, 16, 600
    gen = torch.Generator().manual_seed(7)
    x = rounded(T, heads * (2 * dk + dv), gen=gen, std=0.02)
    offsets = {"q": 0, "k": heads * dk, "v": 2 * heads * dk}
    decay = torch.tensor([0.999, 0.99], dtype=torch.float64)
    act = torch.nn.functional.silu if silu else (lambda t: t)
    for target in (0, 5, 127, 128, 130, 383, 384):
        y = x.clone()
        y[target, heads * dk:] = 4.0
        y[T - 1, : heads * dk] = 2.0
        q, k, v = (act(y.double())[:, a:b].view(T, heads, -1) for a, b in ((0, heads * dk), (heads * dk, 2 * heads * dk), (2 * heads * dk, y.shape[1])))
        want = torch.stack([plain.fixed_decay_recurrence(q[:, h], k[:, h], v[:, h], float(decay[h])) for h in range(heads)], dim=1)[T - 1].float()
        expected = act(torch.tensor(2.0)) * dk * act(torch.tensor(4.0)) ** 2 * decay ** (T - 1 - target)
        assert float(want[0].mean() / expected[0]) > 0.3
        from vosti_b200.parts import StateSpec
        for sizes in ((T,), (T - 1, 1), (300, 300), (130,) + (1,) * 20 + (450,)):
            harness = Harness([None], [StateSpec((heads * dk * dv,))], dtype, max_requests=1)
            at = 0
            for size in sizes:
                ctx = harness.context([StepEntry("r", [0] * size)])
                o = ops.decay_attention(y[at:at + size].to(DEV, dtype).contiguous(), offsets, harness.cache.layer_caches[0].state, ctx, heads=heads,
                                        dk=dk, dv=dv, decay=decay.float().to(DEV), log2_decay=torch.log2(decay).float().to(DEV), silu=silu,
                                        key_scale=1.0, freq=None)
                at += size
            got = o[-1].cpu().view(heads, dv)
            # (bfloat16: SiLU'd activations are rounded in long portions; without an activation everything is exact to 16 bits)
            tol = 1e-4 if dtype == torch.float32 else (2e-2 if silu else 2e-4)
            assert float((got - want).abs().max() / want.abs().max()) < tol, (target, sizes, float((got - want).abs().max() / want.abs().max()))


def test_side_by_side_branches_against_plain():
    gen = torch.Generator().manual_seed(9)
    width, T = 72, 150
    block = dict(left=tiny.left(4, 2, 64, 0.3, 40, 10), right=tiny.right(2, 64, 32, 90.0, 20, [0.95, 0.99]))
    mixer = build_mixer(_mixer("parallel", block, EPS, "layers[0].mixer"), width, None)
    W = weights_of(mixer, gen)
    x = rounded(T, width, gen=gen)
    want = plain.side_by_side(x.double(), double(W), block, EPS).float()
    for dtype in (torch.float32, torch.bfloat16):
        give(mixer, W, dtype)
        for sizes in CUTS(T):
            harness = Harness([mixer.cache_spec()], [mixer.state_spec()], dtype, num_pages=12, page_size=16)
            close(run_mixer(mixer, harness, x, sizes, dtype), want, dtype, sizes)


# ---------------------------------------------------------------- feed-forwards
class Ctx:
    def __init__(self, dtype, all_decode=False):
        self.dtype, self.status, self.extras, self.all_decode = dtype, status_word(), {}, all_decode


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,ff,limit", [(72, 52, 1.3), (64, 17, 0.7), (128, 160, 2.0), (256, 1040, 1.0), (64, 1, 0.5)])
def test_dense_feed_forward_with_biases(dtype, width, ff, limit):
    gen = torch.Generator().manual_seed(ff)
    block = tiny.dense(ff, limit)
    part = build_feed_forward(_feed_forward(block, "mlp"), width)
    W = weights_of(part, gen, "l0.mlp.")
    give(part, W, dtype)
    for rows in (1, 7, 64, 129, 300):
        x = rounded(rows, width, gen=gen)
        ctx = Ctx(dtype)
        y = ops.materialize(part.forward(ctx, x.to(DEV, dtype))).float().cpu() + W["down.b"]      # the block adds the last bias
        close(y, plain.dense_ff(x.double(), double(W), block).float(), dtype, rows)
        assert int(ctx.status.item()) == 0


def test_the_clamped_epilogue_equals_the_separate_step():
    """More than 128 tokens: bias and activation as the product's epilogue, to rounding the same as product, then step."""
    gen = torch.Generator().manual_seed(4)
    for tokens, k, ff in ((129, 64, 32), (300, 192, 272), (1000, 512, 528)):
        x = rounded(tokens, k, gen=gen)
        gate, up = rounded(ff, k, gen=gen, std=1.5 / k ** 0.5), rounded(ff, k, gen=gen, std=1.5 / k ** 0.5)
        bias = torch.randn(2 * ff, generator=gen)
        mixed = interleave_gate_up(gate, up)
        weight = ops.PackedWeight(mixed.to(DEV, torch.bfloat16))
        status = status_word()
        order = interleave_gate_up(torch.arange(ff).view(-1, 1), torch.arange(ff, 2 * ff).view(-1, 1)).view(-1)
        got = ops.gemm_tc_clamped(x.to(DEV, torch.bfloat16), weight, bias[order].to(DEV), status, limit=0.8, sigmoid_scale=1.702).float().cpu()
        want = plain.clamped_gate(x.double() @ gate.double().T + bias[:ff].double(), x.double() @ up.double().T + bias[ff:].double(), 0.8).float()
        assert torch.allclose(got, want, atol=1.5e-2, rtol=1e-2)
        product = torch.cat([x @ gate.T, x @ up.T], dim=1)
        for block, source, b in ((0, product, bias), (16, product[:, order], bias[order])):
            for splits in (1, 3):
                given = source.contiguous().to(DEV) if splits == 1 else partial_of(source.contiguous(), splits, gen, "split_k")
                for dtype in (torch.float32, torch.bfloat16):
                    step = ops.glu_bias(given, b.to(DEV), dtype, block=block, limit=0.8, sigmoid_scale=1.702).float().cpu()
                    tol = 1e-4 if dtype == torch.float32 else 1.5e-2
                    assert torch.allclose(step, want, atol=tol, rtol=tol)
        assert int(status.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,width,ff", [(5, 2, 72, 20), (1, 1, 64, 48), (3, 3, 64, 16), (8, 3, 128, 64), (40, 4, 64, 32), (6, 1, 128, 80)])
def test_experts_weighted_by_a_plain_softmax(dtype, experts, top, width, ff):
    gen = torch.Generator().manual_seed(experts * 10 + top)
    block = tiny.moe(experts, top, ff, 0.9)
    part = build_feed_forward(_feed_forward(block, "mlp"), width)
    W = weights_of(part, gen, "l0.mlp.")
    W["router"] *= 2.0
    give(part, W, dtype)
    assert (part.grouped is not None) == (dtype == torch.bfloat16 and top < experts and ff % 16 == 0 and ff >= 64)
    for rows in (1, 5, 64, 130, 400):
        x = rounded(rows, width, gen=gen)
        ctx = Ctx(dtype, all_decode=rows < 10)
        y = ops.materialize(part.forward(ctx, x.to(DEV, dtype))).float().cpu()
        close(y, plain.routed_ff(x.double(), double(W), block).float(), dtype, rows)
        assert int(ctx.status.item()) == 0
    # the chosen scores are shares of a softmax over all experts, their sum below one
    x = rounded(9, width, gen=gen)
    chosen, weights, dense = ops.moe_router(x.to(DEV), W["router"].to(DEV), top, over_all=2)
    scores = torch.softmax(x.double() @ W["router"].double().T, dim=-1)
    picked = torch.topk(scores, top)
    assert torch.allclose(weights.cpu(), picked.values.float(), atol=1e-5) and torch.equal(chosen.cpu().long(), picked.indices)
    assert torch.allclose(dense.cpu().sum(1), picked.values.sum(1).float(), atol=1e-5)


def test_a_routers_choice_is_sorted_like_a_table():
    gen = torch.Generator().manual_seed(2)
    for tokens, top, experts in ((1, 2, 5), (40, 3, 7), (100, 4, 64), (3000, 4, 16), (5000, 4, 16)):
        chosen = torch.rand(tokens, experts, generator=gen).argsort(dim=1)[:, :top].to(torch.int32).contiguous()
        x = rounded(tokens, 32, gen=gen)
        rows, offsets, where = ops.moe_dispatch(None, chosen.to(DEV), experts, x.to(DEV), status_word())
        counts = torch.bincount(chosen.view(-1).long(), minlength=experts)
        assert torch.equal(offsets.cpu().long(), torch.cat([torch.zeros(1, dtype=torch.long), counts.cumsum(0)]))
        assert torch.equal(rows.cpu()[where.cpu().long()], x[:, None].expand(-1, top, -1))
        owner = torch.searchsorted(offsets.cpu().long(), where.cpu().long(), right=True) - 1
        assert torch.equal(owner, chosen.long())


def test_combinations_no_kernel_takes_are_refused():
    with pytest.raises(ConfigError):
        build_feed_forward(_feed_forward(dict(kind="dense", ff=8, limit=-1.0), "mlp"), 16)
    ctx = Ctx(torch.float32)
    q = torch.zeros((1, 8), device=DEV)
    with pytest.raises(ops.KernelError, match="window"):
        ops.attention_sink(ctx, q, q, q, None, nq=1, nkv=1, dk=8, dv=8, scale=1.0, window=0, bias=None, sink=None, keep=3)


# ---------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (config, seed) in tiny.ALL.items():
        folder = tiny.write_model(tmp_path_factory.mktemp(f"difavik_{name}"), config, seed)
        _, tensors = tiny.tensors_for(config, seed)
        out[name] = (folder, config, tensors)
    return out


def prompt(config, n, seed):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def logits_of(config, W, tokens):
    return plain.forward(config, W, tokens).float()


def close_rows(got, want, dtype):
    """bfloat16: rounding the sublayers' inputs alone moves the plain model's rows by 0.005 to 0.014 in the median, and by up
    to 0.3 where it changes a router's close choice, so the bounds are on the median and on nine rows in ten."""
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if dtype == "float32":
        return bool(err.max() < 2e-4)
    good = err.median() < 0.04 and err.quantile(0.9) < 0.15 if len(err) >= 9 else err.max() < 0.4
    if not good:
        print("median", float(err.median()), "nine in ten", float(err.quantile(0.9)), "largest", float(err.max()))
    return bool(good)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_whole_prompt_portions_and_decoding_against_plain(models, name, dtype):
    folder, config, W = models[name]
    tokens = prompt(config, 157, 1)
    want = logits_of(config, W, tokens)
    for sizes in ((157,), (125,) + (1,) * 32, (2, 5, 1, 1, 17, 2, 3, 30, 96), (3, 2, 2, 150), (2,) * 78 + (1,)):
        page = tiny.PAGE[name]
        runner = ModelRunner(folder, dtype=dtype, num_pages=176 // page, page_size=page, max_requests=2)
        runner.begin("r")
        rows, at = [], 0
        for size in sizes:
            rows.append(runner.step([StepEntry("r", tokens[at:at + size], list(range(size)))]).cpu())
            at += size
        runner.check_status()
        assert close_rows(torch.cat(rows), want, dtype), sizes


WIDE = tiny.model(512, 1024, 1e-5, 101, 3, 8, [
    tiny.parallel(tiny.left(8, 2, 128, 0.09, 70, 20), tiny.right(4, 128, 128, 10000.0, 128, [0.97, 0.99, 0.999, 0.9]), tiny.moe(8, 2, 1024, 3.0)),
    tiny.lightning(8, 64, 128, [0.9] * 4 + [0.99] * 4, tiny.dense(2048, 3.0)),
])


def test_wide_layers_whose_products_split_their_inner_range(tmp_path):
    """Layer sizes at which the bfloat16 products of a few tokens split their inner range: the kernels after them add
    the unsummed splits (of both branches at once, of a dense product with its bias, of a token's experts, and of
    the recurrence's projection)."""
    lib = ops.library()
    assert lib.vosti_gemm_tc_splits(1, 1024, 1024) > 1 and lib.vosti_gemm_tc_grouped_splits(4, 8, 8, 1024, 1024) > 1
    folder = tiny.write_model(tmp_path / "wide", WIDE, 77)
    _, W = tiny.tensors_for(WIDE, 77)
    tokens = prompt(WIDE, 40, 8)
    want = logits_of(WIDE, W, tokens)
    for dtype in ("bfloat16", "float32"):
        runner = ModelRunner(folder, dtype=dtype, num_pages=4, page_size=16, max_requests=2)
        runner.begin("r")
        rows = [runner.step([StepEntry("r", tokens[:4], [0, 1, 2, 3])]).cpu()]
        rows += [runner.step([StepEntry("r", [t], [0])]).cpu() for t in tokens[4:]]
        runner.check_status()
        assert close_rows(torch.cat(rows), want, dtype), dtype


def test_a_checkpoint_without_the_unused_tensors_gives_the_same_logits(models, tmp_path):
    folder, config, W = models["a"]
    bare = tiny.write_model(tmp_path / "bare", config, tiny.ALL["a"][1], unused=False)
    tokens = prompt(config, 19, 3)
    rows = []
    for f in (folder, bare):
        runner = ModelRunner(f, dtype="float32", num_pages=8, page_size=8, max_requests=1)
        runner.begin("r")
        rows.append(runner.step([StepEntry("r", tokens, list(range(19)))]).cpu())
    assert torch.equal(rows[0], rows[1])


def test_first_tokens_of_a_sequence(models):
    """Requests of one, two and three tokens, and the first rows of a longer one: the pair table's last row, an empty
    state, a softmax over one key."""
    for name in ("a", "b", "c"):
        folder, config, W = models[name]
        page = tiny.PAGE[name]
        for dtype in ("float32", "bfloat16"):
            runner = ModelRunner(folder, dtype=dtype, num_pages=32 // page, page_size=page, max_requests=2)
            for n in (1, 2, 3, 9):
                tokens = prompt(config, n, 40 + n)
                for cut in ((n,), (1,) * n):
                    runner.begin("r")
                    rows, at = [], 0
                    for size in cut:
                        rows.append(runner.step([StepEntry("r", tokens[at:at + size], list(range(size)))]).cpu())
                        at += size
                    runner.finish("r")
                    assert close_rows(torch.cat(rows), logits_of(config, W, tokens), dtype), (name, n, cut)
            runner.check_status()


def test_residual_stream_after_every_layer(models):
    for name in ("a", "b", "c"):
        folder, config, W = models[name]
        tokens = prompt(config, 23, 2)
        want = []
        plain.forward(config, W, tokens, streams=want)
        page = tiny.PAGE[name]
        runner = ModelRunner(folder, dtype="float32", num_pages=32 // page, page_size=page, max_requests=1)
        streams = []
        for block in runner.model.blocks:
            inner = block.forward

            def watched(ctx, hidden, residual, cache, writes_cache=True, inner=inner):
                out, rest = inner(ctx, hidden, residual, cache, writes_cache)
                streams.append(out.stream.cpu().clone())
                return out, rest
            block.forward = watched
        runner.begin("r")
        runner.step([StepEntry("r", tokens, [0])])
        assert len(streams) == len(want) == len(config["layers"])
        for i, (got, expected) in enumerate(zip(streams, want)):
            assert torch.allclose(got, expected.float(), atol=5e-4, rtol=3e-4), (name, i)


@pytest.mark.parametrize("name,dtype", [("a", "float32"), ("b", "float32"), ("c", "float32"), ("c", "bfloat16"), ("a", "bfloat16")])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(models, name, dtype):
    """Four requests through two request slots and a pool that holds two of them: portions of some beside single
    tokens of others; every request equals itself alone."""
    folder, config, W = models[name]
    lengths = {"a": 37, "b": 9, "c": 1, "d": 26}
    tokens = {r: prompt(config, n, 10 + i) for i, (r, n) in enumerate(lengths.items())}
    want = {r: logits_of(config, W, t) for r, t in tokens.items()}
    page = tiny.PAGE[name]
    pool = 80 // page
    runner = ModelRunner(folder, dtype=dtype, num_pages=pool, page_size=page, max_requests=2)
    schedule = [
        [("a", 5), ("b", 2)], [("a", 1), ("b", 6)], [("b", 1), ("a", 20)], [("a", 1)],      # b ends in step 2
        [("c", 1), ("a", 1)], [("d", 1), ("a", 1)], [("d", 1), ("a", 8)], [("d", 1)], [("d", 23)],     # c, then a end
    ]
    at = {r: 0 for r in lengths}
    got = {r: [] for r in lengths}
    for step in schedule:
        entries = []
        for r, n in step:
            if r not in runner.cache.live:
                runner.begin(r)
            entries.append(StepEntry(r, tokens[r][at[r]:at[r] + n], list(range(n))))
        logits = runner.step(entries).cpu()
        row = 0
        for r, n in step:
            got[r].append(logits[row:row + n])
            row += n
            at[r] += n
            if at[r] == lengths[r]:
                runner.finish(r)
    runner.check_status()
    runner.cache.check()
    for r in lengths:
        assert at[r] == lengths[r]
        assert close_rows(torch.cat(got[r]), want[r], dtype), r
    assert runner.cache.available_pages() == pool


@pytest.mark.parametrize("name,dtype", [("a", "float32"), ("b", "float32"), ("c", "float32"), ("c", "bfloat16")])
def test_long_decoding_past_every_window(models, name, dtype):
    """A prompt, then token by token far past every window, with a pool that holds little more than the widest one and
    the kept first tokens: pages come back and are used again, those of the kept tokens do not."""
    folder, config, W = models[name]
    total = {"a": 260, "b": 120, "c": 560}[name]
    tokens = prompt(config, total, 4)
    want = logits_of(config, W, tokens)
    page = tiny.PAGE[name]
    first = max(w for w, _ in tiny.windows(config)) + 5
    kept = max(-(-k // page) * page for _, k in tiny.windows(config))
    pool = (first + kept + 2 * page) // page + 1
    assert pool * page < total
    runner = ModelRunner(folder, dtype=dtype, num_pages=pool, page_size=page, max_requests=1)
    runner.begin("r")
    rows = [runner.step([StepEntry("r", tokens[:first], list(range(first)))]).cpu()]
    rows += [runner.step([StepEntry("r", [t], [0])]).cpu() for t in tokens[first:]]
    runner.check_status()
    runner.cache.check()
    assert close_rows(torch.cat(rows), want, dtype)
    runner.finish("r")
    assert runner.cache.available_pages() == pool


@pytest.mark.parametrize("name,dtype,binary", [("a", "float32", True), ("c", "bfloat16", False), ("b", "float32", False), ("c", "float32", False)])
def test_trace_replay_of_a_mixed_schedule(models, name, dtype, binary, tmp_path):
    """The trace runner (the program itself, and the class it wraps) over a schedule of up to four live requests,
    portions beside single tokens, requests that sit a step out and a pool smaller than the sum of all requests:
    every row against the plain implementation of the request alone."""
    import numpy as np
    import replay_util as R
    folder, config, W = models[name]
    requests = {f"q{i}": prompt(config, n, 60 + i) for i, n in enumerate([70, 40, 33, 90, 64, 21])}
    steps = R.number(R.mixed_steps(requests, seed=5))
    max_tokens = R.max_live_tokens(steps)
    assert max_tokens < sum(R.roundup64(len(t)) for t in requests.values())
    if binary:
        R.run_binary(folder, dtype, steps, max_tokens, tmp_path)
    else:
        R.run_in_process(folder, dtype, steps, max_tokens, tiny.PAGE[name], tmp_path)
    rows = R.collect(steps, tmp_path, config["vocab"])
    assert len(rows) == sum(len(t) for t in requests.values())
    for rid, tokens in requests.items():
        got = torch.from_numpy(np.stack([rows[(rid, p)] for p in range(len(tokens))]))
        assert close_rows(got, logits_of(config, W, tokens), dtype), rid


@pytest.mark.parametrize("mode", ["decode", "full"])
def test_batch_invariant_modes_stay_within_the_bounds(models, mode, tmp_path):
    """With one order of arithmetic asked for, the recurrence goes token by token and the attention by portions alone."""
    import numpy as np
    import replay_util as R
    folder, config, W = models["c"]
    tokens = prompt(config, 90, 31)
    cuts = ([90], [2, 40, 1, 30, 17])
    got = []
    for n, sizes in enumerate(cuts):
        at, steps = 0, []
        for size in sizes:
            steps.append({"entries": [{"id": "r", "tokens": tokens[at:at + size], "want": list(range(size))}], "end": ["r"] if at + size == 90 else []})
            at += size
        steps = R.number(steps)
        try:
            R.run_in_process(folder, "bfloat16", steps, 128, 16, tmp_path / str(n), batch_invariant=mode)
        finally:
            ops.set_invariance("off")
        rows = R.collect(steps, tmp_path / str(n), config["vocab"])
        got.append(torch.from_numpy(np.stack([rows[("r", p)] for p in range(90)])))
        assert close_rows(got[-1], logits_of(config, W, tokens), "bfloat16")
    if mode == "full":
        assert torch.equal(got[0], got[1])


def plain_greedy(config, W, tokens, new_tokens):
    tokens, out = list(tokens), []
    for _ in range(new_tokens):
        out.append(int(plain.forward(config, W, tokens)[-1].argmax()))
        tokens.append(out[-1])
    return out


@pytest.mark.parametrize("name,cuda_graphs,async_scheduling", [("a", False, False), ("a", True, False), ("a", True, True), ("c", True, True)])
def test_greedy_generation_through_the_engine(models, name, cuda_graphs, async_scheduling):
    """The framework's own entry point: scheduler, portions under a token budget, CUDA graphs for decode steps (whose
    pair rows follow from tokens the host has not read), two slots for five requests, so few pages that a request is
    preempted and computed again from its first token."""
    folder, config, W = models[name]
    prompts = [prompt(config, n, 20 + n) for n in (5, 17, 2, 11, 8)]
    want = [plain_greedy(config, W, p, 10) for p in prompts]
    blocks, size = (9, 4) if name == "a" else (3, 16)
    engine = Engine(folder, dtype="float32", num_blocks=blocks, block_size=size, max_num_seqs=2, max_num_batched_tokens=16,
                    prefill_chunk_size=8 if name == "a" else 16, cuda_graphs=cuda_graphs, async_scheduling=async_scheduling)
    assert engine.runner.spec.architecture == "Difavik" and engine.runner.cache.has_state
    assert (engine.graphs is not None) == cuda_graphs
    got = engine.generate(prompts, max_tokens=10, arrival_steps=[0, 0, 1, 4, 20])
    assert got == want
    if name == "a":
        assert engine.scheduler.preemptions > 0
    if cuda_graphs:
        assert engine.graphs.replays > 0
    engine.runner.cache.check()
    assert engine.runner.cache.available_pages() == blocks


def test_graphs_give_the_bfloat16_engine_the_same_tokens(models):
    """bfloat16 serving through the grouped products and fused steps, with and without recorded decode steps."""
    folder, config, W = models["c"]
    prompts = [prompt(config, n, 70 + n) for n in (12, 30, 7)]
    tokens = []
    for cuda_graphs in (False, True):
        engine = Engine(folder, dtype="bfloat16", num_blocks=12, block_size=16, max_num_seqs=3, max_num_batched_tokens=64,
                        cuda_graphs=cuda_graphs, async_scheduling=cuda_graphs)
        tokens.append(engine.generate(prompts, max_tokens=16))
        if cuda_graphs:
            assert engine.graphs.replays > 0
    assert tokens[0] == tokens[1]


def test_the_command_line_generates_from_a_difavik_folder(models, capsys):
    from vosti_b200.engine import cli
    folder, config, W = models["b"]
    tokens = prompt(config, 6, 9)
    want = plain_greedy(config, W, tokens, 4)
    code = cli.main(["--model", folder, "--dtype", "float32", "--prompt-ids", ",".join(map(str, tokens)), "--max-tokens", "4"])
    assert code in (0, None)
    assert ",".join(map(str, want)) in capsys.readouterr().out.replace(" ", "")
