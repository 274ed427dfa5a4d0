"""The kernels of Legilix's mechanisms alone, each against a plain float64 restatement (tests/plain_legilix.py), with
inputs made so that a fault shows: queries that point at ONE key each (just inside a window and just outside it, the
last kept token and the first one that is not kept, keys hundreds of positions back), over pages out of order, as
portions of a prompt and decoded alone; a matrix over the heads' scores with entries of both signs; distance biases
from weak to strong on every attention kernel that takes one; the gate per head; norms in groups; the ungated
feed-forward's product; routing weights on the experts' inputs."""

import pytest
import torch

from plain_legilix import (F64, distance_bias, gelu_tanh, grouped_rms_norm, mix_scores, raw_scores, rms_unit, rotate_halves, silu,
                           softmax_over, weigh_values, window_mask)

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _i32(values, device):
    return torch.tensor(list(values), dtype=torch.int32, device=device)


def _case(seed, T, H, G, d, dv, targets, sharp=24.0):
    """q [T, H, d], k [T, G, d], v [T, G, dv] of unit-size values in which query head 0 at position p points at key
    ``targets[p]`` of its key/value head with a score of about ``sharp`` before scaling."""
    g = torch.Generator().manual_seed(seed)
    q, k, v = torch.randn(T, H, d, generator=g), torch.randn(T, G, d, generator=g), torch.randn(T, G, dv, generator=g)
    q *= 2.0 * d ** -0.5
    for p, target in targets.items():
        q[p, 0] = k[target, 0] * (sharp / float(k[target, 0].pow(2).sum()))
    return q, k, v


class Stored:
    """One request's keys and values in pages out of order, written by the engine's own kernel portion by portion."""

    def __init__(self, device, dtype, q, k, v, page):
        from zephyr_b200.kernels import ops

        self.device, self.dtype, self.page = device, DTYPES[dtype], page
        (self.T, self.H, self.d), self.G, self.dv = q.shape, k.shape[1], v.shape[2]
        g = torch.Generator().manual_seed(self.T + page)
        blocks = -(-self.T // page)
        self.table = (torch.randperm(blocks, generator=g) + 1).to(torch.int32).view(1, -1).to(device)
        cache = torch.full((blocks + 1, page * self.G * (self.d + self.dv)), float("nan"), dtype=self.dtype, device=device)
        self.cache = cache.view(blocks + 1, 2, self.G, page, self.d) if self.d == self.dv else cache
        self.status = ops.new_status(device)
        self.projected = torch.cat([q.reshape(self.T, -1), k.reshape(self.T, -1), v.reshape(self.T, -1)], dim=1).float().to(device)

    def write(self, at, n, **norms):
        from zephyr_b200.kernels import ops

        args = dict(norm="none", q_w=None, k_w=None, eps=1e-6, freqs=None, dims=0, mult=1.0, bias=None)
        args.update(norms)
        pos = torch.arange(at, at + n, dtype=torch.int32, device=self.device)
        return ops.qkv_halves(self.projected[at:at + n], self.H, self.G, self.d, self.dv, args["norm"], args["q_w"], args["k_w"],
                              args["eps"], args["freqs"], args["dims"], args["mult"], False, pos,
                              torch.zeros(n, dtype=torch.int32, device=self.device), self.cache, self.table, self.status, self.dtype,
                              bias=args["bias"])

    def rows(self, at, n):
        return _i32([0], self.device), _i32([n], self.device), _i32([at], self.device)

    def tiles(self, n, tokens):
        q0 = torch.arange(0, n, tokens, dtype=torch.int32, device=self.device)
        return torch.zeros_like(q0), q0


def _run(stored, portions, kernel, *, window, scale, keep_first=0, mix=None, bias=None):
    """Attention of every portion on the named kernel."""
    from zephyr_b200.kernels import ops

    s, outs, at = stored, [], 0
    for n in portions:
        q = s.write(at, n)
        rows = s.rows(at, n)
        masks = dict(keep_first=keep_first) if keep_first else {}
        if bias is not None:
            masks["distance_bias"] = bias
        out = torch.full((n, s.H * s.dv), float("nan"), dtype=s.dtype, device=s.device)
        if kernel == "general":
            tile = ops.attention_tile_tokens(s.H // s.G)
            out = ops.paged_attention(q, s.cache, s.table, *s.tiles(n, tile), tile, *rows, s.H, s.G, s.d, window, scale, s.status,
                                      value_dim=s.dv, score_mix=mix, **masks)
        elif kernel == "heads":
            tile = 1 if n == 1 else ops.heads_attention_tile_tokens(s.H, s.G, s.d, s.dv, s.dtype)
            # (a single token's keys by as many CTAs as the kernel chooses, by one, by more than there are tiles)
            splits = [None, 1, 3, 40][at % 4] if n == 1 else None
            ops.heads_attention(q, s.cache, s.table, *s.tiles(n, tile), *rows, s.H, s.G, s.d, s.dv, window, scale, s.status, out,
                                score_mix=mix, single=n == 1, max_context=at + n, splits=splits, **masks)
        elif kernel == "prompt" or n > 1:
            tile = ops.paged_prefill_tile_tokens()
            ops.paged_prefill(q, s.cache, s.table, *s.tiles(n, tile), *rows, s.H, s.G, s.d, window, scale, s.status, out,
                              by_group=kernel == "prompt" and n == 1 and s.H // s.G <= 16, **masks)
        else:
            split = [None, 0, 32, 128][at % 4]          # balanced items and fixed splits
            ops.paged_decode(q, s.cache, s.table, _i32([0], s.device), rows[0], rows[2], at + 1, s.H, s.G, s.d, window, scale,
                             s.status, out, split_size=split, **masks)
        outs.append(out)
        at += n
    ops.check_status(s.status)
    return torch.cat(outs).cpu().double()


def _expected(dtype, q, k, v, visible, scale, mix=None, bias=None):
    """float64, from queries, keys and values as the engine holds them (rounded to its type)."""
    q, k, v = (t.to(DTYPES[dtype]).double() for t in (q, k, v))
    scores = raw_scores(q, k, scale)
    if mix is not None:
        scores = mix_scores(scores, mix.double())
    if bias is not None:
        scores = scores - distance_bias(q.shape[0], *(b.double() for b in bias))
    return weigh_values(softmax_over(scores, visible), v).reshape(q.shape[0], -1)


PORTIONS = ([293] + [1] * 40, [7, 2, 150, 1, 1, 90, 2] + [1] * 20 + [60])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,size,keep,page", [
    (4, 2, 24, 40, 90, 22, 16), (3, 1, 20, 12, 23, 7, 16), (8, 4, 32, 32, 9, 0, 16), (5, 5, 16, 24, 70, 33, 32),
    (12, 4, 128, 96, 33, 40, 16), (16, 8, 128, 128, 64, 16, 16), (3, 1, 64, 64, 5, 1, 64), (32, 2, 16, 16, 300, 4, 16),
    (6, 2, 32, 64, 70, 65, 16), (2, 2, 160, 136, 64, 64, 32), (10, 5, 250, 30, 48, 3, 16), (32, 8, 128, 128, 40, 11, 16),
    (17, 1, 64, 40, 30, 9, 16), (34, 2, 32, 32, 21, 3, 16), (1, 1, 9, 7, 17, 2, 16), (7, 7, 64, 64, 1, 0, 16)])
def test_scores_mixed_ahead_of_the_softmax(cuda_device, dtype, H, G, d, dv, size, keep, page):
    """Queries of head 0 point at the last kept token, the first one that is not kept, the edges of the window and the
    first token; the matrix gives every head a share of head 0's scores."""
    from zephyr_b200.kernels import ops

    T, scale = 333, 0.8
    targets = {p: min(max([keep - 1, keep, p - size + 1, p - size, 0, p - 1][p % 6], 0), p) for p in range(T - 60, T)}
    q, k, v = _case(H * 100 + size + keep, T, H, G, d, dv, targets)
    g = torch.Generator().manual_seed(keep + H)
    mix = torch.eye(H) * 0.7 + torch.randn(H, H, generator=g) * (0.25 if H <= 8 else 0.1)
    mix[:, 0] = torch.where(mix[:, 0] < 0, -0.6, 0.6)
    visible = window_mask(T, size, keep)
    expected = _expected(dtype, q, k, v, visible, scale, mix)
    bound = (4e-5 if dtype == "float32" else 0.03) * max(1.0, float(expected.abs().max()))
    # In bfloat16 the general kernel and the tensor-core one; in float32 the general kernel alone.
    kernels = ["general"]
    tile = ops.heads_attention_tile_tokens(H, G, d, dv, DTYPES[dtype])
    assert (tile > 0) == (dtype == "bfloat16" and H <= 32)
    if tile:
        kernels.append("heads")
    for kernel in kernels:
        for portions in PORTIONS:
            stored = Stored(cuda_device, dtype, q, k, v, page)
            got = _run(stored, portions, kernel, window=size, scale=scale, keep_first=keep, mix=mix.to(cuda_device))
            assert torch.isfinite(got).all(), kernel
            assert (got - expected).abs().max() < bound, (kernel, portions[:3], (got - expected).abs().max())
    # What is pointed at decides: each of these mistakes would not pass.
    mistakes = {"one key less kept": _expected(dtype, q, k, v, window_mask(T, size, keep - 1), scale, mix) if keep and size + keep < T - 60 else None,
                "one key more kept": _expected(dtype, q, k, v, window_mask(T, size, keep + 1), scale, mix) if size + keep < T - 60 else None,
                "a window one shorter": _expected(dtype, q, k, v, window_mask(T, size - 1, keep), scale, mix) if size > 1 and size + keep < T else None,
                "a window one longer": _expected(dtype, q, k, v, window_mask(T, size + 1, keep), scale, mix) if size + keep < T - 60 else None,
                "no mixing": _expected(dtype, q, k, v, visible, scale) if size > 1 else None,
                "the matrix transposed": _expected(dtype, q, k, v, visible, scale, mix.T.contiguous()) if size > 1 and H > 1 else None}
    for name, wrong in mistakes.items():
        if wrong is not None:
            assert (wrong - expected).abs().max() > 5 * bound, name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,size,page", [
    (4, 2, 32, 32, 44, 16), (3, 1, 24, 40, 19, 16), (8, 1, 64, 64, 100, 32), (4, 2, 128, 128, 150, 16), (6, 6, 128, 128, 33, 64),
    (17, 1, 64, 64, 60, 16), (2, 2, 96, 96, 1, 16), (5, 5, 20, 20, 9, 16), (4, 1, 256, 256, 64, 16), (12, 3, 40, 64, 70, 32),
    (33, 3, 12, 8, 25, 16)])
def test_a_logarithmic_bias_on_the_distance(cuda_device, dtype, H, G, d, dv, size, page):
    """On every kernel that takes the layer: the general one, the prompt kernels (mma.sync and, at head size 128,
    tcgen05; single tokens as tiles of a group's heads), the split-context kernel with balanced and fixed splits, and
    the kernel with all heads in one CTA.  The queries point at the window's edges and at keys between."""
    from zephyr_b200.kernels import ops

    T, scale = 333, 0.7
    targets = {p: min(max([p - size + 1, p - size, p - size // 2, p, p - 1, p - size + 2][p % 6], 0), p) for p in range(T - 60, T)}
    q, k, v = _case(H * 10 + size, T, H, G, d, dv, targets, sharp=12.0)
    g = torch.Generator().manual_seed(size)
    r1, r2 = torch.rand(H, generator=g) * 2.0 + 0.05, torch.rand(H, generator=g) * 0.6 + 0.02
    visible = window_mask(T, size)
    expected = _expected(dtype, q, k, v, visible, scale, bias=(r1, r2))
    bound = (4e-5 if dtype == "float32" else 0.03) * max(1.0, float(expected.abs().max()))
    bias = (r1.to(cuda_device), r2.to(cuda_device))
    kernels = ["general"]
    if dtype == "bfloat16":
        if d == dv and ops.paged_prefill_supported(H, G, d, torch.bfloat16):
            kernels.append("prompt")
        if d == dv and ops.paged_decode_supported(H, G, d, torch.bfloat16):
            kernels.append("decode")
        if ops.heads_attention_tile_tokens(H, G, d, dv, torch.bfloat16):
            kernels.append("heads")
        assert len(kernels) > 1 or H > 32
    for kernel in kernels:
        for tcgen05 in ([True, False] if kernel == "prompt" and d == 128 else [True]):
            ops.USE_TCGEN05_PREFILL = tcgen05
            try:
                for portions in PORTIONS:
                    stored = Stored(cuda_device, dtype, q, k, v, page)
                    got = _run(stored, portions, kernel, window=size, scale=scale, bias=bias)
                    assert torch.isfinite(got).all(), kernel
                    assert (got - expected).abs().max() < bound, (kernel, tcgen05, portions[:3], (got - expected).abs().max())
            finally:
                ops.USE_TCGEN05_PREFILL = True
    if size > 1:
        for name, wrong in {"no bias": _expected(dtype, q, k, v, visible, scale),
                            "a distance one longer": _expected(dtype, q, k, v, visible, scale, bias=(r1 * 1.3, r2)),
                            "a window one shorter": _expected(dtype, q, k, v, window_mask(T, size - 1), scale, bias=(r1, r2)),
                            "a window one longer": _expected(dtype, q, k, v, window_mask(T, size + 1), scale, bias=(r1, r2))}.items():
            assert (wrong - expected).abs().max() > 2 * bound, name


@pytest.mark.parametrize("H,G,d,dv", [(8, 2, 32, 48), (16, 4, 64, 64), (4, 4, 128, 128)])
def test_mixed_scores_and_a_distance_bias_together(cuda_device, H, G, d, dv):
    """Another design's combination, without a window: the bias comes behind the mixing."""
    T, scale = 200, 0.5
    q, k, v = _case(H, T, H, G, d, dv, {})
    g = torch.Generator().manual_seed(H)
    mix = torch.eye(H) + torch.randn(H, H, generator=g) * 0.3
    bias = (torch.rand(H, generator=g) + 0.2, torch.rand(H, generator=g) * 0.4 + 0.1)
    for dtype, kernel in (("float32", "general"), ("bfloat16", "general"), ("bfloat16", "heads")):
        expected = _expected(dtype, q, k, v, window_mask(T, T), scale, mix, bias)
        stored = Stored(cuda_device, dtype, q, k, v, 16)
        got = _run(stored, [100, 1, 1, 66, 1, 31], kernel, window=0, scale=scale, mix=mix.to(cuda_device),
                   bias=tuple(b.to(cuda_device) for b in bias))
        assert (got - expected).abs().max() < (4e-5 if dtype == "float32" else 0.03) * max(1.0, float(expected.abs().max())), (dtype, kernel)


def test_unequal_requests_in_one_launch_against_each_alone(cuda_device):
    """Four requests of a batch (a long one, a short one, one of a single token, one with a far context) in one launch
    of tiles give the bits each gives alone."""
    from zephyr_b200.kernels import ops

    H, G, d, dv, window, keep, page = 12, 4, 32, 48, 40, 6, 16
    lengths, contexts = [50, 3, 1, 20], [0, 90, 0, 140]
    g = torch.Generator().manual_seed(5)
    mix = (torch.eye(H) + torch.randn(H, H, generator=g) * 0.2).to(cuda_device)
    total = [n + c for n, c in zip(lengths, contexts)]
    blocks = [-(-t // page) for t in total]
    table = torch.zeros(4, max(blocks), dtype=torch.int32)
    order = (torch.randperm(sum(blocks), generator=g) + 1).to(torch.int32)
    at = 0
    for r, n in enumerate(blocks):
        table[r, :n] = order[at:at + n]
        at += n
    table = table.to(cuda_device)
    cache = torch.randn(sum(blocks) + 1, page * G * (d + dv), generator=g).to(torch.bfloat16).to(cuda_device)
    q = torch.randn(sum(lengths), H * d, generator=g).to(torch.bfloat16).to(cuda_device)
    starts = [sum(lengths[:i]) for i in range(4)]
    rows = tuple(_i32(x, cuda_device) for x in (starts, lengths, contexts))
    status = ops.new_status(cuda_device)
    tokens = ops.heads_attention_tile_tokens(H, G, d, dv, torch.bfloat16)

    def run(which, single=False, splits=None):
        out = torch.zeros(sum(lengths), H * dv, dtype=torch.bfloat16, device=cuda_device)
        tiles = [(r, q0) for r in which for q0 in range(0, lengths[r], 1 if single else tokens)]
        ops.heads_attention(q, cache, table, _i32([t[0] for t in tiles], cuda_device), _i32([t[1] for t in tiles], cuda_device), *rows,
                            H, G, d, dv, window, 0.3, status, out, keep_first=keep, score_mix=mix, single=single, max_context=160,
                            splits=splits)
        return out

    together = run(range(4))
    for r in range(4):
        part = slice(starts[r], starts[r] + lengths[r])
        assert torch.equal(run([r])[part], together[part]), r
    # the same rows as single tokens, over one CTA each and over several: the same result up to rounding
    for splits in (1, 2, 5):
        alone = run([2], single=True, splits=splits)[starts[2]:starts[2] + 1]
        assert (alone.float() - together[starts[2]:starts[2] + 1].float()).abs().max() < 0.02
    ops.check_status(status)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,dims,scaling", [
    (4, 2, 32, 32, 16, {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 0.5}), (3, 1, 24, 40, 24, None),
    (6, 6, 20, 12, 2, {"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 1.0}), (2, 1, 128, 64, 64, {"factor": 40.0, "original": 30, "fast": 3.0, "slow": 0.1})])
def test_biases_then_norms_then_the_yarn_rotation(cuda_device, dtype, H, G, d, dv, dims, scaling):
    """Queries as they come out of the kernel, keys and values through attention over one and two keys."""
    from plain_legilix import yarn

    T, eps = 150, 1e-5
    g = torch.Generator().manual_seed(H * d + dims)
    q, k, v = (torch.randn(T, H, d, generator=g) * 2.0, torch.randn(T, G, d, generator=g) * 0.5, torch.randn(T, G, dv, generator=g) * 3.0)
    bias = torch.randn(H * d + G * (d + dv), generator=g)
    q_w, k_w = torch.randn(d, generator=g) * 0.3 + 1.0, torch.randn(d, generator=g) * 0.3 + 1.0
    rot = {"base": 300.0, "dims": dims, "scaling": scaling}
    qb, kb, vb = bias[:H * d].view(H, d), bias[H * d:H * d + G * d].view(G, d), bias[H * d + G * d:].view(G, dv)
    positions = torch.arange(T)
    qn = rotate_halves(rms_unit((q + qb).double(), eps) * q_w.double(), positions, rot)
    kn = rotate_halves(rms_unit((k + kb).double(), eps) * k_w.double(), positions, rot)
    vn = (v + vb).double()
    freqs, mult = yarn(rot)
    norms = dict(norm="per_head", q_w=q_w.to(cuda_device), k_w=k_w.to(cuda_device), eps=eps, freqs=freqs.float().to(cuda_device),
                 dims=dims, mult=mult, bias=bias.to(cuda_device))
    stored = Stored(cuda_device, dtype, q, k, v, 16)
    queries = torch.cat([stored.write(at, n, **norms) for at, n in ((0, 100), (100, 1), (101, 49))]).cpu().double().view(T, H, d)
    assert (queries - qn).abs().max() < (3e-5 if dtype == "float32" else 2.0 ** -8) * float(qn.abs().max())
    from zephyr_b200.kernels import ops
    for window in (1, 2):
        tile = ops.attention_tile_tokens(H // G)
        got = ops.paged_attention(queries.to(DTYPES[dtype]).reshape(T, -1).contiguous().to(cuda_device), stored.cache, stored.table,
                                  *stored.tiles(T, tile), tile, *stored.rows(0, T), H, G, d, window, 0.2, stored.status, value_dim=dv)
        expected = _expected(dtype, qn.float(), kn.float(), vn.float(), window_mask(T, window), 0.2)
        assert (got.cpu().double() - expected).abs().max() < (5e-5 if dtype == "float32" else 0.04) * max(1.0, float(expected.abs().max()))
    ops.check_status(stored.status)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,vd", [(3, 20), (16, 64), (1, 7)])
def test_the_gate_of_a_head(cuda_device, dtype, heads, vd):
    from zephyr_b200.kernels import ops

    g = torch.Generator().manual_seed(heads)
    x = torch.randn(70, heads * vd, generator=g).to(DTYPES[dtype])
    wide = torch.randn(70, 90 + heads, generator=g) * 3.0
    got = ops.sigmoid_gate(x.clone().to(cuda_device), wide.to(cuda_device)[:, 90:])
    expected = x.double() * torch.sigmoid(wide[:, 90:].double()).repeat_interleave(vd, dim=1)
    assert (got.cpu().double() - expected).abs().max() < (1e-6 if dtype == "float32" else 2.0 ** -8) * float(expected.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,groups", [(60, 3), (256, 4), (257, 1), (1024, 8), (1030, 2), (9000, 2), (48, 48), (4100, 1)])
def test_a_norm_in_groups_joined_to_the_sum(cuda_device, dtype, width, groups):
    """Parts of very different size, so that one statistic for the whole row would be far off."""
    from zephyr_b200.kernels import ops

    g = torch.Generator().manual_seed(width + groups)
    rows, eps = 37, 1e-5
    sizes = torch.logspace(-1, 2, groups).repeat_interleave(width // groups)
    stream = torch.randn(rows, width, generator=g) * sizes
    delta = (torch.randn(rows, width, generator=g) * sizes).to(DTYPES[dtype])
    w = torch.randn(width, generator=g) * 0.2 + 1.0
    for summand in (None, delta):
        x = stream.clone().to(cuda_device)
        out = ops.sum_rms_norm(x, summand.to(cuda_device) if summand is not None else None, None, w.to(cuda_device), eps,
                               out_dtype=DTYPES[dtype], groups=groups)
        total = stream.double() + (summand.double() if summand is not None else 0.0)
        expected = grouped_rms_norm(total, w.double(), groups, eps)
        assert ((x.cpu().double() - total).abs() < 1e-6 * sizes.double() * 10).all()
        assert out.dtype == DTYPES[dtype]
        assert (out.cpu().double() - expected).abs().max() < (1e-5 if dtype == "float32" else 2.0 ** -8) * float(expected.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,width,ff", [(1, 64, 96), (7, 60, 100), (16, 256, 512), (40, 128, 72), (300, 96, 200), (513, 128, 264), (1100, 256, 1000)])
def test_the_ungated_feed_forward(cuda_device, dtype, rows, width, ff):
    """Few rows, many rows and rows between: the activation in the product's epilogue and behind it."""
    from zephyr_b200.config.spec import FeedForwardSpec
    from zephyr_b200.parts import UngatedFeedForward

    g = torch.Generator().manual_seed(rows + ff)
    x = (torch.randn(rows, width, generator=g) * 1.5).to(DTYPES[dtype])
    up, down = (torch.randn(ff, width, generator=g) * width ** -0.5).to(DTYPES[dtype]), (torch.randn(width, ff, generator=g) * ff ** -0.5).to(DTYPES[dtype])
    part = UngatedFeedForward(FeedForwardSpec("ungated", {"hidden_size": width, "intermediate_size": ff, "up_proj": "u", "down_proj": "d"}),
                              {"u": up.to(cuda_device), "d": down.to(cuda_device)}, DTYPES[dtype])
    got = part.forward(x.to(cuda_device)).cpu().double()
    expected = gelu_tanh(x.double() @ up.double().T) @ down.double().T
    assert (got - expected).abs().max() < (2e-5 if dtype == "float32" else 2.0 ** -6) * float(expected.abs().max())


def test_gelu_far_from_zero_and_in_every_form(cuda_device):
    from zephyr_b200.kernels import ops

    z = torch.cat([torch.linspace(-12.0, 12.0, 1001), torch.tensor([-1e4, 1e4, 0.0])])
    got = ops.act_rows(z.to(cuda_device), "gelu_tanh").cpu().double()
    assert (got - gelu_tanh(z.double())).abs().max() < 2e-6 and float(got[-3]) == 0.0 and float(got[-2]) == 1e4
    rounded = ops.act_rows(z.to(cuda_device), "gelu_tanh", torch.bfloat16).cpu().double()
    assert ((rounded - gelu_tanh(z.double())).abs() <= 2.0 ** -8 * gelu_tanh(z.double()).abs() + 1e-6).all()
    g = torch.Generator().manual_seed(1)
    w = (torch.randn(304, 64, generator=g) * 0.4).to(torch.bfloat16)
    x = torch.randn(600, 64, generator=g).to(torch.bfloat16)
    expected = gelu_tanh(x.double() @ w.double().T)
    for block_n in (0, 2, 128, 256):
        y = ops.gemm_tc(x.to(cuda_device), w.to(cuda_device), product_act="gelu_tanh", block_n=block_n).cpu().double()
        assert ((y - expected).abs() <= 2.0 ** -8 * expected.abs() + 2e-5).all()
    y = ops.gemm_small(x[:9].to(cuda_device), w.to(cuda_device), product_act="gelu_tanh").cpu().double()
    assert ((y - expected[:9]).abs() <= 2.0 ** -8 * expected[:9].abs() + 2e-5).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens,experts,top,width,ff", [(1, 4, 2, 64, 48), (33, 5, 1, 40, 24), (200, 3, 3, 64, 64), (700, 8, 2, 128, 136), (50, 6, 4, 60, 27)])
def test_routing_weights_on_the_experts_inputs(cuda_device, dtype, tokens, experts, top, width, ff):
    """expert(s x) with scores from near zero to near one, on every path of the products: the grouped tcgen05 launch,
    tiles on mma.sync, CUDA cores, both layouts of the matrices."""
    from zephyr_b200.kernels import ops

    g = torch.Generator().manual_seed(tokens + experts)
    cast = lambda t: t.to(DTYPES[dtype])
    x = cast(torch.randn(tokens, width, generator=g) * 2.0)
    gate, up = (cast(torch.randn(experts, ff, width, generator=g) * 2.0 * width ** -0.5) for _ in range(2))
    down = cast(torch.randn(experts, width, ff, generator=g) * ff ** -0.5)
    logits = torch.randn(tokens, experts, generator=g) * 2.5
    ids, weights = ops.route(logits.to(cuda_device), None, top, "sigmoid")
    chosen = torch.topk(logits, top, dim=1)
    assert torch.equal(ids.cpu().long(), chosen.indices)
    assert (weights.cpu().double() - torch.sigmoid(chosen.values.double())).abs().max() < 1e-6
    expected = torch.zeros(tokens, width, dtype=F64)
    outputs = torch.zeros(tokens, width, dtype=F64)
    for j in range(top):
        for e in range(experts):
            t = (chosen.indices[:, j] == e).nonzero().flatten()
            s = torch.sigmoid(chosen.values[t, j].double()).unsqueeze(1)
            run = lambda h: (silu(h @ gate[e].double().T) * (h @ up[e].double().T)) @ down[e].double().T
            expected.index_add_(0, t, run(s * x[t].double()))
            outputs.index_add_(0, t, s * run(x[t].double()))
    bound = (3e-5 if dtype == "float32" else 2.0 ** -6) * float(expected.abs().max())
    dev = lambda t: t.contiguous().to(cuda_device)
    forms = [("apart", dev(gate), dev(up))]
    if ff % 8 == 0:
        forms.append(("interleaved", ops.interleave_gate_up(dev(gate), dev(up)), None))
    for name, w_gate, w_up in forms:
        for grouped in ([True, False] if dtype == "bfloat16" and name == "interleaved" else [True]):
            ops.USE_GROUPED_TCGEN05 = grouped
            try:
                got = ops.routed_experts(dev(x), ids, weights, w_gate, w_up, dev(down), weigh_inputs=True).cpu().double()
            finally:
                ops.USE_GROUPED_TCGEN05 = True
            assert (got - expected).abs().max() < bound, (name, grouped)
    assert (outputs - expected).abs().max() > 5 * bound            # a weight on the outputs would not pass
