"""The kernels of Tedulorn's mechanisms alone, each against a plain float64 restatement (tests/plain_tedulorn.py), with
inputs made so that a fault shows: retention in pieces of 64 tokens and token by token, over every cutting of a
request, beside other requests, from a state that is not zero, with keys that stand out hundreds of tokens back;
attention with one added to the denominator where queries point at ONE key each (just inside a window and just outside
it, the last kept token and the first one that is not kept) and where no key scores at all; values mixed with another
layer's on their way into the cache; the router's groups and normalised weights; bounded experts; the squared ReLU;
the gate on a token's row."""

import math

import pytest
import torch

from plain_tedulorn import (F64, bounded_expert, decayed_states, gelu_tanh, mix_values, raw_scores, rms_norm, rotate_halves, route,
                            softmax_plus_one, weigh_values, window_mask)

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _i32(values, device):
    return torch.tensor(list(values), dtype=torch.int32, device=device)


# ------------------------------------------------------------------------------------------- retention
def _run_retention(device, q, k, v, decay, portions, form, state=None):
    """The requests' portions, step by step: ``portions`` lists, per step, how many tokens each request brings."""
    from zephyr_b200.kernels import ops

    R, (_, H, d), dv = len(q), q[0].shape, v[0].shape[2]
    state = torch.zeros(R + 1, H * d * dv, device=device) if state is None else state
    status, at, outs = ops.new_status(device), [0] * R, [[] for _ in range(R)]
    for counts in portions:
        rows = [r for r in range(R) if counts[r] > 0]
        join = lambda parts: torch.cat([parts[r][at[r]:at[r] + counts[r]].reshape(counts[r], -1) for r in rows]).float()
        # (values as a slice of wider rows, as a fused projection leaves them)
        turned = torch.cat([join(q), join(k)], dim=1).contiguous().to(device)
        values = torch.cat([torch.zeros(turned.shape[0], 8), join(v)], dim=1).to(device)[:, 8:]
        starts = [sum(counts[r] for r in rows[:i]) for i in range(len(rows))]
        where = (state, _i32([R - r for r in rows], device), _i32(starts, device), _i32([counts[r] for r in rows], device), status)
        args = (turned[:, :H * d], turned[:, H * d:], values)
        if form == "pieces":
            o = ops.retention(*args, decay.float().to(device), H, d, dv, *where)
        else:
            o = ops.decayed_state_scan("fixed", *args, H, d, dv, *where, decay=decay.float().to(device), segment=form)
        for i, r in enumerate(rows):
            outs[r].append(o[starts[i]:starts[i] + counts[r]].cpu())
            at[r] += counts[r]
    ops.check_status(status)
    return [torch.cat(o).double() for o in outs], state


@pytest.mark.parametrize("H,d,dv", [(3, 20, 12), (1, 64, 64), (2, 33, 50), (2, 128, 136), (1, 250, 24), (4, 16, 200), (1, 7, 1), (2, 256, 128)])
def test_retention_in_every_cutting(cuda_device, H, d, dv):
    """Three requests of unequal length in one step, then in portions that end inside, at and across a piece's edge,
    down to one and two tokens; both forms of the recurrence; strided slots in another order than the rows."""
    g = torch.Generator().manual_seed(H * d + dv)
    lengths = (333, 130, 64)
    q, k, v = ([torch.randn(n, H, w, generator=g) * s for n in lengths] for w, s in ((d, 1.0), (d, d ** -0.5), (dv, 1.0)))
    # One key stands out in the first piece and the queries of the last tokens point at it: what the carry loses shows.
    for r, n in enumerate(lengths):
        k[r][3] *= 6.0
        q[r][n - 20:] += k[r][3] * 3.0
    decay = torch.tensor([0.999, 0.97, 0.4, 1.0][:H] if H > 1 else [0.995], dtype=F64)
    expected = [decayed_states(q[r].double(), k[r].double(), v[r].double(), decay).reshape(lengths[r], -1) for r in range(3)]
    cuttings = {"whole": [lengths], "portions": [(64, 1, 2), (1, 63, 62), (2, 66, 0), (190, 0, 0), (76, 0, 0)],
                "pieces' edges": [(63, 65, 64), (65, 64, 0), (128, 1, 0), (77, 0, 0)]}
    for name, portions in cuttings.items():
        for form, bound in (("pieces", 2e-4), (0, 2e-5), (128, 3e-5)):
            got, _ = _run_retention(cuda_device, q, k, v, decay, portions, form)
            for r in range(3):
                error = (got[r] - expected[r]).abs().max() / expected[r].abs().max()
                assert error < bound, (name, form, r, float(error))


def test_retention_goes_on_from_a_state_and_leaves_one(cuda_device):
    """Pieces leave the state that the token-by-token form leaves, whichever form made the one before; a request's slot
    is its own; without ``write_state`` slots stay as they are."""
    from zephyr_b200.kernels import ops

    H, d, dv, n = 2, 32, 48, 150
    g = torch.Generator().manual_seed(1)
    q, k, v = ([torch.randn(n, H, w, generator=g) for _ in range(2)] for w in (d, d, dv))
    decay = torch.tensor([0.99, 0.9], dtype=F64)
    states = {}
    for forms in (("pieces", "pieces"), ("pieces", 0), (0, "pieces"), (0, 0)):
        state = torch.zeros(3, H * d * dv, device=cuda_device)
        for form, portions in zip(forms, ([(70, 30)], [(80, 120)])):
            part = lambda parts: [parts[r][:70 if r == 0 else 30] if portions[0][0] == 70 else parts[r][70 if r == 0 else 30:] for r in range(2)]
            _, state = _run_retention(cuda_device, part(q), part(k), part(v), decay, portions, form, state)
        states[forms] = state.cpu()
        assert torch.equal(state[0].cpu(), torch.zeros(H * d * dv))
    reference = states[(0, 0)]
    for forms, state in states.items():
        assert (state - reference).abs().max() < 1e-4 * reference.abs().max(), forms
    flat = lambda t: t[0].reshape(n, -1).float().to(cuda_device)
    state = torch.full((1, H * d * dv), 0.5, device=cuda_device)
    status = ops.new_status(cuda_device)
    ops.retention(flat(q), flat(k), flat(v), decay.float().to(cuda_device), H, d, dv, state, _i32([0], cuda_device), _i32([0], cuda_device),
                  _i32([n], cuda_device), status, write_state=False)
    assert (state == 0.5).all()
    # a slot that does not exist is reported and not touched
    ops.retention(flat(q), flat(k), flat(v), decay.float().to(cuda_device), H, d, dv, state, _i32([4], cuda_device), _i32([0], cuda_device),
                  _i32([n], cuda_device), status)
    with pytest.raises(ops.KernelError):
        ops.check_status(status)
    assert (state == 0.5).all()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,dv,dims", [(3, 20, 12, 8), (1, 64, 64, 64), (2, 33, 50, 32), (2, 128, 136, 2), (1, 250, 24, 16), (4, 16, 2000, 16),
                                         (1, 7, 1, 0), (16, 128, 128, 128), (2, 8, 257, 4)])
def test_one_token_a_request_from_the_projection_to_the_gate(cuda_device, dtype, H, d, dv, dims):
    """Five requests of different histories, twelve tokens each, every step one token a request: rotation at the
    request's own position, state, unit norm, gate."""
    from zephyr_b200.kernels import ops

    R, steps, eps, rot = 5, 12, 1e-5, {"base": 50.0, "dims": dims}
    g = torch.Generator().manual_seed(H * d + dv)
    width = 2 * H * (d + dv)
    rows = torch.randn(R, steps, width + 3, generator=g)                # (rows of a wider tensor)
    rows[:, :, H * d:2 * H * d] = 0.6 * rows[:, :, H * d:2 * H * d] + 0.8 * rows[:, :, :H * d]
    first = [0, 3, 40, 900, 17]
    decay = torch.tensor([[0.999, 0.97, 0.4, 1.0][h % 4] for h in range(H)], dtype=F64)
    freqs = torch.tensor([50.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64).float().to(cuda_device) if dims else None
    state = torch.randn(R + 2, H * d * dv, generator=g) * 0.2
    before = state.clone()
    state = state.to(cuda_device)
    slots, status = [6, 0, 3, 5, 1], ops.new_status(cuda_device)
    outs = []
    for i in range(steps):
        outs.append(ops.retention_step(rows[:, i].contiguous().to(cuda_device)[:, :width], decay.float().to(cuda_device), freqs, dims, d ** -0.5, eps,
                                       H, d, dv, state, _i32(slots, cuda_device), _i32(range(R), cuda_device), _i32([1] * R, cuda_device),
                                       _i32([f + i for f in first], cuda_device), status, DTYPES[dtype]).cpu().double())
    ops.check_status(status)
    for r in range(R):
        x = rows[r].double()
        q, k = (x[:, at:at + H * d].view(steps, H, d) for at in (0, H * d))
        v, gate = (x[:, at:at + H * dv].view(steps, H, dv) for at in (2 * H * d, 2 * H * d + H * dv))
        if dims:
            positions = torch.arange(first[r], first[r] + steps)
            q, k = rotate_halves(q, positions, rot), rotate_halves(k, positions, rot)
        S = before[slots[r]].double().view(H, d, dv)
        for i in range(steps):
            S = decay.view(H, 1, 1) * S + (k[i] * d ** -0.5).unsqueeze(-1) * v[i].unsqueeze(1)
            o = torch.einsum("hdv,hd->hv", S, q[i])
            o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * gate[i] * torch.sigmoid(gate[i])
            bound = (1e-3 if dtype == "float32" else 0.012) * max(1.0, float(o.abs().max()))
            assert (outs[i][r] - o.reshape(-1)).abs().max() < bound, (r, i)
        assert (state[slots[r]].cpu().double() - S.reshape(-1)).abs().max() < 1e-3 * max(1.0, float(S.abs().max()))
    for slot in (2, 4):
        assert torch.equal(state[slot].cpu(), before[slot])
    # a row that brings two tokens is refused where it is seen
    ops.retention_step(rows[:1, 0].contiguous().to(cuda_device)[:, :width], decay.float().to(cuda_device), freqs, dims, 1.0, eps, H, d, dv, state,
                       _i32([2], cuda_device), _i32([0], cuda_device), _i32([2], cuda_device), _i32([0], cuda_device), status, DTYPES[dtype])
    with pytest.raises(ops.KernelError):
        ops.check_status(status)
    assert torch.equal(state[2].cpu(), before[2])


@pytest.mark.parametrize("heads,dim,dims", [(3, 20, 8), (2, 64, 64), (1, 33, 32), (5, 16, 2), (4, 10, 0)])
def test_queries_and_keys_turn_before_the_keys_are_scaled(cuda_device, heads, dim, dims):
    from zephyr_b200.kernels import ops

    T, rot = 60, {"base": 300.0, "dims": dims}
    g = torch.Generator().manual_seed(dim)
    x = torch.randn(T, 2 * heads * dim + 5, generator=g)
    positions = torch.randint(0, 3000, (T,), generator=g)
    freqs = torch.tensor([300.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64).float() if dims else None
    got = ops.rotate_qk(x.to(cuda_device), heads, dim, freqs.to(cuda_device) if dims else None, dims, 0.25, positions.int().to(cuda_device)).cpu().double()
    q, k = (x[:, at:at + heads * dim].double().view(T, heads, dim) for at in (0, heads * dim))
    if dims:
        q, k = rotate_halves(q, positions, rot), rotate_halves(k, positions, rot)
    expected = torch.cat([q.reshape(T, -1), 0.25 * k.reshape(T, -1)], dim=1)
    assert (got - expected).abs().max() < 2e-3          # (an angle of a few thousand is a float32 product)
    near = positions < 60
    assert (got - expected)[near].abs().max() < 2e-5 if near.any() else True


# ------------------------------------------------------------------------------------------- attention
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

    def write(self, at, n, **mixing):
        from zephyr_b200.kernels import ops

        pos = torch.arange(at, at + n, dtype=torch.int32, device=self.device)
        return ops.qkv_halves(self.projected[at:at + n], self.H, self.G, self.d, self.dv, "none", None, None, 1e-6, None, 0, 1.0, False,
                              pos, torch.zeros(n, dtype=torch.int32, device=self.device), self.cache, self.table, self.status,
                              self.dtype, **mixing)

    def rows(self, at, n):
        return _i32([0], self.device), _i32([n], self.device), _i32([at], self.device)

    def tiles(self, n, tokens):
        q0 = torch.arange(0, n, tokens, dtype=torch.int32, device=self.device)
        return torch.zeros_like(q0), q0


def _run(stored, portions, kernel, *, window, scale, keep_first, sinks):
    from zephyr_b200.kernels import ops

    s, outs, at = stored, [], 0
    for n in portions:
        q = s.write(at, n)
        rows = s.rows(at, n)
        masks = dict(keep_first=keep_first) if keep_first else {}
        out = torch.full((n, s.H * s.dv), float("nan"), dtype=s.dtype, device=s.device)
        if kernel == "general":
            tile = ops.attention_tile_tokens(s.H // s.G)
            out = ops.paged_attention(q, s.cache, s.table, *s.tiles(n, tile), tile, *rows, s.H, s.G, s.d, window, scale, s.status,
                                      value_dim=s.dv, sinks=sinks, **masks)
        elif kernel == "heads":
            tile = 1 if n == 1 else ops.heads_attention_tile_tokens(s.H, s.G, s.d, s.dv, s.dtype)
            splits = [None, 1, 3, 40][at % 4] if n == 1 else None      # (one CTA, several, more than there are tiles)
            ops.heads_attention(q, s.cache, s.table, *s.tiles(n, tile), *rows, s.H, s.G, s.d, s.dv, window, scale, s.status, out,
                                single=n == 1, max_context=at + n, splits=splits, sinks=sinks, **masks)
        elif kernel == "prompt" or n > 1:
            tile = ops.paged_prefill_tile_tokens()
            ops.paged_prefill(q, s.cache, s.table, *s.tiles(n, tile), *rows, s.H, s.G, s.d, window, scale, s.status, out,
                              by_group=kernel == "prompt" and n == 1 and s.H // s.G <= 16, sinks=sinks, **masks)
        else:
            ops.paged_decode(q, s.cache, s.table, _i32([0], s.device), rows[0], rows[2], at + 1, s.H, s.G, s.d, window, scale,
                             s.status, out, split_size=[None, 0, 32, 128][at % 4], sinks=sinks)
        outs.append(out)
        at += n
    ops.check_status(s.status)
    return torch.cat(outs).cpu().double()


def _expected(dtype, q, k, v, visible, scale, one=True):
    q, k, v = (t.to(DTYPES[dtype]).double() for t in (q, k, v))
    scores = raw_scores(q, k, scale)
    weights = softmax_plus_one(scores, visible) if one else torch.softmax(scores.masked_fill(~visible, -math.inf), -1)
    return weigh_values(weights, v).reshape(q.shape[0], -1)


PORTIONS = ([293] + [1] * 40, [7, 2, 150, 1, 1, 90, 2] + [1] * 20 + [60])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,size,keep,page", [
    (4, 2, 24, 40, 90, 22, 16), (3, 1, 20, 12, 23, 7, 16), (8, 4, 32, 32, 9, 0, 16), (5, 5, 16, 24, 70, 33, 32),
    (12, 4, 128, 96, 33, 40, 16), (16, 8, 128, 128, 64, 16, 16), (3, 1, 64, 64, 5, 1, 64), (32, 2, 16, 16, 300, 4, 16),
    (6, 2, 32, 64, 70, 65, 16), (8, 2, 160, 136, 64, 64, 32), (34, 2, 32, 24, 21, 3, 16), (1, 1, 9, 7, 17, 2, 16),
    (6, 3, 48, 64, 1, 0, 16), (4, 4, 128, 128, 90, 0, 16)])
def test_one_in_the_denominator_over_a_kept_window(cuda_device, dtype, H, G, d, dv, size, keep, page):
    """On every kernel that takes the layer.  Head 0 points at single keys (the last kept token, the first that is not
    kept, the window's edges, the first token), the last head at nothing: its scores lie far below zero, so that the one
    in the denominator takes nearly all the weight, and the middle ones around zero."""
    from zephyr_b200.kernels import ops

    T, scale = 333, 0.8
    targets = {p: min(max([keep - 1, keep, p - size + 1, p - size, 0, p - 1][p % 6], 0), p) for p in range(T - 60, T)}
    q, k, v = _case(H * 100 + size + keep, T, H, G, d, dv, targets)
    if H > 1:
        q[:, -1] *= 0.2
        if G > 1 or H == G:
            k[:, -1] += 1.0
            q[:, -1] -= 0.5
    visible = window_mask(T, size, keep)
    expected = _expected(dtype, q, k, v, visible, scale)
    bound = (4e-5 if dtype == "float32" else 0.03) * max(1.0, float(expected.abs().max()))
    sinks = torch.zeros(H, device=cuda_device)
    kernels = ["general"]
    if dtype == "bfloat16":
        if ops.heads_attention_tile_tokens(H, G, d, dv, torch.bfloat16):
            kernels.append("heads")
        if d == dv and ops.paged_prefill_supported(H, G, d, torch.bfloat16):
            kernels.append("prompt")
        if d == dv and not keep and ops.paged_decode_supported(H, G, d, torch.bfloat16):
            kernels.append("decode")
        assert len(kernels) > 1 or H > 32
    for kernel in kernels:
        for portions in PORTIONS:
            got = _run(Stored(cuda_device, dtype, q, k, v, page), portions, kernel, window=size, scale=scale, keep_first=keep, sinks=sinks)
            assert torch.isfinite(got).all(), kernel
            assert (got - expected).abs().max() < bound, (kernel, portions[:3], (got - expected).abs().max())
    # Each of these mistakes would not pass.
    mistakes = {"one key less kept": _expected(dtype, q, k, v, window_mask(T, size, keep - 1), scale) if keep and size + keep < T - 60 else None,
                "one key more kept": _expected(dtype, q, k, v, window_mask(T, size, keep + 1), scale) if size + keep < T - 60 else None,
                "a window one shorter": _expected(dtype, q, k, v, window_mask(T, size - 1, keep), scale) if size > 1 and size + keep < T else None,
                "a window one longer": _expected(dtype, q, k, v, window_mask(T, size + 1, keep), scale) if size + keep < T - 60 else None,
                "no one in the denominator": _expected(dtype, q, k, v, visible, scale, one=False)}
    for name, wrong in mistakes.items():
        if wrong is not None:
            assert (wrong - expected).abs().max() > 5 * bound, name


@pytest.mark.parametrize("kernel", ["general", "heads", "prompt", "decode"])
def test_sinks_of_different_heights_on_every_kernel(cuda_device, kernel):
    """A sink of its own per head, from far below the scores to far above them: the general form of the same term."""
    H, G, d, T, scale = 8, 4, 64, 333, 0.5
    q, k, v = _case(3, T, H, G, d, d, {})
    sinks = torch.tensor([-40.0, -3.0, -1.0, 0.0, 0.5, 2.0, 5.0, 40.0])
    rounded = [t.to(torch.bfloat16).double() for t in (q, k, v)]
    scores = raw_scores(rounded[0], rounded[1], scale).masked_fill(~window_mask(T, 50), -math.inf)
    weights = torch.softmax(torch.cat([scores, sinks.double().view(H, 1, 1).expand(H, T, 1)], dim=-1), -1)[..., :-1]
    expected = weigh_values(weights, rounded[2]).reshape(T, -1)
    got = _run(Stored(cuda_device, "bfloat16", q, k, v, 16), PORTIONS[1], kernel, window=50, scale=scale, keep_first=0, sinks=sinks.to(cuda_device))
    assert (got - expected).abs().max() < 0.03 * float(expected.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 24, 40), (3, 3, 32, 32), (6, 1, 16, 7)])
def test_values_are_mixed_on_their_way_into_the_cache(cuda_device, dtype, H, G, d, dv):
    """Both sides unrounded, one rounding of the mixture; queries and keys are not touched.  Read back through attention
    over one key: with a window of one token the output is that token's values."""
    from zephyr_b200.kernels import ops

    T = 90
    q, k, v = _case(H + dv, T, H, G, d, dv, {})
    g = torch.Generator().manual_seed(9)
    first = torch.randn(T, 3 + G * dv, generator=g)                # (a slice of wider rows)
    share = torch.tensor([0.37])
    stored, plain = (Stored(cuda_device, dtype, q, k, v, 16) for _ in range(2))
    wide = first.to(cuda_device)
    queries = torch.cat([stored.write(at, n, v_first=wide[at:at + n, 3:], v_share=share.to(cuda_device)) for at, n in ((0, 60), (60, 1), (61, 29))])
    assert torch.equal(queries, plain.write(0, T))
    tile = ops.attention_tile_tokens(H // G)
    read = lambda s: ops.paged_attention(queries, s.cache, s.table, *s.tiles(T, tile), tile, *s.rows(0, T), H, G, d, 1, 1.0, s.status,
                                         value_dim=dv).cpu().double().view(T, H, dv)
    mixed = mix_values(v.double(), first[:, 3:].double().view(T, G, dv), share.double()).repeat_interleave(H // G, dim=1)
    bound = (1e-6 if dtype == "float32" else 2.0 ** -8) * float(mixed.abs().max())
    assert (read(stored) - mixed).abs().max() < bound
    assert (read(plain) - v.double().repeat_interleave(H // G, dim=1)).abs().max() < (1e-6 if dtype == "float32" else 2.0 ** -8) * 5
    ops.check_status(stored.status)


# ---------------------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("experts,top,count,keep", [(6, 2, 3, 2), (16, 4, 8, 5), (8, 8, 1, 1), (12, 4, 4, 2), (7, 3, 1, 1), (64, 6, 8, 3), (9, 1, 3, 1)])
def test_the_router_against_the_plain_one(cuda_device, experts, top, count, keep):
    """Corrections that make choice scores negative, so that a group left out must count as minus infinity."""
    from zephyr_b200.kernels import ops

    g = torch.Generator().manual_seed(experts * top)
    z = torch.randn(500, experts, generator=g) * 2.0
    correction = torch.randn(experts, generator=g) * 0.3 - 0.4
    ids, weights, margin = route(z.double(), correction.double(), {"top": top, "groups": {"count": count, "keep": keep}})
    got_ids, got_weights = ops.route(z.to(cuda_device), correction.to(cuda_device), top, "softmax", (count, keep, 1) if count > 1 else None,
                                     normalize=True)
    clear = margin > 1e-5
    assert clear.float().mean() > 0.95
    # the set that is taken, and each one's weight (an order among equals does not matter)
    scatter = lambda i, w: torch.zeros(500, experts, dtype=F64).scatter_(1, i.long(), w.double())
    got, expected = scatter(got_ids.cpu(), got_weights.cpu()), scatter(ids, weights)
    assert (got - expected)[clear].abs().max() < 1e-5
    assert (got.sum(1) - 1.0).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens,experts,top,count,keep,width,ff,shared_ff", [
    (1, 4, 2, 2, 1, 64, 48, 16), (33, 6, 1, 3, 2, 40, 24, 30), (200, 3, 3, 1, 1, 64, 64, 72), (700, 8, 2, 4, 3, 128, 136, 64), (50, 6, 4, 3, 2, 60, 27, 13)])
def test_bounded_experts_with_a_shared_one(cuda_device, dtype, tokens, experts, top, count, keep, width, ff, shared_ff):
    """On every path of the products (the grouped tcgen05 launch, tiles on mma.sync, CUDA cores, both layouts of the
    matrices), with products far beyond the bounds and bounds of their own for the shared expert."""
    from zephyr_b200.config.spec import FeedForwardSpec
    from zephyr_b200.kernels import ops
    from zephyr_b200.parts import RoutedFeedForward

    g = torch.Generator().manual_seed(tokens + experts)
    cast = lambda t: t.to(DTYPES[dtype])
    x = cast(torch.randn(tokens, width, generator=g) * 2.0)
    names = tuple((f"e{e}.gate", f"e{e}.up", f"e{e}.down") for e in range(experts))
    w = {"router": cast(torch.randn(experts, width, generator=g) * 2.0 * width ** -0.5), "correction": torch.randn(experts, generator=g) * 0.3}
    for prefix, size in [(f"e{e}", ff) for e in range(experts)] + [("shared", shared_ff)]:
        w.update({f"{prefix}.gate": cast(torch.randn(size, width, generator=g) * 1.5 * width ** -0.5),
                  f"{prefix}.up": cast(torch.randn(size, width, generator=g) * 1.5 * width ** -0.5),
                  f"{prefix}.down": cast(torch.randn(width, size, generator=g) * size ** -0.5)})
    shape = {"hidden_size": width, "activation": "clamped_swish", "alpha": 1.702, "up_shift": 1.0}
    spec = FeedForwardSpec("routed", {**shape, "intermediate_size": ff, "limit": 0.9, "experts": experts, "top": top, "normalize": True,
                                      "groups": {"count": count, "keep": keep, "top": 1}, "router": "router", "correction": "correction",
                                      "expert_names": names,
                                      "shared": {**shape, "intermediate_size": shared_ff, "limit": 2.5, "gate_proj": "shared.gate",
                                                 "up_proj": "shared.up", "down_proj": "shared.down"}})
    assert set(RoutedFeedForward.weight_decls(spec)) == set(w)
    part = RoutedFeedForward(spec, {name: t.to(cuda_device) for name, t in w.items()}, DTYPES[dtype])
    ids, weights = (t.cpu() for t in part.route(x.to(cuda_device)))
    d = {name: t.double() for name, t in w.items()}
    expected = bounded_expert(x.double(), d, "shared", 2.5)
    unbounded = expected.clone()
    for j in range(top):
        for e in range(experts):
            t = (ids[:, j] == e).nonzero().flatten()
            expected.index_add_(0, t, weights[t, j].double().unsqueeze(1) * bounded_expert(x[t].double(), d, f"e{e}", 0.9))
            unbounded.index_add_(0, t, weights[t, j].double().unsqueeze(1) * bounded_expert(x[t].double(), d, f"e{e}", 1e9))
    bound = (3e-5 if dtype == "float32" else 2.0 ** -6) * float(expected.abs().max())
    for grouped in ([True, False] if dtype == "bfloat16" else [True]):
        ops.USE_GROUPED_TCGEN05 = grouped
        try:
            summands = part.forward_summands(x.to(cuda_device))
            assert len(summands) == 2
            got = sum(s.cpu().double() for s in summands)
            joined = part.forward(x.to(cuda_device)).cpu().double()
        finally:
            ops.USE_GROUPED_TCGEN05 = True
        assert (got - expected).abs().max() < bound, grouped
        assert (joined - expected).abs().max() < bound + 2.0 ** -8 * float(expected.abs().max()), grouped
    assert (unbounded - expected).abs().max() > 5 * bound


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,width,ff", [(1, 64, 96), (7, 60, 100), (16, 256, 512), (40, 128, 72), (300, 96, 200), (513, 128, 264), (1100, 256, 1000)])
def test_the_squared_relu_feed_forward(cuda_device, dtype, rows, width, ff):
    """Few rows, many rows and rows between: the activation in the product's epilogue and behind it."""
    from zephyr_b200.config.spec import FeedForwardSpec
    from zephyr_b200.parts import UngatedFeedForward

    g = torch.Generator().manual_seed(rows + ff)
    x = (torch.randn(rows, width, generator=g) * 1.5).to(DTYPES[dtype])
    up, down = (torch.randn(ff, width, generator=g) * width ** -0.5).to(DTYPES[dtype]), (torch.randn(width, ff, generator=g) * ff ** -0.5).to(DTYPES[dtype])
    part = UngatedFeedForward(FeedForwardSpec("ungated", {"hidden_size": width, "intermediate_size": ff, "activation": "relu_squared",
                                                          "up_proj": "u", "down_proj": "d"}),
                              {"u": up.to(cuda_device), "d": down.to(cuda_device)}, DTYPES[dtype])
    got = part.forward(x.to(cuda_device)).cpu().double()
    expected = torch.relu(x.double() @ up.double().T) ** 2 @ down.double().T
    assert (got - expected).abs().max() < (2e-5 if dtype == "float32" else 2.0 ** -6) * float(expected.abs().max())


def test_the_squared_relu_in_every_form(cuda_device):
    from zephyr_b200.kernels import ops

    z = torch.cat([torch.linspace(-12.0, 12.0, 1001), torch.tensor([-1e4, 1e4, 0.0])])
    assert torch.equal(ops.act_rows(z.to(cuda_device), "relu_squared").cpu(), torch.relu(z) ** 2)
    g = torch.Generator().manual_seed(1)
    w = (torch.randn(304, 64, generator=g) * 0.4).to(torch.bfloat16)
    x = torch.randn(600, 64, generator=g).to(torch.bfloat16)
    expected = torch.relu(x.double() @ w.double().T) ** 2
    for block_n in (0, 2, 128, 256):
        y = ops.gemm_tc(x.to(cuda_device), w.to(cuda_device), product_act="relu_squared", block_n=block_n).cpu().double()
        assert ((y - expected).abs() <= 2.0 ** -8 * expected.abs() + 2e-5).all()
    y = ops.gemm_small(x[:9].to(cuda_device), w.to(cuda_device), product_act="relu_squared").cpu().double()
    assert ((y - expected[:9]).abs() <= 2.0 ** -8 * expected[:9].abs() + 2e-5).all()


# ------------------------------------------------------------------------------- the gate on a token's row
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,width,dim,layers", [(1, 64, 12, 3), (9, 60, 7, 5), (16, 64, 7, 5), (30, 128, 64, 2), (600, 96, 24, 4)])
def test_the_token_gate_behind_a_layer(cuda_device, dtype, rows, width, dim, layers):
    """The part alone, for every layer's share of the table: the summand, and the stream with the next norm of it."""
    from types import SimpleNamespace

    from zephyr_b200.config.spec import NormSpec, SideSpec
    from zephyr_b200.kernels import ops
    from zephyr_b200.parts import RMSNorm, TokenGate

    vocab, eps = 50, 1e-5
    g = torch.Generator().manual_seed(rows + dim)
    cast = lambda t: t.to(DTYPES[dtype])
    w = {"table": cast(torch.randn(vocab, dim * layers, generator=g)), "gate": cast(torch.randn(dim, width, generator=g) * 1.5 * width ** -0.5),
         "proj": cast(torch.randn(width, dim, generator=g) * dim ** -0.5), "norm": cast(torch.randn(width, generator=g) * 0.2 + 1.0),
         "next": cast(torch.randn(width, generator=g) * 0.2 + 1.0)}
    on = {name: t.to(cuda_device) for name, t in w.items()}
    d = {name: t.double() for name, t in w.items()}
    ids = torch.randint(0, vocab, (rows,), generator=g)
    stream, a, b = torch.randn(rows, width, generator=g) * 3.0, cast(torch.randn(rows, width, generator=g)), cast(torch.randn(rows, width, generator=g))
    then = RMSNorm(NormSpec("rmsnorm", width, eps, "next"), on, DTYPES[dtype])
    ctx = SimpleNamespace(token_ids=ids.int().to(cuda_device), status=ops.new_status(cuda_device))
    for index in range(layers):
        part = TokenGate(SideSpec("token_gate", {"hidden_size": width, "vocab_size": vocab, "dim": dim, "offset": index * dim, "row": layers * dim,
                                                 "table": "table", "gate": "gate", "proj": "proj", "norm": NormSpec("rmsnorm", width, eps, "norm")}),
                         on, DTYPES[dtype])
        hidden = stream.clone().to(cuda_device)
        x = then.sum_rounded(hidden, (a.to(cuda_device), b.to(cuda_device)))
        total = stream.double() + a.double() + b.double()
        assert (hidden.cpu().double() - total).abs().max() < 1e-5 and x.dtype == DTYPES[dtype]
        assert (x.cpu().double() - total).abs().max() <= (1e-5 if dtype == "float32" else 2.0 ** -8 * float(total.abs().max()))
        own = x.clone()                    # (in float32 the sum is the stream itself, which goes on)
        normed = part.forward(x, ctx).apply(hidden, then=then)
        y = (gelu_tanh(own.cpu().double() @ d["gate"].T) * d["table"][ids, index * dim:(index + 1) * dim]) @ d["proj"].T
        expected = total + rms_norm(y, d["norm"], eps)
        bound = 3e-5 if dtype == "float32" else 0.02
        assert (hidden.cpu().double() - expected).abs().max() < bound * float(expected.abs().max()), index
        expected_norm = rms_norm(expected, d["next"], eps)
        assert (normed.cpu().double() - expected_norm).abs().max() < 2 * bound * float(expected_norm.abs().max()), index
    ops.check_status(ctx.status)


def test_a_token_outside_the_table_is_reported(cuda_device):
    from zephyr_b200.kernels import ops

    status = ops.new_status(cuda_device)
    z, table = torch.ones(2, 4, device=cuda_device), torch.ones(5, 8, device=cuda_device)
    out = ops.token_gate(z, table, 4, _i32([3, 5], cuda_device), status)
    assert (out[1] == 0).all() and (out[0] > 0.8).all()
    with pytest.raises(ops.KernelError):
        ops.check_status(status)
