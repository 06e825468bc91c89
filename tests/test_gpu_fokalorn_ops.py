"""The kernels behind the Fokalorn parts, each against a few lines of plain float64 arithmetic."""
import numpy as np
import pytest
import torch

import plain_fokalorn as plain
from test_gpu_dobelix_ops import DEV, make_step

pytestmark = pytest.mark.gpu


def dev(a, dtype=torch.float32):
    return torch.tensor(np.ascontiguousarray(a), dtype=dtype, device=DEV)


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def close(got, want, tol):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    return np.max(np.abs(got - want)) <= tol * max(np.max(np.abs(want)), 1e-30)


@pytest.mark.parametrize("width,groups", [(64, 1), (64, 4), (96, 3), (50, 5), (256, 16), (1500, 12), (4096, 2), (48, 48)])
def test_group_norm(width, groups):
    """Groups of whole 16-byte pieces and odd ones, fewer and more groups than warps; chosen rows."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(width + groups)
    x, w = rng.normal(size=(9, width)) * rng.uniform(0.1, 5.0, size=width), rng.normal(size=width) + 1.0
    want = plain.group_norm(x, w, 1e-3, groups)
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 8e-3)):
        out = torch.empty((9, width), dtype=dtype, device=DEV)
        ops.group_rmsnorm(dev(x), dev(w), out, 1e-3, groups)
        assert close(host(out), want, tol)
    rows = [7, 0, 3, 3]
    out = torch.empty((4, width), device=DEV)
    ops.group_rmsnorm(dev(x), dev(w), out, 1e-3, groups, rows=dev(rows, torch.int32))
    assert close(host(out), want[rows], 3e-6)


@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8])
@pytest.mark.parametrize("width,groups", [(64, 2), (30, 3)])
def test_stream_step(streams, width, groups):
    """Update, weighted sum and norm in one pass: from equal streams, from streams that differ, and the final sum of
    chosen rows; the streams that were read stay as they were."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(streams)
    n = 7
    X, y = rng.normal(size=(streams, n, width)), rng.normal(size=(n, width))
    a, b, M, w = rng.normal(size=streams), rng.normal(size=streams), rng.normal(size=(streams, streams)), rng.normal(size=width)
    tok = dev(X.transpose(1, 0, 2).copy())
    norm = lambda u: plain.group_norm(u, w, 1e-4, groups)
    out = torch.empty((n, width), device=DEV)
    ops.stream_step(tok, dev(w), 1e-4, groups, out, dev(a))                       # nothing to update yet
    assert close(host(out), norm(plain.collect_streams(X, a)), 1e-5)
    new = torch.empty_like(tok)
    ops.stream_step(tok, dev(w), 1e-4, groups, out, dev(a), (dev(y), dev(M), dev(b)), new)
    want = plain.spread_streams(X, M, b, y)
    assert close(host(new).transpose(1, 0, 2), want, 1e-5) and close(host(out), norm(plain.collect_streams(want, a)), 2e-5)
    assert close(host(tok).transpose(1, 0, 2), X, 1e-6)
    same = np.repeat(X[:1], streams, axis=0)                                      # equal streams: one row per token
    ops.stream_step(dev(X[0]), dev(w), 1e-4, groups, out, dev(a), (dev(y), dev(M), dev(b)), new)
    want = plain.spread_streams(same, M, b, y)
    assert close(host(new).transpose(1, 0, 2), want, 1e-5)
    rows = [6, 2]
    last = torch.empty((2, width), device=DEV)
    ops.stream_step(tok, dev(w), 1e-4, groups, last, None, (dev(y), dev(M), dev(b)), None, rows=dev(rows, torch.int32))
    assert close(host(last), norm(plain.spread_streams(X, M, b, y).sum(axis=0))[rows], 2e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [40, 18])
def test_token_shift_across_portions_and_slots(dtype, width):
    """Steps of unequal portions of several requests: the row in front of a portion comes from the request's own state,
    which single tokens, short portions and portions longer than a block's run renew; other slots stay as they are."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(width)
    lengths = {5: 2600, 0: 47, 2: 9}
    a, w, mu = rng.normal(size=2), rng.normal(size=width) + 1, rng.uniform(size=width)
    X = {s: rng.normal(size=(2, n, width)) for s, n in lengths.items()}
    want = {s: plain.token_shift(plain.group_norm(plain.collect_streams(x, a), w, 1e-5, 2), mu) for s, x in X.items()}
    state = torch.full((8, width), 9.0, device=DEV)                               # stale content of earlier requests
    for s in lengths:
        state[s].zero_()                                                          # what admission does
    at = {s: 0 for s in lengths}
    got = {s: [] for s in lengths}
    for sizes in ({5: 1, 0: 20}, {5: 2, 2: 1}, {0: 1, 5: 2500, 2: 3}, {2: 5, 5: 90, 0: 26}, {5: 7}):
        slots = list(sizes)
        step = make_step(list(sizes.values()), lengths=[at[s] for s in slots], slots=slots)
        x = dev(np.concatenate([X[s][:, at[s]:at[s] + n].transpose(1, 0, 2) for s, n in sizes.items()]))
        out = torch.empty((step.n, width), dtype=dtype, device=DEV)
        ops.stream_step(x, dev(w), 1e-5, 2, out, dev(a), shift=(dev(mu), state, True), step=step)
        again = torch.empty_like(out)
        keep = state.clone()
        o, i = host(out), 0
        for s, n in sizes.items():
            got[s].append(o[i:i + n]); i += n; at[s] += n
        ops.stream_step(x, dev(w), 1e-5, 2, again, dev(a), shift=(dev(mu), state, False), step=step)       # a reader only
        assert torch.equal(keep, state)
    for s in lengths:
        assert close(np.concatenate(got[s]), want[s], 1e-5 if dtype == torch.float32 else 8e-3), s
    assert torch.all(state[[1, 3, 4, 6, 7]] == 9.0)


SHAPES = [(2, 2, 16, 24), (4, 2, 64, 64), (3, 1, 5, 7), (2, 1, 72, 40), (1, 1, 128, 128), (2, 2, 96, 33), (1, 1, 200, 16), (2, 2, 33, 50), (1, 1, 256, 20)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,qk,dim,vdim", SHAPES)
@pytest.mark.parametrize("rate", [-3.0, 3.0])
def test_channel_delta(dtype, heads, qk, dim, vdim, rate):
    """Portions of one token, of less than a tile, of whole tiles and more, of several requests in one step, from a
    slot's state on; decays next to 1 (rate -3) and decays that vanish within a tile (rate 3)."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(heads * dim + vdim)
    lengths = {3: 90, 0: 35, 6: 4}
    cols = 2 * qk * dim + heads * vdim
    pad = -(-cols // 8) * 8
    data = {}
    for s, n in lengths.items():
        qkv = dev(rng.normal(size=(n, pad)), dtype)
        b = dev(rng.normal(size=(n, heads)) * 2, dtype)
        z = dev(rng.normal(size=(n, heads * dim)) * 2)
        data[s] = (qkv, b, z)
    a_log, dt = rng.uniform(rate - 1, rate, size=heads), rng.uniform(-3, 0, size=heads * dim)
    share = np.arange(heads) // (heads // qk)
    want, want_state = {}, {}
    for s, (qkv, b, z) in data.items():
        x, n = host(qkv), lengths[s]
        q = plain.unit_vectors(x[:, :qk * dim].reshape(n, qk, dim))[:, share] * dim ** -0.5
        k = plain.unit_vectors(x[:, qk * dim:2 * qk * dim].reshape(n, qk, dim))[:, share]
        v = x[:, 2 * qk * dim:cols].reshape(n, heads, vdim)
        g = np.exp(-np.exp(a_log)[None, :, None] * plain.softplus((host(z) + dt).reshape(n, heads, dim)))
        want[s] = plain.channel_delta_scan(q, k, v, plain.sigmoid(host(b)), g).reshape(n, heads * vdim)
    state = torch.full((8, heads, dim, vdim), 5.0, device=DEV)
    for s in lengths:
        state[s].zero_()
    at, got = {s: 0 for s in lengths}, {s: [] for s in lengths}
    ws = torch.empty(ops.channel_delta_workspace(8, 128, heads, dim, vdim), device=DEV)
    for sizes in ({3: 1, 0: 1}, {0: 2, 3: 17}, {6: 1, 3: 33, 0: 16}, {3: 1, 0: 1, 6: 1}, {0: 15, 6: 2, 3: 38}):
        slots = list(sizes)
        step = make_step(list(sizes.values()), lengths=[at[s] for s in slots], slots=slots)
        qkv, b, z = (torch.cat([data[s][i][at[s]:at[s] + n] for s, n in sizes.items()]) for i in range(3))
        out = torch.full((step.n, heads * vdim), 7.0, device=DEV)
        before = state.clone()
        args = (qkv, 0, qk * dim, 2 * qk * dim, b, z, dev(a_log), dev(dt), state, step, out, heads, qk, dim, vdim)
        ops.channel_delta(*args, False, ws)
        assert torch.equal(before, state)                                         # a reader only
        first = out.clone()
        ops.channel_delta(*args, True, ws)
        assert torch.equal(first, out)
        o, i = host(out), 0
        for s, n in sizes.items():
            got[s].append(o[i:i + n]); i += n; at[s] += n
    for s in lengths:
        assert close(np.concatenate(got[s]), want[s], 2e-5), s
    assert torch.all(state[[1, 2, 4, 5, 7]] == 5.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("heads,dim,rot,rank", [(4, 16, 8, 24), (3, 5, 2, 7), (1, 32, 40, 130)])
def test_latent_attend_prepare(dtype, interleaved, heads, dim, rot, rank):
    """The cached vector (normed latent, rotated tail) on its page, and the queries' rotated parts in their places."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(rank)
    page, n0, n = 16, 21, 13                                                      # across a page's edge
    qc = heads * (dim + rot)
    proj = dev(rng.normal(size=(n, qc + rank + rot + 3)), dtype)
    w = rng.normal(size=rank) + 1
    x = host(proj)
    f = np.array([300.0 ** (-2.0 * i / rot) for i in range(rot // 2)])
    step = make_step([n], lengths=[n0], slots=[1])
    cs = torch.empty((n, rot // 2, 2), device=DEV)
    ops.rope_table(step.positions, dev(f, torch.float64), cs)
    table = torch.tensor([[5, 2, 7, -1], [3, 0, 6, 4], [-1] * 4, [-1] * 4], dtype=torch.int32, device=DEV)
    pool = torch.zeros((8, 1, page, rank + rot), dtype=dtype, device=DEV)
    stride = rank + rot + 1
    q_out = torch.full((n, heads * stride), 2.0, dtype=dtype, device=DEV)
    ops.latent_attend_prepare(proj, qc, rank, rot, interleaved, dev(w), 1e-4, cs, step, heads, dim, dim + rot, q_out, rank, stride,
                              pool, table, page)
    perm = np.arange(rot) if interleaved else np.arange(rot).reshape(2, rot // 2).T.reshape(-1)

    def turned(part):                                                             # [n, h, rot] at positions n0..
        full = np.zeros((n0 + n,) + part.shape[1:]); full[n0:] = part[..., perm]
        out = np.zeros_like(part); out[..., perm] = plain.rotate(full, rot, 300.0)[n0:]
        return out
    want_q = turned(x[:, :qc].reshape(n, heads, dim + rot)[..., dim:])
    want_c = np.concatenate([plain.unit_rms(x[:, qc:qc + rank], 1e-4) * w, turned(x[:, None, qc + rank:qc + rank + rot])[:, 0]], axis=1)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    q = host(q_out).reshape(n, heads, stride)
    assert close(q[..., rank:rank + rot], want_q, tol) and np.all(q[..., :rank] == 2.0) and np.all(q[..., -1] == 2.0)
    cells = [host(pool[[3, 0, 6, 4][p // page], 0, p % page]) for p in range(n0, n0 + n)]
    assert close(np.stack(cells), want_c, tol) and torch.count_nonzero(pool[[1, 2, 5, 7]]) == 0
    q2 = torch.full_like(q_out, 2.0)
    ops.latent_attend_prepare(proj, qc, rank, rot, interleaved, dev(w), 1e-4, cs, step, heads, dim, dim + rot, q2, rank, stride, None, table, page)
    assert torch.equal(q_out, q2)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dk,dv,window", [(5, 80, 64, 0), (2, 32, 16, 0), (70, 48, 32, 40), (3, 144, 128, 25), (4, 320, 256, 0)])
@pytest.mark.parametrize("level", [None, 0.0, 60.0, -300.0])
def test_latent_attention_with_a_sink(dtype, heads, dk, dv, window, level):
    """A prompt portion behind cached tokens, single tokens with their keys in one piece and split among blocks (also
    into more pieces than there are key blocks); sinks of the scores' size, far above and far below them."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(heads + dk)
    page, before, new = 16, [300, 37, 0], [1, 1, 1]
    pages = 24
    table = torch.tensor(rng.permutation(3 * pages).reshape(3, pages), dtype=torch.int32, device=DEV)
    pool = torch.full((3 * pages, 1, page, dk), 50.0, dtype=dtype, device=DEV)    # stale content where no key lies
    keys = [dev(rng.normal(size=(b + 40, dk)), dtype) for b in before]
    for r in range(3):
        for p in range(before[r] + 40):
            pool[table[r, p // page], 0, p % page] = keys[r][p]
    sink = None if level is None else level + rng.normal(size=heads)

    def want(r, pos, q):
        lo = max(0, pos - window + 1) if window else 0
        k = host(keys[r])[lo:pos + 1]
        out = np.zeros((heads, dv))
        for h in range(heads):
            s = (k @ q[h]) * 0.2
            p = plain.sink_softmax(s[None], sink[h] if sink is not None else -np.inf)[0]
            out[h] = p @ k[:, :dv]
        return out.reshape(-1)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    scratch = torch.empty(32 * 3 * heads * (dv + 2), device=DEV)
    dev_sink = None if sink is None else dev(sink)
    for counts in (new, [23, 1, 40]):
        step = make_step(counts, lengths=before, slots=[0, 1, 2])
        q = dev(rng.normal(size=(step.n, heads * dk)), dtype)
        qh = host(q).reshape(step.n, heads, dk)
        ref = np.stack([want(r, before[r] + t, qh[sum(counts[:r]) + t]) for r in range(3) for t in range(counts[r])])
        scale = np.max(np.abs(ref))
        for splits in (1, None, 3, 32):
            out = torch.full((step.n, heads * dv), 9.0, dtype=dtype, device=DEV)
            step.attention_splits, step.planning_context = splits, step.max_context
            ops.latent_attention(q, pool, table, page, step, out, heads, dk, dv, 0.2, window, dev_sink, scratch)
            assert np.max(np.abs(host(out) - ref)) <= tol * max(scale, 1e-3), (counts, splits)


@pytest.mark.parametrize("heads,dk,dv,window", [(8, 112, 64, 0), (32, 288, 256, 0), (3, 144, 128, 70), (128, 80, 64, 0), (5, 576, 512, 0),
                                                (16, 320, 320, 33), (1, 64, 64, 0)])
@pytest.mark.parametrize("page", [64, 128])
def test_latent_attention_of_prompt_portions(heads, dk, dv, window, page):
    """The tcgen05 kernel: portions that start at 0, inside a key block and at its edge, beside a single token and a short
    portion; pages in any order with stale not-a-numbers wherever no key of the request lies; sinks of every size."""
    from hfee_b200.kernels import ops
    rng = np.random.default_rng(dk + heads)
    assert ops.latent_tc_supports(heads, dk, dv, page)
    before, new = [0, 64, 131, 200], [150, 67, 1, 9]
    pages = 4
    table = torch.tensor(rng.permutation(4 * pages).reshape(4, pages), dtype=torch.int32, device=DEV)
    pool = torch.full((4 * pages, 1, page, dk), float("nan"), dtype=torch.bfloat16, device=DEV)
    keys = [dev(rng.normal(size=(b + n, dk)), torch.bfloat16) for b, n in zip(before, new)]
    for r in range(4):
        for p in range(before[r] + new[r]):
            pool[table[r, p // page], 0, p % page] = keys[r][p]
    step = make_step(new, lengths=before, slots=[0, 1, 2, 3])
    q = dev(rng.normal(size=(step.n, heads * dk)), torch.bfloat16)
    qh, scale = q.float().reshape(step.n, heads, dk), 2.0 * dk ** -0.5
    for level in (None, 0.0, 40.0):
        sink = None if level is None else dev(level + rng.normal(size=heads))
        want, at = [], 0
        for r in range(4):
            k = keys[r].float()
            s = torch.einsum("thd,kd->htk", qh[at:at + new[r]].double(), k.double()) * scale
            pos = torch.arange(before[r], before[r] + new[r], device=DEV)[:, None]
            j = torch.arange(k.shape[0], device=DEV)[None]
            s = s.masked_fill(~((j <= pos) & ((j > pos - window) if window else (j >= 0)))[None], -torch.inf)
            if sink is not None:
                s = torch.cat([s, sink.double()[:, None, None].expand(heads, new[r], 1)], dim=2)
            w = torch.softmax(s, dim=2)[:, :, :k.shape[0]]
            want.append(torch.einsum("htk,kd->thd", w, k[:, :dv].double()).reshape(new[r], heads * dv))
            at += new[r]
        want = torch.cat(want)
        out = torch.full((step.n, heads * dv), 9.0, dtype=torch.bfloat16, device=DEV)
        ops.latent_attention(q, pool, table, page, step, out, heads, dk, dv, scale, window, sink)
        err = (out.double() - want).abs()
        assert torch.isfinite(out).all() and float(err.max()) <= 1.5e-2 * max(float(want.abs().max()), 1e-2), level
    ops.check_status()
