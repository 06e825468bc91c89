"""Fokalorn on the CPU: configuration and its errors, the run order, tensor names, what each layer asks of the cache
manager, and the plain implementation's own consistency."""
import copy

import numpy as np
import pytest

import fokalorn_util as fu
import plain_fokalorn as plain


def resolved(cfg):
    from hfee_b200.config.registry import resolve
    return resolve(fu.with_ranks(cfg))


def test_config_reads_every_size_and_constant():
    arch, c = resolved(fu.FOK_A)
    assert arch.name == "Fokalorn" and (c.vocab, c.width, c.streams, c.groups, c.eps, c.embedding_scale) == (200, 64, 3, 4, 1e-5, 3.0)
    assert (c.loop.start, c.loop.stop, c.loop.times) == (1, 3, 3)
    m = c.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.taps, m.decay_rank, m.gate_rank) == (4, 2, 16, 24, 4, 6, 10)
    m = c.layers[1].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.scale, m.rot_base) == (4, 24, 8, 16, 40, 0.3, 500.0)
    assert c.layers[1].mlp.ff == 96
    _, b = resolved(fu.FOK_B)
    assert b.loop is None and b.layers[0].mlp is None and (b.layers[1].mixer.decay_rank, b.layers[1].mixer.gate_rank) == (3, 17)


def test_run_order_gives_every_pass_a_cache_of_its_own():
    for loop, want in (((1, 3, 3), [0, 1, 2, 1, 2, 1, 2, 3]), ((0, 4, 2), [0, 1, 2, 3, 0, 1, 2, 3]), ((3, 4, 3), [0, 1, 2, 3, 3, 3]),
                       ((2, 2, 5), [0, 1, 2, 3]), (None, [0, 1, 2, 3])):
        cfg = dict(fu.FOK_A, loop=None if loop is None else {"start": loop[0], "stop": loop[1], "times": loop[2]})
        arch, c = resolved(cfg)
        sched = arch.build_spec(c).schedule
        assert [r.layer for r in sched] == want == plain.run_order(cfg)
        assert [r.cache for r in sched] == list(range(len(want))) and not any(r.adds_embedding for r in sched)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="delta"), "not a mixer of this design"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "not a feed-forward of this design"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), "equal rot_dim"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "positive integer"),
    (lambda c: c["norm"].update(groups=5), "does not divide"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c["embedding"].pop("scale"), "scale"),
    (lambda c: c["loop"].update(stop=9), "does not fit"),
    (lambda c: c["layers"][2]["mixer"].pop("conv"), "conv"),
])
def test_config_errors_name_the_key(change, message):
    from hfee_b200.config.llama import ConfigError
    cfg = copy.deepcopy(fu.FOK_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        resolved(cfg)


def test_the_ranks_come_from_the_tensors():
    from hfee_b200.config.llama import ConfigError
    from hfee_b200.config.registry import resolve
    with pytest.raises(ConfigError, match="rank"):
        resolve(fu.stored(fu.FOK_A))
    shapes = {"l0.mix.a1": (11, 64), "l0.mix.g1": (5, 64), "l2.mix.a1": (7, 64), "l2.mix.g1": (9, 64)}
    _, c = resolve(fu.stored(fu.FOK_A), shapes)
    assert [(c.layers[i].mixer.decay_rank, c.layers[i].mixer.gate_rank) for i in (0, 2)] == [(11, 5), (7, 9)]


def test_tensor_names_and_shapes():
    from hfee_b200.parts.model import model_tensor_needs
    arch, c = resolved(fu.FOK_A)
    needs = model_tensor_needs(arch.build_spec(c))
    shape = lambda n: tuple(needs[n].shape)
    assert shape("embed") == (200, 64) == shape("head") and shape("final.norm") == (64,)
    assert shape("l0.mix.q") == (32, 64) and shape("l0.mix.v") == (96, 64) and shape("l0.mix.k.conv") == (32, 4)
    assert shape("l0.mix.a1") == (6, 64) and shape("l0.mix.a2") == (64, 6) and shape("l0.mix.dt_bias") == (64,) and shape("l0.mix.A_log") == (4,)
    assert shape("l0.mix.g1") == (10, 64) and shape("l0.mix.g2") == (96, 10) and shape("l0.mix.norm") == (24,) and shape("l0.mix.b") == (4, 64)
    assert shape("l1.mix.q") == (4 * 32, 64) and shape("l1.mix.dkv") == (48, 64) and shape("l1.mix.uk") == (96, 40) and shape("l1.mix.sink") == (4,)
    assert shape("l1.mix.g") == (4, 64) and shape("l1.hc2.mix") == (3, 3) and shape("l1.shift") == (64,) and shape("l1.mlp.up") == (96, 64)
    _, b = resolved(fu.FOK_B)
    spec = arch.build_spec(b)
    needs = model_tensor_needs(spec)
    assert "l0.norm2" not in needs and "l0.hc2.in" not in needs and "l0.norm2" in spec.ignorable and "l1.norm2" in needs


def test_cache_needs_per_run():
    """Pages of [latent | rotated part] where a layer attends; float32 states for the convolution, the recurrence and the
    row of the token before; every pass of a looped layer has its own, and a slot that is taken again starts at zero."""
    import torch
    from hfee_b200.cache import CacheManager
    from hfee_b200.cache.needs import CacheBundle, FixedState, PagedKV
    needs = {0: CacheBundle.of(None, conv=FixedState((3, 160)), recurrent=FixedState((4, 16, 24)), shift=FixedState((64,))),
             1: CacheBundle.of(PagedKV(1, 48, None, None, 0), shift=FixedState((64,))),
             2: CacheBundle.of(PagedKV(1, 48, None, None, 0), shift=FixedState((64,)))}
    m = CacheManager(needs, 16, 12, 3, 96, torch.float32)
    assert m.view(1).k.shape == (12, 1, 16, 48) and m.view(1).v is None and m.view(1).k.data_ptr() != m.view(2).k.data_ptr()
    assert tuple(m.view(0).states["shift"].shape) == (3, 64) and m.view(0).states["shift"].data_ptr() != m.view(1).states["shift"].data_ptr()
    s = m.open()
    m.reserve(s, 40); m.commit(s, 40); m.check_invariants()
    for t in m.view(0).states.values():
        t[s].fill_(3.0)
    m.close(s)
    assert m.open() == s and all(float(t[s].abs().sum()) == 0.0 for t in m.view(0).states.values())


def test_streams_and_blocks_must_fit():
    from hfee_b200.config.spec import PartSpec
    from hfee_b200.parts.base import part_class
    cls = part_class("block", "hyper_connected")
    assert cls.on_streams and not getattr(part_class("block", "pre_norm"), "on_streams", False)
    with pytest.raises(ValueError, match="mixer_streams"):
        cls(PartSpec("hyper_connected", width=8), {}, None, {"mixer": None, "mixer_norm": None})
    with pytest.raises(ValueError, match="divide"):
        part_class("norm", "group_rms_norm")(PartSpec("group_rms_norm", width=10, eps=1e-5, groups=3), {"weight": None}, None)


# ------------------------------------------------------------------ the plain implementation against itself
def test_channel_delta_scan_equals_its_tiled_form():
    """The recurrence against the triangular system over a whole sequence from a zero state."""
    rng = np.random.default_rng(0)
    T, d, dv = 11, 5, 4
    q, k, v = rng.normal(size=(T, 1, d)), plain.unit_vectors(rng.normal(size=(T, 1, d))), rng.normal(size=(T, 1, dv))
    beta, g = rng.uniform(size=(T, 1)), rng.uniform(0.3, 1.0, size=(T, 1, d))
    o = plain.channel_delta_scan(q, k, v, beta, g)[:, 0]
    L = np.cumsum(np.log(g[:, 0]), axis=0)
    ratio = np.exp(L[:, None] - L[None, :])
    A = np.tril(np.einsum("td,tjd,jd->tj", k[:, 0], ratio, k[:, 0]), -1)
    B = np.tril(np.einsum("td,tjd,jd->tj", q[:, 0], ratio, k[:, 0]))
    u = np.linalg.solve(np.eye(T) + beta * A, beta * v[:, 0])
    assert np.allclose(o, B @ u)


def test_token_shift_and_streams():
    h = np.arange(6.0).reshape(3, 2)
    assert np.allclose(plain.token_shift(h, np.array([1.0, 0.25])), [[0, 0.75], [0, 2.5], [2, 4.5]])
    X = np.random.default_rng(1).normal(size=(3, 4, 5))
    y = np.ones((4, 5))
    M, b = np.zeros((3, 3)), np.array([1.0, 0.0, 2.0])
    M[0, 1] = 1.0                                    # from stream 0 to stream 1
    out = plain.spread_streams(X, M, b, y)
    assert np.allclose(out[0], y) and np.allclose(out[1], X[0]) and np.allclose(out[2], 2 * y)
    assert np.allclose(plain.collect_streams(X, b), X[0] + 2 * X[2])


def test_group_norm_and_sink():
    x = np.array([[3.0, 4.0, 0.0, 2.0]])
    assert np.allclose(plain.group_norm(x, np.array([1, 1, 1, 2.0]), 0.0, 2), [[3 / 12.5 ** .5, 4 / 12.5 ** .5, 0, 2 * 2 ** .5]])
    s = np.array([[0.0, -np.inf], [1.0, 2.0]])
    p = plain.sink_softmax(s, 0.0)
    assert np.allclose(p[0], [0.5, 0.0]) and np.allclose(p[1].sum(), (np.e + np.e ** 2) / (1 + np.e + np.e ** 2))


def test_rotation_keeps_relative_angles():
    rng = np.random.default_rng(3)
    a, b = rng.normal(size=8), rng.normal(size=8)
    x = np.zeros((12, 1, 8)); x[:] = a
    y = np.zeros((12, 1, 8)); y[:] = b
    rx, ry = plain.rotate(x, 8, 50.0)[:, 0], plain.rotate(y, 8, 50.0)[:, 0]
    assert np.allclose(rx[5] @ ry[2], rx[11] @ ry[8]) and np.allclose(rx[0], a)
    assert np.allclose(rx[1, :2], [a[0] * np.cos(1) - a[1] * np.sin(1), a[1] * np.cos(1) + a[0] * np.sin(1)])
