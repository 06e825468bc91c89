"""Bumisun on the CPU: configuration and its errors, tensor names, what each layer asks of the cache manager, pages of first
tokens that stay behind a window, and the plain implementation's own consistency."""
import copy

import numpy as np
import pytest

import bumisun_util as bu
import plain_bumisun as plain


def resolved(cfg):
    from hfee_b200.config.registry import resolve
    return resolve(copy.deepcopy(cfg))


def test_config_reads_every_size_and_constant():
    arch, c = resolved(bu.BUM_A)
    assert arch.name == "Bumisun" and (c.vocab, c.width, c.eps, c.residual_mult, c.logit_scale) == (200, 64, 1e-5, 0.6, 1.7)
    a = c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.window, a.keep_first) == (4, 2, 16, 24, 0.3, 4.0, 21, 5)
    assert (a.rot_dims, a.rot_base, a.v_mix) == (8, 1000.0, True) and c.layers[0].mlp.ff == 80 and not c.layers[3].mixer.v_mix
    m = c.layers[1].mixer
    assert (m.heads, m.vdim, m.state, m.groups, m.taps, m.norm_groups) == (4, 24, 16, 2, 3, 2)
    f = c.layers[1].mlp
    assert (f.experts, f.top, f.expert.ff, f.expert.limit, f.shared.ff, f.shared.limit) == (6, 2, 24, 0.9, 40, 1.1)
    assert c.layers[2].mlp.shared is None and c.layers[3].mlp is None
    _, b = resolved(bu.BUM_B)
    a = b.layers[1].mixer
    assert a.window is None and a.softcap is None and a.rot_dims == 0 and a.keep_first == 0


def test_no_rotation_means_no_rotation():
    arch, c = resolved(bu.BUM_B)
    spec = arch.build_spec(c)
    assert spec.layers[1].parts["mixer"][1].position.kind == "none" and spec.layers[2].parts["mixer"][1].position.rope_dim == 16


def test_the_first_layer_that_mixes_values_is_not_the_first_layer():
    for cfg, kinds in ((bu.BUM_A, ["first", "mixed", None, "mixed"]), (bu.BUM_B, [None, "first", "mixed"])):
        arch, c = resolved(cfg)
        mixers = [l.parts["mixer"][1] for l in arch.build_spec(c).layers]
        assert [m.value_mix for m in mixers if m.kind == "softmax_attention"] == kinds


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="mamba"), "not a mixer of this design"),
    (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "not a feed-forward of this design"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "at most dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0.0), "must be positive"),
    (lambda c: c["layers"][0]["mixer"].update(v_mix="yes"), "true or false"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "positive integer"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("keep_first"), "keep_first"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=16), "values of one size"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "multiple of groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "does not divide"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "exceeds"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(limit=-1.0), "must be positive"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "limit"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_config_errors_name_the_key(change, message):
    from hfee_b200.config.llama import ConfigError
    cfg = copy.deepcopy(bu.BUM_A)
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        resolved(cfg)


def test_tensor_names_and_shapes():
    from hfee_b200.parts.model import model_tensor_needs
    arch, c = resolved(bu.BUM_A)
    spec = arch.build_spec(c)
    needs = model_tensor_needs(spec)
    shape = lambda n: tuple(needs[n].shape)
    assert shape("embed") == (200, 64) and shape("embed.norm") == shape("final.norm") == (64,) and shape("head") == (200, 64)
    assert shape("l0.mix.q") == (64, 64) and shape("l0.mix.v") == (48, 64) and shape("l0.mix.o") == (64, 96) and shape("l0.mix.sink") == (4,)
    assert shape("l2.mix.vmix") == () and needs["l0.mix.vmix"].optional and not needs["l2.mix.vmix"].optional and "l3.mix.vmix" not in needs
    assert shape("l1.mix.in") == (2 * 96 + 2 * 32 + 4, 64) and shape("l1.mix.conv") == (160, 3) and shape("l1.mix.conv.b") == (160,)
    assert shape("l1.mix.dt_bias") == shape("l1.mix.A_log") == shape("l1.mix.D") == (4,) and shape("l1.mix.norm") == (96,)
    assert shape("l1.mlp.router.b") == (6,) and shape("l1.mlp.shared.sg") == (1, 64) and shape("l1.mlp.e5.down") == (64, 24)
    assert "l2.mlp.shared.sg" not in needs and "l3.norm2" not in needs and "l3.norm2" in spec.ignorable and "l3.mix.vmix" in spec.ignorable
    assert needs["l1.mix.A_log"].role == needs["l0.mix.sink"].role == "vector" and needs["l1.mix.norm"].role == "scale"


def test_cache_needs_of_the_mixers():
    from hfee_b200.cache.needs import CacheBundle, FixedState, PagedKV
    from hfee_b200.parts.base import part_class
    arch, c = resolved(bu.BUM_A)
    layers = arch.build_spec(c).layers

    def need(i):
        spec = layers[i].parts["mixer"][1]
        part = object.__new__(part_class("mixer", spec.kind))
        part.__dict__.update(kv_heads=spec.get("kv_heads"), value_dim=spec.get("value_dim"), window=spec.get("window"), keep_first=spec.get("keep_first"),
                             head_dim=spec.head_dim, taps=spec.get("taps"), heads=spec.heads, n_state=spec.get("state"),
                             conv_cols=0 if spec.kind != "head_scan" else spec.heads * spec.head_dim + 2 * spec.groups * spec.state)
        return part.cache_need()
    assert need(0) == PagedKV(2, 16, 21, None, 24, 5) and need(3) == PagedKV(1, 24, 34, None, 40, 17)
    assert need(1) == CacheBundle.of(None, conv=FixedState((2, 160), "float32"), recurrent=FixedState((4, 16, 24), "float32"))


@pytest.mark.parametrize("keep,page,window", [(0, 16, 21), (1, 16, 21), (16, 16, 5), (17, 16, 40), (40, 16, 21), (200, 16, 8), (3, 64, 30)])
def test_pages_of_first_tokens_stay_behind_the_window(keep, page, window):
    """Every page that a later token can read is held, the others go back, in steps of several sizes; a closed request holds
    nothing and its pages and slot are used again."""
    import torch
    from hfee_b200.cache import CacheManager
    from hfee_b200.cache.needs import PagedKV
    m = CacheManager({0: PagedKV(1, 8, window, None, 8, keep), 1: PagedKV(1, 8)}, page, 40, 2, 400, torch.float32)
    windowed = m.paged[0]
    for _ in range(2):
        s = m.open()
        length = 0
        for n in (1, 2, page - 3, 1, 1, 50, 3, page, 1, 40, 2, 77):
            m.reserve(s, length + n); m.commit(s, length + n)
            length += n
            m.check_invariants()
            needed = {p // page for p in range(length) if p < keep or length - p < window}
            held = {i for i, p in enumerate(windowed.table[s]) if p >= 0}
            assert needed <= held and all(h in needed or h * page >= length - window - page + 1 or h < -(-keep // page) for h in held)
        assert len(held) <= -(-keep // page) + window // page + 2
        assert int((m.paged[1].table[s] >= 0).sum()) == -(-length // page)
        m.close(s)
        assert m.free_pages() == 40


# ------------------------------------------------------------------ the plain implementation against itself
def test_the_scan_equals_its_closed_form():
    rng = np.random.default_rng(0)
    T, H, N, dv = 9, 2, 3, 4
    x, B, C = rng.normal(size=(T, H, dv)), rng.normal(size=(T, H, N)), rng.normal(size=(T, H, N))
    dt, A, D = rng.uniform(0.1, 1.0, size=(T, H)), rng.uniform(0.1, 2.0, size=H), rng.normal(size=H)
    y = plain.head_scan(x, B, C, dt, A, D)
    for h in range(H):
        for t in range(T):
            want = D[h] * x[t, h]
            for u in range(t + 1):
                want = want + np.exp(-A[h] * dt[u + 1:t + 1, h].sum()) * dt[u, h] * (C[t, h] @ B[u, h]) * x[u, h]
            assert np.allclose(y[t, h], want)


def test_the_mask():
    seen = plain.visible(12, 4, 2)
    for i in range(12):
        assert [j for j in range(12) if seen[i, j]] == sorted({j for j in range(i + 1) if i - j < 4 or j < 2})
    assert np.array_equal(plain.visible(6, None, 0), np.tril(np.ones((6, 6), dtype=bool))) and np.array_equal(plain.visible(6, 6, 0), plain.visible(6, None, 0))


def test_cap_sink_and_rotation():
    s = np.array([0.0, 1e-3, 5.0, -80.0])
    assert np.allclose(plain.cap(s, 2.0), [0.0, 1e-3, 2 * np.tanh(2.5), -2.0]) and plain.cap(s, None) is s
    w = plain.sink_softmax(np.array([[1.0, 2.0, -np.inf]]), 0.5)[0]
    assert np.allclose(w, np.exp([1.0, 2.0, -np.inf]) / (np.exp(1) + np.exp(2) + np.exp(0.5)))
    x = np.random.default_rng(1).normal(size=(5, 2, 6))
    y = plain.rotate(x, 4, 10.0)
    assert np.allclose(y[0], x[0]) and np.allclose(y[..., 4:], x[..., 4:])
    assert np.allclose(y[3, :, 1], x[3, :, 1] * np.cos(3 * 10 ** -0.5) - x[3, :, 3] * np.sin(3 * 10 ** -0.5))


def test_the_router_and_the_values_of_the_first_layer():
    chosen, weight = plain.choose(np.array([[1.0, 3.0, 2.0, 3.0]]), 3)
    assert chosen.tolist() == [[1, 3, 2]] and np.allclose(weight, np.exp([3.0, 3.0, 2.0]) / np.exp([3.0, 3.0, 2.0]).sum())
    assert np.allclose(plain.mix_values(np.array([2.0]), np.array([6.0]), 0.25), 3.0)


def test_greedy_and_prefixes(tmp_path):
    d = bu.write_model(str(tmp_path), bu.BUM_A, seed=1)
    c, w = plain.load(d)
    seq = bu.sequences(200, (40,), seed=2)[0]
    whole = plain.forward(c, w, seq)
    assert np.allclose(plain.forward(c, w, seq[:17]), whole[:17])              # nothing looks ahead
    out = plain.greedy(c, w, seq[:3], 4)
    assert len(out) == 4 and out[0] == int(np.argmax(whole[2]))
