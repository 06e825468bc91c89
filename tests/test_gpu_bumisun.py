"""The Bumisun decoder on the GPU against the plain implementation of tests/plain_bumisun.py: each mixer and feed-forward
alone, whole prompts, prefill then token by token, portions down to two tokens, mixed batches over few pages and slots,
window and page edges, kept first tokens, far keys and far writes, mixed values, long decoding, other sizes, and greedy
generation through the engine's entry point."""
import numpy as np
import pytest

import bumisun_util as bu
import plain_bumisun as plain
import replay_util as ru

pytestmark = pytest.mark.gpu

# Largest |difference| relative to the largest |logit| of the plain float64 result on the same stored weights,
# and the root mean square of the differences relative to that of the logits.  float32: rounding of float32
# sums only.  bfloat16: activations between kernels are rounded to 8 bits of mantissa.
TOL = {"float32": 1e-4, "bfloat16": 4e-2}
RMS_TOL = {"float32": 2e-5, "bfloat16": 1.5e-2}
LENGTHS = (5, 17, 33, 100, 1, 71, 40, 9)


def rms_err(got, ref):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    return float(np.sqrt(np.mean((got - ref) ** 2)) / (np.sqrt(np.mean(ref ** 2)) + 1e-30))


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg, seed in (("A", bu.BUM_A, 4), ("B", bu.BUM_B, 10)):
        d = bu.write_model(str(tmp_path_factory.mktemp("bumisun" + name)), cfg, seed)
        c, w = plain.load(d)
        seqs = bu.sequences(cfg["vocab"], LENGTHS, seed=11)
        assert bu.smallest_route_margin(plain, c, w, seqs) > 0.5          # no router's choice is a close call
        out[name] = (d, cfg, seqs, [plain.forward(c, w, s) for s in seqs])
    return out


def check(got, ref, dtype, what="", rms_tol=None):
    assert sorted(got) == list(range(len(ref)))
    for i in range(len(ref)):
        assert got[i].shape == ref[i].shape
        err, rms = ru.rel_err(got[i], ref[i]), rms_err(got[i], ref[i])
        assert err < TOL[dtype] and rms < (rms_tol or RMS_TOL[dtype]), f"{what} request {i}: relative error {err:.3g}, rms {rms:.3g}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
@pytest.mark.parametrize("scheme", ["whole", "prefill_then_decode", "portions", "mixed"])
def test_replay(models, name, dtype, scheme):
    d, cfg, seqs, ref = models[name]
    if scheme == "mixed":
        steps = ru.mixed(seqs, live=4, seed=2)
        # the four longest at once need 100+71+40+33 -> 17 pages of 16 with rounding; slots and pages are used again
        runner = bu.make_runner(d, dtype, max_tokens=17 * 16, context=112)
    else:
        steps = {"whole": ru.whole, "prefill_then_decode": lambda s: ru.prefill_then_decode(s, tail=20),
                 "portions": ru.portions}[scheme](seqs)
        runner = bu.make_runner(d, dtype, max_tokens=112, max_requests=1)
    check(ru.run_in_process(runner, steps), ref, dtype, scheme)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_pages_of_64(models, name, dtype):
    """Pages of whole key blocks: long portions beside short ones and single tokens, in and across key blocks and runs."""
    d, cfg, _, _ = models[name]
    c, w = plain.load(d)
    seqs = bu.sequences(cfg["vocab"], (300, 130, 65, 64), seed=12)
    ref = [plain.forward(c, w, s) for s in seqs]
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(130, 2, 63, 1, 64)), ru.mixed(seqs, live=3, seed=4, chunk_sizes=(2, 40, 64, 90))):
        check(ru.run_in_process(bu.make_runner(d, dtype, 10 * 64, page_size=64, max_requests=3, context=320), steps), ref, dtype)


def test_batch_of_unequal_requests_equals_each_alone(models):
    """float32: a row's sums hardly depend on what else is in the batch (the scan takes runs of tokens side by side in long
    portions only)."""
    d, cfg, seqs, ref = models["A"]
    alone = ru.run_in_process(bu.make_runner(d, "float32", 112, max_requests=1), ru.whole(seqs))
    runner = bu.make_runner(d, "float32", max_tokens=512, max_requests=8, context=112)
    steps = [{"entries": [(i, s, list(range(len(s)))) for i, s in enumerate(seqs)], "end": list(range(len(seqs)))}]
    together = ru.run_in_process(runner, steps)
    for i in range(len(seqs)):
        assert ru.rel_err(together[i], alone[i]) < 5e-6


A, M = bu.attn, bu.mamba
ALONE = {
    "attention_plain": [A(4, 2, 16, 16)],
    "attention_everything": [A(6, 3, 24, 8, 19, 7, rot=12, base=70.0, softcap=1.5)],
    "attention_tensor_core_sizes": [A(8, 2, 64, 64, 70, 3, rot=64, softcap=5.0)],
    "attention_head_size_128": [A(2, 1, 128, 128, 33, 1, rot=64, softcap=5.0, scale=0.1)],
    "attention_one_head_window_of_one": [A(1, 1, 8, 40, 1, 1, rot=2, softcap=3.0)],
    "attention_more_kept_than_window": [A(3, 1, 16, 24, 6, 30, rot=16, softcap=4.0)],
    "attention_many_heads": [A(34, 2, 8, 16, 12, 2, softcap=2.0)],
    "values_mixed_twice": [A(2, 1, 16, 24, 30, 2, rot=8, softcap=6.0, v_mix=True), A(4, 1, 8, 24, 9, 1, v_mix=True), A(1, 1, 16, 24, v_mix=True)],
    "scan": [M(4, 16, 16, 1, 4, 1)],
    "scan_groups_and_parts": [M(6, 8, 24, 3, 3, 4)],
    "scan_wide_heads": [M(1, 136, 72, 1, 2, 1)],
    "scan_one_column": [M(3, 1, 8, 3, 2, 1)],
    "scan_large_state": [M(2, 24, 136, 2, 1, 2)],
    "dense": [M(2, 8, 8, 1, 2, 1, mlp=bu.dense(72))],
    "moe_every_expert": [M(2, 8, 8, 1, 2, 1, mlp=bu.moe(3, 3, 24, 0.8))],
    "moe_shared": [A(2, 1, 8, 8, mlp=bu.moe(5, 2, 16, 1.2, 40, 0.5))],
    "moe_one_expert": [A(2, 1, 8, 8, mlp=bu.moe(1, 1, 40, 2.0, 8, 3.0))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layers", list(ALONE.values()), ids=list(ALONE))
def test_each_mechanism_alone(tmp_path, layers, dtype):
    """A layer or two: whole, and in portions through the cache or state."""
    cfg = bu.config(48, 90, layers, residual_mult=0.9, logit_scale=1.3)
    d = bu.write_model(str(tmp_path), cfg, seed=7)
    c, w = plain.load(d)
    seqs = bu.sequences(90, (37, 3, 64, 90), seed=5)
    assert bu.smallest_route_margin(plain, c, w, seqs) > 0.5
    ref = [plain.forward(c, w, s) for s in seqs]
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(2, 9, 1, 1, 30, 2))):
        check(ru.run_in_process(bu.make_runner(d, dtype, 96, max_requests=1), steps), ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_fit_no_vector_access(tmp_path, dtype):
    """Width, vocabulary and head sizes that are multiples of neither 8 nor 4: every kernel takes its scalar path."""
    layers = [A(3, 1, 10, 14, 11, 3, rot=6, base=77.0, softcap=3.0, v_mix=True, mlp=bu.moe(5, 2, 14, 0.8, 18, 1.1)),
              M(3, 7, 5, 1, 3, 3, mlp=bu.dense(30)), A(2, 1, 6, 14, v_mix=True), M(2, 11, 13, 2, 2, 1, mlp=bu.moe(3, 1, 10, 1.3))]
    cfg = bu.config(50, 77, layers, eps=3e-6, residual_mult=0.8, logit_scale=0.9)
    d = bu.write_model(str(tmp_path), cfg, seed=13)
    c, w = plain.load(d)
    seqs = bu.sequences(77, (41, 2, 19, 70), seed=6)
    assert bu.smallest_route_margin(plain, c, w, seqs) > 0.5
    ref = [plain.forward(c, w, s) for s in seqs]
    rms_tol = 2.5e-2 if dtype == "bfloat16" else None       # short sums average less of the rounding than wider models' do
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(3, 2, 17, 1, 5)), ru.mixed(seqs, live=2, seed=1)):
        check(ru.run_in_process(bu.make_runner(d, dtype, 144, max_requests=2, context=80), steps), ref, dtype, rms_tol=rms_tol)


@pytest.mark.parametrize("taps", [1, 2, 5])
def test_convolution_taps_and_first_tokens(tmp_path, taps):
    """The first tokens of a sequence see zeros in front of it; a portion of one or two tokens is shorter than the
    convolution's history; with one tap there is no history at all."""
    cfg = bu.config(40, 70, [M(2, 8, 8, 1, taps, 1, mlp=bu.dense(48))])
    d = bu.write_model(str(tmp_path), cfg, seed=9)
    c, w = plain.load(d)
    seqs = bu.sequences(70, (9, 2, 1, 30), seed=1)
    ref = [plain.forward(c, w, s) for s in seqs]
    runner = bu.make_runner(d, "float32", 32, max_requests=1)
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(1, 1, 2, 1, 3, 17, 2)), ru.prefill_then_decode(seqs, tail=6)):
        check(ru.run_in_process(runner, steps), ref, "float32", f"taps={taps}")
    if taps > 1:        # and the history matters
        w2 = dict(w)
        w2["l0.mix.conv"] = w["l0.mix.conv"].copy()
        w2["l0.mix.conv"][:, :-1] = 0.0
        assert ru.rel_err(plain.forward(c, w2, seqs[0])[1:], ref[0][1:]) > 20 * TOL["float32"]


MARK = 12.0         # the marks' size: the norm behind the embedding leaves them large beside the random entries


def _marked(length, at, vocab=50, seed=8):
    """Tokens 2.. at random with token 0 at the places ``at`` (token 1 nowhere); and the same with token 1 there."""
    base = [2 + t % (vocab - 2) for t in bu.sequences(vocab, (length,), seed=seed)[0]]
    a, b = list(base), list(base)
    for p in at:
        a[p], b[p] = 0, 1
    return a, b


def _loud_key(tensors):
    """A marked token's key stands out for every query that is not one, next to a sink that would swallow ordinary keys, and
    its value says which of the two marks it is."""
    bu.mark_tokens(tensors, MARK)
    t = lambda k: tensors["l0.mix." + k]
    for n in "qkv":
        t(n).mul_(0.05)
    t("k")[:, bu.MARK_A] = t("k")[:, bu.MARK_B] = 0.5
    t("k")[:, bu.MARK_LATER] = 0.0
    t("q")[:, bu.MARK_LATER] = 0.5
    t("v")[:, bu.MARK_A], t("v")[:, bu.MARK_B] = 0.5, -0.5
    t("sink").fill_(4.0)
    t("o").mul_(4.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(16, 16, 24), (64, 64, 64)], ids=["16x24", "64x64"])
@pytest.mark.parametrize("window,keep,place", [(50, 4, 3), (50, 4, 4), (50, 4, 5), (50, 0, 0), (50, 16, 15), (50, 16, 16), (50, 33, 32), (50, 4, 63), (50, 4, 64),
                                               (63, 2, 65), (64, 2, 65), (65, 1, 100), (16, 5, 127), (130, 3, 128), (130, 70, 69), (130, 70, 70)])
def test_edges_of_the_window_and_of_the_kept_tokens(tmp_path, dtype, sizes, window, keep, place):
    """The marked token is seen up to the last position of its window and, where it is a kept one, for ever: the plain
    implementation says that the two marks differ there and nowhere else, and the engine agrees at every position, for one
    portion, small ones and single tokens, over pages of 16 and of 64."""
    dim, rot, vdim = sizes
    cfg = bu.config(32, 50, [A(2, 1, dim, vdim, window, keep, scale=0.4 * (16 / dim) ** 0.5, softcap=12.0)], residual_mult=1.0)
    d = bu.write_model(str(tmp_path), cfg, seed=33, edit=_loud_key)
    c, w = plain.load(d)
    seq, other = _marked(270, [place])
    ref, ref_other = plain.forward(c, w, seq), plain.forward(c, w, other)
    last = 269 if place < keep else min(269, place + window - 1)
    scale = np.max(np.abs(ref))
    moved = np.max(np.abs(ref - ref_other), axis=1) / scale
    assert np.all(moved[place + 1:last + 1] > 6 * TOL[dtype]) and np.all(moved[last + 1:] < 1e-9) and np.all(moved[:place] < 1e-9)
    for page, steps in ((16, ru.portions([seq], sizes=(130, 2, 3, 1, 1, 90, 2))), (64, ru.prefill_then_decode([seq], tail=100)), (64, ru.whole([seq]))):
        got = ru.run_in_process(bu.make_runner(d, dtype, 320, page_size=page, max_requests=1), steps)
        # bfloat16: every logit here hangs on a handful of rounded numbers, so it is held to a part of what the mark changes
        limit = TOL[dtype] if dtype == "float32" else max(TOL[dtype], float(moved[place + 1:last + 1].min()) / 4)
        assert ru.rel_err(got[0], ref) < limit and rms_err(got[0], ref) < 1.5 * RMS_TOL[dtype], (page,)


def _far_check(d, dtype, places, length=400, rotated=False):
    c, w = plain.load(d)
    seq, other = _marked(length, places)
    ref, ref_other = plain.forward(c, w, seq), plain.forward(c, w, other)
    effect = ru.rel_err(ref_other[-8:], ref[-8:])
    assert effect > 5 * TOL[dtype]                                       # the far token matters
    # float32: rounding of sums.  bfloat16: every logit here hangs on a handful of rounded numbers, so the largest difference is
    # held to a tenth of what the far token changes, and the root mean square to the usual bound.
    limit = TOL[dtype] if dtype == "float32" else max(TOL[dtype], effect / 10)
    runner = bu.make_runner(d, dtype, 416, page_size=32, max_requests=1)
    for s, r in ((other, ref_other), (seq, ref)):                        # the same slot and pages twice
        steps = ru.portions([s], sizes=(130, 2, 67, 1, 1, 100, 64)) if s is seq else ru.prefill_then_decode([s], tail=40)
        got = ru.run_in_process(runner, steps)
        assert ru.rel_err(got[0], r) < limit and rms_err(got[0], r) < RMS_TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("place", [0, 7, 31, 32, 63, 64, 127])
def test_a_far_key_among_hundreds(tmp_path, dtype, place):
    """No window: the marked key, at the start and at pages' and key blocks' edges, decides what the last tokens of 400 read."""
    cfg = bu.config(32, 50, [A(2, 2, 16, 8, scale=0.4, softcap=12.0)], residual_mult=1.0)
    _far_check(bu.write_model(str(tmp_path), cfg, seed=33, edit=_loud_key), dtype, [place])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_write_reaches_through_the_state(tmp_path, dtype):
    """Decays next to 1 and a large step for the marked tokens alone: what they wrote still shows hundreds of tokens later,
    after portions, decoded tokens, and a slot that another request used before."""
    cfg = bu.config(32, 50, [M(2, 16, 16, 1, 3, 1)], residual_mult=1.0)

    def slow(tensors):
        bu.mark_tokens(tensors, MARK)
        t = lambda k: tensors["l0.mix." + k]
        inner, n = 32, 16
        z, x, B, C, dt = (t("in")[a:b] for a, b in ((0, inner), (inner, 2 * inner), (2 * inner, 2 * inner + n), (2 * inner + n, 2 * inner + 2 * n),
                                                    (2 * inner + 2 * n, 2 * inner + 2 * n + 2)))
        t("A_log").fill_(-9.0); t("dt_bias").fill_(-3.0)
        dt.zero_()
        dt[:, bu.MARK_A] = dt[:, bu.MARK_B] = 1.0                             # the marked tokens write, the others hardly
        dt[:, bu.MARK_LATER] = -1.5
        t("conv").zero_(); t("conv")[:, -1] = 1.0; t("conv.b").zero_()
        x[:, bu.MARK_A], x[:, bu.MARK_B] = 0.6, -0.6
        B[:, bu.MARK_A] = B[:, bu.MARK_B] = 0.6
        C[:, bu.MARK_LATER] = 0.6
        t("D").fill_(0.1)
    _far_check(bu.write_model(str(tmp_path), cfg, seed=35, edit=slow), dtype, [0, 1, 2])


def test_strong_decays_forget_within_a_run(tmp_path):
    """Decays so strong that a product over a few tokens underflows: the forms that take runs of tokens must not divide by it."""
    cfg = bu.config(32, 50, [M(2, 16, 16, 1, 2, 1)])

    def strong(tensors):
        tensors["l0.mix.A_log"].fill_(4.5)
        tensors["l0.mix.dt_bias"].uniform_(-1.0, 3.0)
    d = bu.write_model(str(tmp_path), cfg, seed=41, edit=strong)
    c, w = plain.load(d)
    seqs = bu.sequences(50, (200, 18), seed=4)
    ref = [plain.forward(c, w, s) for s in seqs]
    for dtype in ("float32", "bfloat16"):
        for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(66, 1, 17, 2, 30)), ru.prefill_then_decode(seqs, tail=9)):
            check(ru.run_in_process(bu.make_runner(d, dtype, 208, max_requests=1), steps), ref, dtype)


def test_mixed_values_are_cached_mixed(tmp_path):
    """A share of one: every later mixing layer attends over the first layer's values alone, also those of tokens that earlier
    steps brought, whatever slots and pages the requests use."""
    layers = [A(2, 1, 16, 24, 30, 2, softcap=6.0, v_mix=True), M(2, 8, 8, 1, 2, 1), A(4, 1, 8, 24, v_mix=True), A(2, 1, 8, 24, 9, 3, v_mix=True)]
    cfg = bu.config(32, 40, layers, residual_mult=1.0)
    d = bu.write_model(str(tmp_path), cfg, seed=19, edit=lambda t: [t[f"l{i}.mix.vmix"].fill_(1.0) for i in (2, 3)])
    c, w = plain.load(d)
    seqs = bu.sequences(40, (60, 21, 9, 34), seed=2)
    ref = [plain.forward(c, w, s) for s in seqs]
    assert ru.rel_err(plain.forward(c, {**w, "l2.mix.v": 0 * w["l2.mix.v"], "l3.mix.v": 0 * w["l3.mix.v"]}, seqs[0]), ref[0]) < 1e-12
    for dtype in ("float32", "bfloat16"):
        for steps in (ru.portions(seqs, sizes=(1, 1, 2, 7, 1, 3)), ru.mixed(seqs, live=2, seed=5), ru.prefill_then_decode(seqs, tail=8)):
            check(ru.run_in_process(bu.make_runner(d, dtype, 112, max_requests=2, context=64), steps), ref, dtype)


def test_the_sink_takes_its_share(tmp_path):
    """Sinks far above the scores shrink every head's output, sinks far below change nothing: the plain implementation says so,
    and the kernels agree for prompts, portions and decoded tokens."""
    cfg = bu.config(32, 50, [A(4, 2, 16, 16, 100, 8, softcap=3.0)])
    seq = bu.sequences(50, (230,), seed=3)
    refs = {}
    for level in (-30.0, 0.0, 5.0):
        d = bu.write_model(str(tmp_path / f"s{level}"), cfg, seed=5, edit=lambda t: t["l0.mix.sink"].copy_(level + 0.1 * t["l0.mix.sink"]))
        c, w = plain.load(d)
        refs[level] = plain.forward(c, w, seq[0])
        for dtype in ("float32", "bfloat16"):
            runner = bu.make_runner(d, dtype, 256, page_size=32, max_requests=1)
            for steps in (ru.whole(seq), ru.prefill_then_decode(seq, tail=25), ru.portions(seq, sizes=(100, 2, 31, 1, 1, 80))):
                check(ru.run_in_process(runner, steps), [refs[level]], dtype, f"sink {level}")
    assert ru.rel_err(refs[5.0], refs[-30.0]) > 0.02 and ru.rel_err(refs[0.0][:8], refs[-30.0][:8]) > 0.01


def test_variants_of_the_plain_implementation_show_in_the_logits(tmp_path, monkeypatch):
    """What a wrong reading would compute gives other logits, so the comparison would see it."""
    layers = [A(4, 2, 16, 16, 12, 3, rot=8, base=50.0, softcap=1.0, v_mix=True, mlp=bu.dense(24)), M(4, 8, 8, 2, 3, 2, mlp=bu.moe(4, 2, 16, 0.5, 24, 0.6)),
              A(2, 2, 16, 16, 20, 5, rot=16, softcap=1.0, v_mix=True, mlp=bu.moe(5, 3, 16, 0.4))]
    cfg = bu.config(48, 40, layers, residual_mult=0.5)
    d = bu.write_model(str(tmp_path), cfg, seed=5)
    c, w = plain.load(d)
    seq = bu.sequences(40, (60,), seed=3)[0]
    ref = plain.forward(c, w, seq)
    differs = lambda got: ru.rel_err(got, ref) > 1e-3

    def mixer(i, **change):
        out = dict(c, layers=list(c["layers"]))
        out["layers"][i] = dict(out["layers"][i], mixer={**out["layers"][i]["mixer"], **change})
        return out
    for i, change in ((0, {"mask": {"size": 12, "keep_first": 2}}), (0, {"mask": {"size": 13, "keep_first": 3}}), (0, {"mask": {"size": 12, "keep_first": 0}}),
                      (2, {"softcap": None}), (2, {"softcap": 2.0}), (2, {"v_mix": False}), (0, {"rot": None}), (0, {"rot": {"dims": 8, "base": 55.0}}),
                      (1, {"norm_groups": 1}), (1, {"norm_groups": 4})):
        assert differs(plain.forward(mixer(i, **change), w, seq)), (i, change)
    assert differs(plain.forward(dict(c, residual_mult=1.0), w, seq)) and differs(plain.forward(dict(c, logit_scale=1.0), w, seq))
    for name, value in (("l0.mix.sink", -100.0), ("l2.mix.sink", -100.0), ("l1.mix.D", 0.0), ("l1.mlp.router.b", 0.0), ("l1.mix.conv.b", 0.0),
                        ("l1.mlp.shared.sg", 0.0), ("embed.norm", 1.0), ("l1.mix.dt_bias", 0.0)):
        assert differs(plain.forward(c, {**w, name: np.full_like(w[name], value)}, seq)), name
    limits = dict(c, layers=[dict(l, mlp=None if not l["mlp"] else dict(l["mlp"], expert={"ff": 16, "limit": 50.0}) if l["mlp"]["kind"] == "moe" else l["mlp"])
                             for l in c["layers"]])
    assert differs(plain.forward(limits, w, seq))
    monkeypatch.setattr(plain, "norm_in_parts", lambda x, v, eps, parts: plain.unit_rms(x, eps) * v)
    assert differs(plain.forward(c, w, seq))
    monkeypatch.undo()
    got = ru.run_in_process(bu.make_runner(d, "float32", 64, max_requests=1), ru.whole([seq]))
    assert ru.rel_err(got[0], ref) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_graphs(models, dtype):
    """300 tokens one by one behind a short prompt, replayed from CUDA graphs, two requests side by side: windows pass over
    decoded tokens and their pages go back while the kept ones stay."""
    d, cfg, _, _ = models["A"]
    c, w = plain.load(d)
    seqs = bu.sequences(cfg["vocab"], (330, 317), seed=4)
    ref = [plain.forward(c, w, s) for s in seqs]
    runner = bu.make_runner(d, dtype, 704, page_size=16, max_requests=2, graphs=True, context=352)
    assert runner.model.graph_safe
    got = ru.run_in_process(runner, ru.batched_decode(seqs, tails=[300, 300]))
    assert runner.graph_replays > 250
    check(got, ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_replayed_from_graphs(models, dtype):
    """Equal portions beside decoding requests, whose shapes repeat and are captured."""
    d, cfg, _, _ = models["B"]
    c, w = plain.load(d)
    seqs = bu.sequences(cfg["vocab"], (96, 16, 96), seed=6)
    ref = [plain.forward(c, w, s) for s in seqs]
    runner = bu.make_runner(d, dtype, 256, page_size=16, max_requests=3, graphs=True, context=112)
    steps = []
    for i in range(8):
        steps.append({"entries": [(0, seqs[0][12 * i:12 * i + 12], list(range(12))), (1, seqs[1][2 * i:2 * i + 1], [0]),
                                  (2, seqs[2][12 * i:12 * i + 12], list(range(12)))], "end": []})
        steps.append({"entries": [(1, seqs[1][2 * i + 1:2 * i + 2], [0])], "end": []})
    got = ru.run_in_process(runner, steps)
    assert runner.graph_replays > 8
    check(got, ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_binary(models, tmp_path, dtype):
    d, cfg, seqs, ref = models["A"]
    steps = ru.mixed(seqs, live=4, seed=5)
    got = ru.run_trace_binary(d, dtype, steps, str(tmp_path), max_tokens=5 * 64, vocab=cfg["vocab"])
    check(got, ref, dtype)


def test_unused_tensors_are_skipped(tmp_path):
    """A file may carry norm2 of a layer without feed-forward and the share of a layer that does not mix values; the first
    mixing layer's share may be missing."""
    import torch
    cfg = bu.config(32, 40, [A(2, 1, 8, 8), A(2, 1, 8, 8, v_mix=True), A(2, 1, 8, 8, v_mix=True)])

    def change(tensors):
        tensors.update({"l0.norm2": torch.ones(32), "l0.mix.vmix": torch.tensor(0.5)})
        tensors.pop("l1.mix.vmix", None)
    d = bu.write_model(str(tmp_path), cfg, seed=3, edit=change)
    c, w = plain.load(d)
    seqs = bu.sequences(40, (12,), seed=1)
    with pytest.warns(UserWarning, match="not used"):
        runner = bu.make_runner(d, "float32", 32, max_requests=1)
    check(ru.run_in_process(runner, ru.whole(seqs)), [plain.forward(c, w, seqs[0])], "float32")


@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_engine(models, name):
    """Engine.generate (scheduler, sampler, pipelined decode) gives the plain implementation's greedy tokens."""
    from hfee_b200 import Engine, SamplingOptions
    d, cfg, seqs, _ = models[name]
    c, w = plain.load(d)
    prompts = [seqs[0], seqs[1], seqs[7], seqs[2], seqs[6]]
    want = [plain.greedy(c, w, p, 12) for p in prompts]
    eng = Engine(d, dtype="float32", page_size=16, max_context=128, max_requests=3, max_batch_tokens=48, prefill_chunk=11)
    got = [r.token_ids for r in eng.generate(prompts, SamplingOptions.greedy(num_predict=12))]
    assert got == want


def test_command_line_generates(models):
    """``bin/hfee-b200 run`` on a Bumisun folder: greedy tokens of the plain implementation, and a seeded draw through
    the sampling chain that repeats."""
    import os, subprocess, sys
    d, cfg, seqs, _ = models["B"]
    c, w = plain.load(d)
    toks = plain.greedy(c, w, [5, 6, 7], 6)
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "hfee-b200")
    base = [sys.executable, exe, "run", d, "--prompt-ids", "5,6,7", "--num-predict", "6", "--dtype", "float32", "--num-ctx", "256"]
    p = subprocess.run(base + ["--temperature", "0", "--repeat-penalty", "1"], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert p.stdout.split("\n")[0].split() == [str(t) for t in toks]
    draws = [subprocess.run(base + ["--temperature", "0.9", "--top-k", "20", "--seed", "7"], capture_output=True, text=True,
                            timeout=300).stdout.split("\n")[0] for _ in range(2)]
    assert draws[0] == draws[1] and len(draws[0].split()) == 6
