"""The Fokalorn decoder on the GPU against the plain implementation of tests/plain_fokalorn.py: each mechanism alone, whole
prompts, prefill then token by token, portions down to two tokens, mixed batches over few pages and slots, page and tile
edges, far keys and far writes, the first tokens, loops, long decoding, other sizes, and greedy generation through the
engine's entry point."""
import numpy as np
import pytest

import fokalorn_util as fu
import plain_fokalorn as plain
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
    for name, cfg, seed in (("A", fu.FOK_A, 3), ("B", fu.FOK_B, 4)):
        d = fu.write_model(str(tmp_path_factory.mktemp("fokalorn" + name)), cfg, seed)
        c, w = plain.load(d)
        seqs = fu.sequences(cfg["vocab"], LENGTHS, seed=11)
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
        runner = fu.make_runner(d, dtype, max_tokens=17 * 16, context=112)
    else:
        steps = {"whole": ru.whole, "prefill_then_decode": lambda s: ru.prefill_then_decode(s, tail=20),
                 "portions": ru.portions}[scheme](seqs)
        runner = fu.make_runner(d, dtype, max_tokens=112, max_requests=1)
    check(ru.run_in_process(runner, steps), ref, dtype, scheme)


def test_batch_of_unequal_requests_equals_each_alone(models):
    """float32: a row's sums run in one order whatever else is in the batch."""
    d, cfg, seqs, ref = models["A"]
    alone = ru.run_in_process(fu.make_runner(d, "float32", 112, max_requests=1), ru.whole(seqs))
    runner = fu.make_runner(d, "float32", max_tokens=512, max_requests=8, context=112)
    steps = [{"entries": [(i, s, list(range(len(s)))) for i, s in enumerate(seqs)], "end": list(range(len(seqs)))}]
    together = ru.run_in_process(runner, steps)
    for i in range(len(seqs)):
        assert ru.rel_err(together[i], alone[i]) < 2e-6


# name: (layer, streams, groups)
ALONE = {
    "delta": (fu.delta(2, 2, 16, 24, 4), 2, 2),
    "delta_grouped_odd_sizes": (fu.delta(6, 2, 20, 12, 2, ranks=(1, 2)), 4, 3),
    "delta_wide_keys": (fu.delta(1, 1, 144, 40, 3), 3, 1),
    "delta_narrow_keys_wide_values": (fu.delta(2, 1, 4, 72, 1), 1, 4),
    "latent": (fu.latent(4, 16, 8, 16, 24, 0.5, base=100.0), 3, 2),
    "latent_one_head": (fu.latent(1, 8, 24, 40, 8, 0.3), 2, 6),
    "latent_tensor_core_sizes": (fu.latent(5, 24, 16, 40, 32, 0.4, base=300.0), 4, 1),
    "latent_many_heads": (fu.latent(34, 8, 16, 8, 80, 0.3, base=50.0), 1, 1),
    "latent_and_feed_forward": (fu.latent(2, 8, 2, 8, 16, 0.3, ff=40), 6, 12),
    "delta_and_feed_forward": (fu.delta(1, 1, 8, 8, 3, ff=36), 9, 2),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(ALONE.values()), ids=list(ALONE))
def test_each_mixer_alone(tmp_path, case, dtype):
    """One layer: whole, and in portions through the cache or state, under several numbers of streams and groups."""
    layer, streams, groups = case
    cfg = fu.config(48, 90, [layer], streams=streams, groups=groups)
    d = fu.write_model(str(tmp_path), cfg, seed=7)
    c, w = plain.load(d)
    seqs = fu.sequences(90, (37, 3, 64), seed=5)
    ref = [plain.forward(c, w, s) for s in seqs]
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(2, 9, 1, 1, 30, 2))):
        check(ru.run_in_process(fu.make_runner(d, dtype, 64, max_requests=1), steps), ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sizes_that_fit_no_vector_access(tmp_path, dtype):
    """Width, vocabulary, ranks and head sizes that are multiples of neither 8 nor 4: every kernel takes its scalar path."""
    layers = [fu.delta(3, 1, 10, 14, 3, ff=36, ranks=(5, 3)), fu.latent(3, 10, 6, 14, 22, 0.4, base=77.0, ff=30),
              fu.delta(2, 2, 6, 7, 2)]
    cfg = fu.config(50, 77, layers, streams=3, groups=5, loop=(0, 2, 2), eps=3e-6, scale=0.7)
    d = fu.write_model(str(tmp_path), cfg, seed=13)
    c, w = plain.load(d)
    seqs = fu.sequences(77, (41, 2, 19), seed=6)
    ref = [plain.forward(c, w, s) for s in seqs]
    rms_tol = 2.5e-2 if dtype == "bfloat16" else None       # short sums average less of the rounding than wider models' do
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(3, 2, 17, 1, 5)), ru.mixed(seqs, live=2, seed=1)):
        check(ru.run_in_process(fu.make_runner(d, dtype, 96, max_requests=2, context=48), steps), ref, dtype, rms_tol=rms_tol)


@pytest.mark.parametrize("loop", [None, (0, 1, 2), (1, 2, 4), (0, 3, 2), (2, 3, 1), (1, 1, 3)])
def test_loops(tmp_path, loop):
    """A stretch of layers run several times over: at the start, in the middle, the whole model, once, and an empty one.
    Every pass has states, pages and a row of the token before of its own (shared ones would show at once)."""
    layers = [fu.delta(2, 1, 8, 8, 3, ff=24), fu.latent(2, 8, 4, 8, 16, 0.4, ff=20), fu.delta(1, 1, 8, 16, 2)]
    cfg = fu.config(32, 60, layers, streams=2, groups=2, loop=loop)
    d = fu.write_model(str(tmp_path), cfg, seed=17)
    c, w = plain.load(d)
    seqs = fu.sequences(60, (23, 6), seed=9)
    ref = [plain.forward(c, w, s) for s in seqs]
    if loop is not None and loop[2] > 1 and loop[1] > loop[0]:
        assert ru.rel_err(plain.forward({**c, "loop": None}, w, seqs[0]), ref[0]) > 1e-2
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(2, 5, 1, 9, 2)), ru.mixed(seqs, live=2, seed=3)):
        check(ru.run_in_process(fu.make_runner(d, "float32", 64, max_requests=2, context=32), steps), ref, "float32", str(loop))


@pytest.mark.parametrize("taps", [1, 2, 5])
def test_convolution_taps_and_first_tokens(tmp_path, taps):
    """The first tokens of a sequence see zeros in front of it, in the convolution and in the token shift; a portion of one
    or two tokens is shorter than the convolution's history; with one tap there is no history at all."""
    cfg = fu.config(40, 70, [fu.delta(2, 1, 8, 8, taps, ff=48)], streams=2, groups=1)
    d = fu.write_model(str(tmp_path), cfg, seed=9)
    c, w = plain.load(d)
    seqs = fu.sequences(70, (9, 2, 1, 30), seed=1)
    ref = [plain.forward(c, w, s) for s in seqs]
    runner = fu.make_runner(d, "float32", 32, max_requests=1)
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(1, 1, 2, 1, 3, 17, 2)), ru.prefill_then_decode(seqs, tail=6)):
        check(ru.run_in_process(runner, steps), ref, "float32", f"taps={taps}")


def test_the_row_before_a_portion_belongs_to_the_request(tmp_path):
    """A shift of one: the mixer reads the row of the token before and nothing else, so a lost or stale row (a slot's
    earlier user, the batch's neighbour, another pass) would change every logit."""
    cfg = fu.config(32, 40, [fu.latent(2, 8, 4, 8, 16, 0.4), fu.delta(1, 1, 8, 8, 1)], streams=2, groups=1, loop=(0, 2, 2))
    d = fu.write_model(str(tmp_path), cfg, seed=19, edit=lambda t: (t["l0.shift"].fill_(1.0), t["l1.shift"].fill_(1.0)))
    c, w = plain.load(d)
    seqs = fu.sequences(40, (30, 21, 9, 14), seed=2)
    ref = [plain.forward(c, w, s) for s in seqs]
    still = plain.forward(c, {**w, "l0.shift": 0 * w["l0.shift"], "l1.shift": 0 * w["l1.shift"]}, seqs[0])
    assert ru.rel_err(still, ref[0]) > 0.05
    for steps in (ru.portions(seqs, sizes=(1, 1, 2, 7, 1, 3)), ru.mixed(seqs, live=2, seed=5), ru.prefill_then_decode(seqs, tail=8)):
        check(ru.run_in_process(fu.make_runner(d, "float32", 64, max_requests=2, context=32), steps), ref, "float32")


def test_portions_longer_than_a_run_of_rows(tmp_path):
    """A step of more tokens than one wave of blocks takes one by one: a block then keeps several tokens, and the request
    that begins in one block ends in another."""
    cfg = fu.config(16, 30, [fu.delta(1, 1, 4, 4, 2), fu.delta(1, 1, 4, 4, 2)], streams=2, groups=2)
    d = fu.write_model(str(tmp_path), cfg, seed=23)
    c, w = plain.load(d)
    seqs = fu.sequences(30, (1500, 611, 3), seed=8)
    ref = [plain.forward(c, w, s) for s in seqs]
    runner = fu.make_runner(d, "float32", 2304, max_requests=3, context=1536)
    steps = [{"entries": [(i, s[:-2], list(range(len(s) - 2))) for i, s in enumerate(seqs)], "end": []}]
    steps += [{"entries": [(i, s[-2 + k:][:1], [0]) for i, s in enumerate(seqs)], "end": []} for k in range(2)]
    check(ru.run_in_process(runner, steps), ref, "float32")


MARK = 6.0          # the marks' size: the norm in front leaves them large


def _marked_sequence(length, at, vocab=50, seed=8):
    """Tokens 2.. at random with token 0 at the places ``at`` (token 1 nowhere); and the same with token 1 there."""
    base = [2 + t % (vocab - 2) for t in fu.sequences(vocab, (length,), seed=seed)[0]]
    a, b = list(base), list(base)
    for p in at:
        a[p], b[p] = 0, 1
    return a, b


def _far_check(d, dtype, places, length=400):
    c, w = plain.load(d)
    seq, other = _marked_sequence(length, places)
    ref, ref_other = plain.forward(c, w, seq), plain.forward(c, w, other)
    effect = ru.rel_err(ref_other[-8:], ref[-8:])
    assert effect > 5 * TOL[dtype]                                       # the far token matters
    # float32: rounding of sums.  bfloat16: every logit here hangs on a handful of rounded numbers (one layer, weights
    # made so that one key or a few writes decide), so the largest difference is held to a tenth of what the far
    # token changes, and the root mean square to the usual bound.
    limit = TOL[dtype] if dtype == "float32" else max(TOL[dtype], effect / 10)
    runner = fu.make_runner(d, dtype, 416, page_size=32, max_requests=1)
    for s, r in ((other, ref_other), (seq, ref)):                        # the same slot and pages twice
        steps = ru.portions([s], sizes=(130, 2, 67, 1, 1, 100, 64)) if s is seq else ru.prefill_then_decode([s], tail=40)
        got = ru.run_in_process(runner, steps)
        assert ru.rel_err(got[0], r) < limit and rms_err(got[0], r) < RMS_TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("place", [0, 7, 31, 32, 63, 64, 127])
def test_a_far_key_among_hundreds(tmp_path, dtype, place):
    """The marked key, at the start, at pages' and key blocks' edges, decides what the last tokens of 400 read, next to a
    sink that would swallow the weight of ordinary keys."""
    cfg = fu.config(32, 50, [fu.latent(2, 8, 8, 8, 16, 1.0, base=1.0e4)], streams=2, groups=1)

    def marked(tensors):
        fu.mark_first_tokens(tensors, MARK)
        t = lambda k: tensors["l0.mix." + k]
        tensors["l0.shift"].zero_()
        t("dkv").mul_(0.2)
        t("dkv")[:8, fu.MARK_A], t("dkv")[:8, fu.MARK_B] = 1.0, 1.0           # latent dimensions 0..7: a marked token
        t("dkv")[:8, fu.MARK_LATER] = 0.0
        t("dkv")[8:16, fu.MARK_LATER] = 0.6                                   # 8..15: any other token
        t("dkv")[8:12, fu.MARK_A], t("dkv")[8:12, fu.MARK_B] = 1.0, -1.0      # and which of the two marks
        t("q").mul_(0.2)
        t("uk").mul_(0.1)
        for h in range(2):
            t("uk")[8 * h:8 * h + 8, :8] = 0.5
            t("q")[16 * h:16 * h + 8, fu.MARK_LATER] = 0.5
        t("uv").mul_(0.3)
        t("uv")[:, 8:12] += 0.5
        t("sink").fill_(4.0)
        t("o").mul_(3.0)
    _far_check(fu.write_model(str(tmp_path), cfg, seed=33, edit=marked), dtype, places=[place])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_sink_takes_its_share(tmp_path, dtype):
    """Sinks far above the scores shrink every head's output, sinks far below change nothing: the plain implementation
    says so, and the kernels agree for prompts, portions and decoded tokens (whose keys are split among thread blocks)."""
    cfg = fu.config(32, 50, [fu.latent(4, 16, 16, 16, 32, 0.3)], streams=2, groups=2)
    seqs = fu.sequences(50, (330,), seed=3)
    refs = {}
    for level in (-30.0, 0.0, 6.0):
        d = fu.write_model(str(tmp_path / f"s{level}"), cfg, seed=5, edit=lambda t: t["l0.mix.sink"].copy_(level + 0.1 * t["l0.mix.sink"]))
        c, w = plain.load(d)
        refs[level] = plain.forward(c, w, seqs[0])
        runner = fu.make_runner(d, dtype, 352, page_size=32, max_requests=1)
        for steps in (ru.whole(seqs), ru.prefill_then_decode(seqs, tail=25), ru.portions(seqs, sizes=(100, 2, 31, 1, 1, 200))):
            check(ru.run_in_process(runner, steps), [refs[level]], dtype, f"sink {level}")
    # a denominator that is larger by e^6 than a few hundred keys' sum
    assert ru.rel_err(refs[6.0], refs[-30.0]) > 0.02 and ru.rel_err(refs[0.0][:8], refs[-30.0][:8]) > 0.01


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_write_reaches_through_the_state(tmp_path, dtype):
    """Decays next to 1 for every channel: what the marked tokens wrote still shows hundreds of tokens later, after
    portions, decoded tokens, and a slot that another request used before."""
    cfg = fu.config(32, 50, [fu.delta(2, 1, 16, 16, 3)], streams=2, groups=1)

    def slow(tensors):
        fu.mark_first_tokens(tensors, MARK)
        t = lambda k: tensors["l0.mix." + k]
        tensors["l0.shift"].zero_()
        t("A_log").fill_(-7.0); t("dt_bias").fill_(-4.0)
        t("b").zero_()
        t("b")[:, fu.MARK_A] = t("b")[:, fu.MARK_B] = 1.0                     # the marked tokens write, the others hardly
        t("b")[:, fu.MARK_LATER] = -2.5
        for n in "qkv":
            t(n + ".conv").zero_()
            t(n + ".conv")[:, -1] = 1.0
        t("k")[:8, fu.MARK_A] = t("k")[:8, fu.MARK_B] = 1.0
        t("k")[8:, fu.MARK_LATER] = 1.0                                       # the others write elsewhere
        t("k")[:8, fu.MARK_LATER] = -1.0
        t("q")[:8, fu.MARK_LATER] = 1.0
        t("v")[:, fu.MARK_A], t("v")[:, fu.MARK_B] = 1.0, -1.0
        t("o").mul_(4.0)
    _far_check(fu.write_model(str(tmp_path), cfg, seed=35, edit=slow), dtype, places=[0, 1, 2])


def test_strong_decays_forget_within_a_tile(tmp_path):
    """Decays so strong that a product over a few tokens underflows: the chunked form must not divide by it."""
    cfg = fu.config(32, 50, [fu.delta(2, 2, 16, 16, 2)], streams=2, groups=1)

    def strong(tensors):
        tensors["l0.mix.A_log"].fill_(4.0)
        tensors["l0.mix.dt_bias"].uniform_(-1.0, 3.0)
    d = fu.write_model(str(tmp_path), cfg, seed=41, edit=strong)
    c, w = plain.load(d)
    seqs = fu.sequences(50, (70, 18), seed=4)
    ref = [plain.forward(c, w, s) for s in seqs]
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(16, 1, 17, 2, 30)), ru.prefill_then_decode(seqs, tail=9)):
        check(ru.run_in_process(fu.make_runner(d, "float32", 80, max_requests=1), steps), ref, "float32")


def test_variants_of_the_plain_implementation_show_in_the_logits(tmp_path, monkeypatch):
    """What a wrong reading would compute gives other logits, so the comparison would see it."""
    layers = [fu.delta(4, 2, 16, 16, 3, ff=24), fu.latent(2, 16, 8, 16, 24, 0.4, 50.0, ff=24)]
    cfg = fu.config(48, 40, layers, streams=3, groups=4, loop=(0, 2, 2))
    d = fu.write_model(str(tmp_path), cfg, seed=5)
    c, w = plain.load(d)
    seq = fu.sequences(40, (40,), seed=3)[0]
    ref = plain.forward(c, w, seq)
    other = {
        "no sink": {"l1.mix.sink": w["l1.mix.sink"] - 100.0},
        "no shift": {"l0.shift": 0 * w["l0.shift"]},
        "mix indexed the other way": {"l1.hc1.mix": w["l1.hc1.mix"].T},
        "streams all read alike": {"l0.hc2.in": np.full(3, w["l0.hc2.in"].mean())},
        "one decay per head": {"l0.mix.dt_bias": np.repeat(w["l0.mix.dt_bias"].reshape(4, 16).mean(1), 16)},
        "no head gate": {"l1.mix.g": w["l1.mix.g"] * 0},
        "no latent norm weight": {"l1.mix.dkv.norm": np.ones(24)},
        "one tap fewer": {"l0.mix.k.conv": w["l0.mix.k.conv"] * np.array([0, 1, 1])},
    }
    for what, change in other.items():
        assert ru.rel_err(plain.forward(c, {**w, **change}, seq), ref) > 1e-3, what
    assert ru.rel_err(plain.forward({**c, "norm": {**c["norm"], "groups": 1}}, w, seq), ref) > 1e-3
    assert ru.rel_err(plain.forward({**c, "embedding": {"scale": 2.0}}, w, seq), ref) > 1e-3
    turned = plain.rotate

    def halves(x, dims, base):
        perm = np.arange(dims).reshape(2, dims // 2).T.reshape(-1)
        out = np.empty_like(x)
        out[..., perm] = turned(x[..., perm], dims, base)
        return out
    monkeypatch.setattr(plain, "rotate", halves)
    assert ru.rel_err(plain.forward(c, w, seq), ref) > 1e-3
    monkeypatch.undo()
    got = ru.run_in_process(fu.make_runner(d, "float32", 48, max_requests=1), ru.whole([seq]))
    assert ru.rel_err(got[0], ref) < TOL["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_graphs(models, dtype):
    """300 tokens one by one behind a short prompt, replayed from CUDA graphs, two requests side by side."""
    d, cfg, _, _ = models["B"]
    c, w = plain.load(d)
    seqs = fu.sequences(cfg["vocab"], (330, 317), seed=4)
    ref = [plain.forward(c, w, s) for s in seqs]
    runner = fu.make_runner(d, dtype, 704, page_size=16, max_requests=2, graphs=True, context=352)
    assert runner.model.graph_safe
    got = ru.run_in_process(runner, ru.batched_decode(seqs, tails=[300, 300]))
    assert runner.graph_replays > 250
    check(got, ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_replayed_from_graphs(models, dtype):
    """Equal portions beside decoding requests, whose shapes repeat and are captured."""
    d, cfg, _, _ = models["A"]
    c, w = plain.load(d)
    seqs = fu.sequences(cfg["vocab"], (96, 16, 96), seed=6)
    ref = [plain.forward(c, w, s) for s in seqs]
    runner = fu.make_runner(d, dtype, 256, page_size=16, max_requests=3, graphs=True, context=112)
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


def test_unused_tensors_of_a_layer_without_feed_forward(tmp_path):
    """A file may carry norm2 and hc2.* of a layer that has no feed-forward: they are skipped with a warning."""
    import torch
    cfg = fu.config(32, 40, [fu.delta(1, 1, 8, 8, 2)], streams=2, groups=1)

    def more(tensors):
        tensors.update({"l0.norm2": torch.ones(32), "l0.hc2.in": torch.ones(2), "l0.hc2.out": torch.ones(2), "l0.hc2.mix": torch.ones(2, 2)})
    d = fu.write_model(str(tmp_path), cfg, seed=3, edit=more)
    c, w = plain.load(d)
    seqs = fu.sequences(40, (12,), seed=1)
    with pytest.warns(UserWarning, match="not used"):
        runner = fu.make_runner(d, "float32", 32, max_requests=1)
    check(ru.run_in_process(runner, ru.whole(seqs)), [plain.forward(c, w, seqs[0])], "float32")


def test_greedy_generation_through_the_engine(models):
    """Engine.generate (scheduler, sampler, pipelined decode) gives the plain implementation's greedy tokens."""
    from hfee_b200 import Engine, SamplingOptions
    d, cfg, seqs, _ = models["A"]
    c, w = plain.load(d)
    prompts = [seqs[0], seqs[1], seqs[7], seqs[2], seqs[6]]
    want = [plain.greedy(c, w, p, 12) for p in prompts]
    eng = Engine(d, dtype="float32", page_size=16, max_context=128, max_requests=3, max_batch_tokens=48, prefill_chunk=11)
    got = [r.token_ids for r in eng.generate(prompts, SamplingOptions.greedy(num_predict=12))]
    assert got == want


def test_command_line_generates(models):
    """``bin/hfee-b200 run`` on a Fokalorn folder: greedy tokens of the plain implementation, and a seeded draw through
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_pages_of_64(models, dtype):
    """Pages that the tcgen05 attention takes: long portions beside short ones and single tokens, in and across key blocks."""
    d, cfg, _, _ = models["B"]
    c, w = plain.load(d)
    seqs = fu.sequences(cfg["vocab"], (300, 130, 65, 64), seed=12)
    ref = [plain.forward(c, w, s) for s in seqs]
    for steps in (ru.whole(seqs), ru.portions(seqs, sizes=(130, 2, 63, 1, 64)), ru.mixed(seqs, live=3, seed=4, chunk_sizes=(2, 40, 64, 90))):
        check(ru.run_in_process(fu.make_runner(d, dtype, 10 * 64, page_size=64, max_requests=3, context=320), steps), ref, dtype)
