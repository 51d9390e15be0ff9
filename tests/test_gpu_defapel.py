"""The Defapel design in the engine against the plain implementation (GPU): every mechanism alone, whole prompts, cuts
down to two tokens, decoding, unequal batches, pages and state slots used again, keys far away, at page borders and just
inside and outside the window, the first token of a sequence in a state hundreds of tokens later, other sizes than any real
model's, and greedy generation through the entry point and the scheduler."""
import os

import numpy as np
import pytest

from defapel_helpers import (CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_D, SCALING, bf16_round, channel, config, delta, draw_weights, make_folder, moe, parallel,
                             rot, scaling, tokens, window)
from plain import defapel_plain as P

pytestmark = pytest.mark.gpu

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D}
TOL = {"float32": 2e-4, "bfloat16": 6e-2}


def f64(w):
    return {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}


class Models:
    """Per configuration and dtype: (folder, config, weights for the plain implementation); the same values stored in 32
    bits for the float32 runs and as bfloat16 for the others."""

    def __init__(self, factory):
        self.items = {}
        for i, (name, cfg) in enumerate(CONFIGS.items()):
            w = draw_weights(cfg, 900 + i)
            self.items[name, "float32"] = (make_folder(factory.mktemp(f"df_{name}_f32"), cfg, w, "F32"), cfg, f64(w))
            self.items[name, "bfloat16"] = (make_folder(factory.mktemp(f"df_{name}_bf16"), cfg, w, "BF16"), cfg, f64(w))

    def __getitem__(self, key):
        return self.items[key if isinstance(key, tuple) else (key, "float32")]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return Models(tmp_path_factory)


def engine_for(folder, dtype, **kw):
    from purhie_b200.engine import Engine
    opts = dict(page_size=8, max_tokens=512, max_requests=4, poison_cache=True)
    opts.update(kw)
    return Engine.from_folder(folder, dtype=dtype, **opts)


def error(got, ref):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape
    assert np.isfinite(got).all()
    return np.abs(got - ref).max() / max(np.abs(ref).max(), 1e-30)


def close(got, ref, tol):
    err = error(got, ref)
    assert err < tol, f"relative error {err:.3e} (allowed {tol:.1e})"


def close_logits(got, ref, dtype):
    """float32: every number.  bfloat16: a router's choice among near-equal scores may turn on a rounding, and such a row is
    far off as a whole; nearly all rows must be close, and none may be wild."""
    if dtype == "float32":
        return close(got, ref, TOL[dtype])
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape and np.isfinite(got).all()
    rows = np.sqrt(((got - ref) ** 2).mean(axis=-1)) / np.sqrt((ref ** 2).mean())
    assert np.mean(rows > TOL[dtype]) <= 0.1 and np.median(rows) < TOL[dtype] / 2, (np.sort(rows)[-8:], np.median(rows))


def moves(other, ref, by):
    assert np.abs(other - ref).max() > by * np.abs(ref).max()


def run_cut(engine, rid, toks, cuts):
    """Feed ``toks`` in portions of the given sizes (the last portion takes what is left); all logits."""
    from purhie_b200.engine import StepEntry
    engine.add_request(rid)
    rows, at = [], 0
    for n in list(cuts) + [len(toks)]:
        n = min(n, len(toks) - at)
        if n <= 0:
            break
        rows.append(engine.step([StepEntry(rid, toks[at:at + n], list(range(n)))]))
        at += n
    engine.release(rid)
    return np.concatenate(rows)


def part_of(cfg, layer, name):
    from purhie_b200.config import ModelConfig
    spec = ModelConfig.from_dict(cfg).model_spec()
    part = spec["layers"][layer]["parts"][name]
    return part["kind"], part["params"]


def probe(kind, params, folder, dtype, pages=80, slots=3):
    from purhie_b200.parts import PartProbe
    p = PartProbe("mixer", kind, params, dtype=dtype)
    p.bind_folder(folder)
    p.mixer_cache(8, pages, slots)
    return p


def mixer_in_pieces(p, x, pieces, request=1):
    p.add_request(request)
    out, at = [], 0
    for n in pieces:
        out.append(p.mixer_step([(request, n)], x[at:at + n]))
        at += n
    assert at == len(x)
    p.release(request)
    return np.concatenate(out)


def inputs(T, width, seed, dtype, scale=1.0):
    x = np.random.default_rng(seed).normal(0, scale, (T, width)).astype(np.float32)
    return bf16_round(x) if dtype == "bfloat16" else x


# ---- whole models ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts_cuts_and_decoding_agree_with_the_plain_implementation(models, name, dtype):
    folder, cfg, w = models[name, dtype]
    eng = engine_for(folder, dtype)
    toks = tokens(75, cfg["vocab"], 7)
    ref = P.forward(cfg, w, toks)
    whole = run_cut(eng, "whole", toks, [])
    close_logits(whole, ref, dtype)
    # one token (the first of a sequence alone), then two, then portions of changing size, single tokens between them
    cut = run_cut(eng, "cut", toks, [1, 2, 2, 5, 1, 1, 16, 3, 17, 2, 1])
    close_logits(cut, ref, dtype)
    # a prompt, then token by token: every decode step replays a graph
    tail = run_cut(eng, "tail", toks, [30] + [1] * 45)
    close_logits(tail, ref, dtype)
    if dtype == "float32":                      # the 32-bit kernels add in one order however the tokens arrive
        assert np.abs(cut - whole).max() <= 1e-5 * np.abs(ref).max()
        assert np.abs(tail - whole).max() <= 1e-5 * np.abs(ref).max()
    eng.check_cache()
    eng.close()


def test_every_layer_agrees_with_the_plain_implementation(models):
    """The residual after each layer, so that a fault shows where it starts."""
    from purhie_b200.engine import StepEntry
    for name in sorted(CONFIGS):
        folder, cfg, w = models[name]
        toks = tokens(40, cfg["vocab"], 3)
        ref = []
        P.forward(cfg, w, toks, ref)
        eng = engine_for(folder, "float32")
        got = {}
        eng.set_layer_dump(lambda entry, x: got.__setitem__(entry, np.array(x)))
        eng.add_request("x")
        eng.step([StepEntry("x", toks, [len(toks) - 1])])
        assert sorted(got) == list(range(len(cfg["layers"])))
        for entry, r in enumerate(ref):
            close(got[entry], r, 1e-4)
        eng.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(models, name, dtype):
    from purhie_b200.engine import StepEntry
    folder, cfg, w = models[name, dtype]
    # room for two requests' states and about 100 tokens: five requests must take turns, pages come back poisoned
    eng = engine_for(folder, dtype, max_tokens=104, max_requests=2)
    lengths = [41, 9, 1, 56, 23]
    reqs = {f"r{i}": tokens(n, cfg["vocab"], 20 + i) for i, n in enumerate(lengths)}
    at = {r: 0 for r in reqs}
    got = {r: [] for r in reqs}
    waiting, live, step = list(reqs), [], 0
    portions = [2, 7, 1, 1, 35, 2, 1, 5, 1, 1, 1, 9]
    while waiting or live:
        while waiting and len(live) < 2:
            r = waiting.pop(0)
            eng.add_request(r)
            live.append(r)
        entries = []
        for j, r in enumerate(live):
            n = min(portions[(step + 3 * j) % len(portions)], len(reqs[r]) - at[r])
            entries.append(StepEntry(r, reqs[r][at[r]:at[r] + n], list(range(n))))
        out = eng.step(entries)
        row = 0
        for e in entries:
            n = len(e.tokens)
            got[e.request_id].append(out[row:row + n])
            row += n
            at[e.request_id] += n
        for r in list(live):
            if at[r] == len(reqs[r]):
                eng.release(r)
                live.remove(r)
        step += 1
        eng.check_cache()
    close_logits(np.concatenate([np.concatenate(got[r]) for r in reqs]), np.concatenate([P.forward(cfg, w, reqs[r]) for r in reqs]), dtype)
    eng.close()


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "bfloat16"), ("C", "float32"), ("D", "bfloat16")])
def test_a_long_prompt_alone_and_beside_a_decode_row_and_a_two_token_portion(models, name, dtype):
    """330 tokens: several chunks of the recurrence, windows passed over many times."""
    from purhie_b200.engine import StepEntry
    folder, cfg, w = models[name, dtype]
    eng = engine_for(folder, dtype, max_tokens=1024)
    toks = tokens(330, cfg["vocab"], 11)
    ref = P.forward(cfg, w, toks)
    close_logits(run_cut(eng, "whole", toks, []), ref, dtype)
    close_logits(run_cut(eng, "cut", toks, [2, 63, 64, 65, 1, 2, 100]), ref, dtype)
    eng.add_request("a"); eng.add_request("b"); eng.add_request("c")
    eng.step([StepEntry("b", toks[:5], []), StepEntry("c", toks[:9], [])])
    out = eng.step([StepEntry("b", toks[5:6], [0]), StepEntry("a", toks[:300], list(range(300))), StepEntry("c", toks[9:11], [0, 1])])
    close_logits(out, np.concatenate([ref[5:6], ref[:300], ref[9:11]]), dtype)
    eng.close()


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "bfloat16")])
def test_long_decoding_keeps_its_state(models, name, dtype):
    folder, cfg, w = models[name, dtype]
    eng = engine_for(folder, dtype, max_tokens=256)
    toks = tokens(230, cfg["vocab"], 3)
    close_logits(run_cut(eng, "long", toks, [2] + [1] * 228), P.forward(cfg, w, toks), dtype)
    eng.close()


# ---- every mechanism alone -------------------------------------------------------------------------------------------
PIECES = [1, 2, 61, 2, 1, 1, 64, 37, 2, 30] + [1] * 59                        # 260 rows


def whole_cut_decoded_and_batched(p, x, ref, tol):
    close(mixer_in_pieces(p, x, [len(x)], 1), ref, tol)
    # portions down to two tokens and one, cut inside pages, chunks and key blocks; then single tokens to the end
    close(mixer_in_pieces(p, x, PIECES, 2), ref, tol)
    # two requests side by side, one decoding while the other brings a portion; pages and slots of the first two again
    p.add_request(3); p.add_request(4)
    a = p.mixer_step([(3, 150)], x[:150])
    both = p.mixer_step([(3, 1), (4, 90)], np.concatenate([x[150:151], x[:90]]))
    again = p.mixer_step([(4, 2), (3, 1)], np.concatenate([x[90:92], x[151:152]]))
    close(np.concatenate([a, both[:1], again[2:]]), ref[:152], tol)
    close(np.concatenate([both[1:], again[:2]]), ref[:92], tol)
    # a long portion late in a request beside a decode row, a short portion, and another long one
    p.release(3); p.release(4)
    for r in (5, 6, 7):
        p.add_request(r)
    first = p.mixer_step([(5, 40), (6, 33)], np.concatenate([x[:40], x[:33]]))
    mixed = p.mixer_step([(6, 1), (5, 140), (7, 129)], np.concatenate([x[33:34], x[40:180], x[:129]]))
    last = p.mixer_step([(7, 3), (5, 2), (6, 1)], np.concatenate([x[129:132], x[180:182], x[34:35]]))
    close(np.concatenate([first[:40], mixed[1:141], last[3:5]]), ref[:182], tol)
    close(np.concatenate([first[40:], mixed[:1], last[5:]]), ref[:35], tol)
    close(np.concatenate([mixed[141:], last[:3]]), ref[:132], tol)
    for r in (5, 6, 7):
        p.release(r)


# one head alone, groups of 1 to 4, keys wider and narrower than values, one to six taps, widths without a vector access; in
# bfloat16 those with dim a multiple of 16 up to 128 run long portions in chunks on the tensor cores
CHANNELS = {
    "d16": (channel(3, 3, 16, 24, 3, 5, 9), 48), "d10": (channel(4, 1, 10, 7, 6, 3, 3), 40), "d32": (channel(4, 2, 32, 16, 2, 16, 8), 64),
    "d64": (channel(2, 2, 64, 40, 4, 8, 24), 56), "d128": (channel(2, 1, 128, 96, 4, 24, 16), 72), "d80": (channel(1, 1, 80, 30, 1, 6, 2), 32),
    "d144": (channel(2, 2, 144, 12, 4, 8, 8), 40), "d30": (channel(6, 3, 30, 50, 5, 7, 5), 42), "v200": (channel(2, 2, 48, 200, 3, 8, 8), 32),
}
HEADS = {
    "d16": (delta(4, 2, 16, 32, 4), 40), "d12": (delta(3, 1, 12, 20, 3), 36), "d64": (delta(2, 1, 64, 64, 4), 64), "d128": (delta(4, 4, 128, 32, 2), 48),
    "d9": (delta(5, 5, 9, 11, 6), 33), "d48": (delta(6, 2, 48, 16, 1), 56), "d160": (delta(2, 1, 160, 24, 3), 24), "d256": (delta(1, 1, 256, 8, 4), 40),
}


def delta_case(tmp_path, per_channel, which, dtype, change=None):
    """(probe of the delta rule alone, the plain function of its input, weights as float64, tensor prefix, width)"""
    if per_channel:
        kind_m, width = CHANNELS[which]
        cfg, prefix, m, f = config(width, 20, [(kind_m, None)]), "l0.mix.", kind_m[1], P.channel_delta
    else:
        m, width = HEADS[which]
        cfg, prefix, f = config(width, 20, [(parallel(window(1, 1, 8, 8, 4, rot(0)), m, 1.0, 1.0), None)]), "l0.mix.right.", P.head_delta
    w = draw_weights(cfg, 3, std=0.4)
    if change:
        change(w, prefix)
    folder = make_folder(tmp_path, cfg, w, "F32" if dtype == "float32" else "BF16")
    kind, params = part_of(cfg, 0, "mixer")
    if not per_channel:
        kind, params = params["right"]["kind"], params["right"]["params"]
    run = lambda x, weights: f(np.asarray(x, dtype=np.float64), weights, prefix, m, cfg["norm"]["eps"])
    return probe(kind, params, folder, dtype), run, f64(w), prefix, width, m


DELTA_TOL = {"float32": 2e-4, "bfloat16": 4e-2}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("per_channel,which", [(True, k) for k in sorted(CHANNELS)] + [(False, k) for k in sorted(HEADS)])
def test_the_delta_rule_alone(tmp_path, per_channel, which, dtype):
    p, run, w, pre, width, m = delta_case(tmp_path, per_channel, which, dtype)
    x = inputs(260, width, 1, dtype)
    ref = run(x, w)
    tol = DELTA_TOL[dtype]
    # each of these left out, or taken another way, shows
    changed = lambda **kw: dict(w, **{pre + k.replace("_conv", ".conv"): v for k, v in kw.items()})
    for n in ("A_log", "dt_bias", "b"):
        moves(run(x, changed(**{n: 0 * w[pre + n]})), ref, 6e-4)
    if m["conv"] > 1:
        moves(run(x, changed(k_conv=w[pre + "k.conv"][:, ::-1])), ref, 2 * tol)
        moves(run(x, changed(v_conv=w[pre + "v.conv"][:, ::-1])), ref, 2 * tol)
    moves(run(x, changed(norm=1 + 0 * w[pre + "norm"])), ref, 2 * tol)
    g = "g2" if per_channel else "g"
    moves(run(x, changed(**{g: 0 * w[pre + g]})), ref, 2 * tol)
    whole_cut_decoded_and_batched(p, x, ref, tol)


@pytest.mark.parametrize("per_channel", [True, False])
def test_chunks_and_single_steps_of_the_delta_rule_agree_wherever_a_prompt_is_cut(tmp_path, per_channel):
    """bfloat16: the same rows in one portion (chunks), in portions either side of a chunk's edge, in portions short enough to
    go token by token, and one by one."""
    p, run, w, _, width, _ = delta_case(tmp_path, per_channel, "d64", "bfloat16")
    x = inputs(200, width, 4, "bfloat16")
    ref = run(x, w)
    one_by_one = mixer_in_pieces(p, x, [1] * 200, 1)
    close(one_by_one, ref, 4e-2)
    for pieces in ([200], [64, 64, 72], [63, 65, 72], [32, 31, 33, 104], [31] * 6 + [14], [1, 128, 1, 70], [2, 33, 2, 2, 161]):
        got = mixer_in_pieces(p, x, pieces, 1)
        close(got, ref, 4e-2)
        close(got, one_by_one, 1e-2)                                           # what differs is the rounding of the output product alone


@pytest.mark.parametrize("rate", [3.0, 8.0])
def test_chunks_with_decays_that_would_overflow_an_inverse(tmp_path, rate):
    """Decays of exp(-20) and less per token: within a chunk's block the inverse of a decay leaves float32, and neighbouring
    channels hardly decay at all."""
    def change(w, pre):
        w[pre + "A_log"] = np.full_like(w[pre + "A_log"], rate / 2)
        w[pre + "dt_bias"] = bf16_round(np.where(np.arange(w[pre + "dt_bias"].size) % 3 == 0, rate, -9.0).astype(np.float32))
    for dtype in ("float32", "bfloat16"):
        p, run, w, _, width, _ = delta_case(tmp_path / dtype, True, "d64", dtype, change)
        x = inputs(150, width, 5, dtype)
        ref = run(x, w)
        for pieces in ([150], [70, 80], [33, 1, 2, 114], [1] * 20 + [130]):
            close(mixer_in_pieces(p, x, pieces, 1), ref, DELTA_TOL[dtype])


@pytest.mark.parametrize("per_channel", [True, False])
def test_the_first_token_still_shows_hundreds_of_tokens_later_in_a_state_that_hardly_forgets(tmp_path, per_channel):
    """The later tokens' steps are tiny and their decays next to none: what the first token wrote stays in S."""
    def change(w, pre):
        w[pre + "A_log"] = np.full_like(w[pre + "A_log"], -7.0)
    for dtype in ("float32", "bfloat16"):
        p, run, w, pre, width, m = delta_case(tmp_path / dtype, per_channel, "d16", dtype, change)
        x = inputs(400, width, 4, dtype, 0.05)
        b = w[pre + "b"].sum(axis=0)
        x[1:] -= (4.0 * b / np.linalg.norm(b) / np.sqrt(width) * 3).astype(np.float32)      # steps near zero
        x = bf16_round(x)
        y = x.copy()
        y[0] = bf16_round((np.random.default_rng(1).normal(0, 2.0, width) + 6.0 * b / np.linalg.norm(b)).astype(np.float32))
        ref_x, ref_y = run(x, w), run(y, w)
        moves(ref_y[-1], ref_x[-1], 0.1)
        tol = DELTA_TOL[dtype]
        close(mixer_in_pieces(p, y, [1, 200] + [1] * 199, 1), ref_y, tol)
        close(mixer_in_pieces(p, y, [400], 2), ref_y, tol)
        close(mixer_in_pieces(p, x, [400], 1), ref_x, tol)                      # the slot again: nothing is left of y


# heads of 128 take the tcgen05 and TMA kernels, 16, 32, 48 and 64 (with other values too) the tile kernel, the rest the plain
# one; windows from one token to longer than the prompt; rotation over all, some and none of a head's dimensions
WINDOWS = {
    "h4": (window(4, 2, 16, 16, 20, rot(16, 1e4, SCALING), 0.9, 2.0), 64), "h6": (window(6, 1, 24, 40, 1, rot(6), 0.5, 3.0), 48),
    "h1": (window(1, 1, 40, 8, 8, rot(0), 0.6, 1.5), 40), "h8": (window(8, 2, 48, 48, 64, rot(48, 500.0, scaling(2.0, 1.0, 1.0, 30)), 0.3, 5.0), 72),
    "h3": (window(3, 3, 64, 32, 100, rot(20, 1e5, scaling(16.0, 1.0, 8.0, 32)), 0.3, 4.0), 24), "h40": (window(40, 8, 8, 8, 33, rot(8), 1.2, 2.0), 56),
    "h24": (window(24, 4, 32, 32, 700, rot(32), 0.5, 6.0), 48), "d128": (window(4, 1, 128, 128, 65, rot(128, 1e6, SCALING), 0.25, 3.0), 48),
    "d128h8": (window(8, 4, 128, 128, 300, rot(64), 0.4, 2.0), 64), "d128w": (window(2, 2, 128, 128, 128, rot(0), 0.1, 60.0), 64),
    "d64": (window(4, 1, 64, 64, 47, rot(64, 50.0), 0.3, 30.0), 64), "d5": (window(2, 1, 5, 9, 12, rot(4), 1.0, 2.0), 22),
}


def window_case(tmp_path, m, width, dtype, std=0.5, seed=4):
    cfg = config(width, 20, [(parallel(m, delta(1, 1, 4, 4, 2), 1.0, 1.0), None)])
    w = draw_weights(cfg, seed, std=std)
    folder = make_folder(tmp_path, cfg, w, "F32" if dtype == "float32" else "BF16")
    left = part_of(cfg, 0, "mixer")[1]["left"]
    run = lambda x, weights, mixer=m: P.window_attention(np.asarray(x, dtype=np.float64), weights, "l0.mix.left.", mixer, cfg["norm"]["eps"])
    return probe(left["kind"], left["params"], folder, dtype), run, f64(w)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(WINDOWS))
def test_window_attention_alone(tmp_path, which, dtype):
    m, width = WINDOWS[which]
    p, run, w = window_case(tmp_path, m, width, dtype)
    x = inputs(260, width, 2, dtype)
    ref = run(x, w)
    tol = 2e-4 if dtype == "float32" else 3e-2
    pre = "l0.mix.left."
    # what is left out or taken another way shows: the cap, the window one token longer, the rotation, its scaling, biases, the
    # norm per head instead of over the row, the gate
    if m["mask"]["size"] > 1:
        if m["softcap"] < 50.0:
            moves(run(x, w, dict(m, softcap=1e6)), ref, 2e-3)
        if m["rot"]["dims"]:
            moves(run(x, w, dict(m, rot=dict(m["rot"], dims=0))), ref, 1e-2)
        if m["rot"]["scaling"]:
            moves(run(x, w, dict(m, rot=dict(m["rot"], scaling=None))), ref, 2e-3)
        moves(run(x, dict(w, **{pre + "k.norm": 1 + 0 * w[pre + "k.norm"]})), ref, 1e-2)
    moves(run(x, dict(w, **{pre + "v.b": 0 * w[pre + "v.b"]})), ref, 2 * tol)
    moves(run(x, dict(w, **{pre + "g": 0 * w[pre + "g"]})), ref, 2 * tol)
    if m["mask"]["size"] < 260:
        moves(run(x, w, dict(m, mask={"size": m["mask"]["size"] + 1})), ref, 6e-4)
    whole_cut_decoded_and_batched(p, x, ref, tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,size", [(16, 40), (24, 17), (64, 64), (128, 90), (128, 128)])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dim, size, dtype):
    """Row `at` has the key that every later query asks for: it takes most of their weight as long as it is in the window, in
    prompts and in decoding, wherever the prompt is cut, and none from the next position on."""
    T, at = 300, 39                                                            # the last slot of a page
    m = window(2, 1, dim, dim, size, rot(0), 24.0 / dim, 40.0)
    p, run, w = window_case(tmp_path, m, 64, dtype, std=0.4, seed=6)
    pre = "l0.mix.left."
    x = np.random.default_rng(3).normal(0, 1.0, (T, 64))
    x[at + 1:] = x[at + 1] + 0.05 * x[at + 1:]                                  # later queries all ask for about the same key
    q = P.rms(x[at + 1] @ w[pre + "q"].T + w[pre + "q.b"], 1e-5, w[pre + "q.norm"])[:dim]
    x[at] = 6.0 * np.linalg.lstsq(w[pre + "k"], q / w[pre + "k.norm"] * np.sqrt(dim) / np.linalg.norm(q) - w[pre + "k.b"] / 6.0, rcond=None)[0]
    x = bf16_round(x.astype(np.float32))
    ref = run(x, w)
    other = x.astype(np.float64).copy()
    other[at] = -other[at]
    without = run(other, w)
    seen = np.abs(ref - without).max(axis=-1) > 0.1 * np.abs(ref).max()
    assert seen[at + size - 1] and not seen[at + size], "the row at the window's edge must show"
    tol = 2e-4 if dtype == "float32" else 4e-2
    edge = at + size
    for pieces in ([T], [at, 1, 7, T - at - 8], [at - 1, 2, T - at - 1], [edge - 1, 2, T - edge - 1], [edge, T - edge], [edge - 2] + [1] * 4 + [T - edge - 2],
                   [T - 60] + [1] * 60):
        close(mixer_in_pieces(p, x, pieces, 1), ref, tol)


def test_the_two_sides_of_a_parallel_layer_are_weighed_and_share_a_cache_entry(models):
    for name, layer, dtype in (("A", 0, "float32"), ("A", 2, "float32"), ("C", 1, "bfloat16"), ("D", 0, "bfloat16")):
        folder, cfg, w = models[name, dtype]
        m, eps = cfg["layers"][layer]["mixer"], cfg["norm"]["eps"]
        x = inputs(260, cfg["width"], layer, dtype)
        at = lambda mixer: P.parallel(x.astype(np.float64), w, f"l{layer}.mix.", mixer, eps)
        ref = at(m)
        moves(at(dict(m, left_scale=m["right_scale"], right_scale=m["left_scale"])), ref, 0.08)
        p = probe(*part_of(cfg, layer, "mixer"), folder, dtype)
        whole_cut_decoded_and_batched(p, x, ref, 2e-4 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 3, 40, 300])
def test_experts_take_their_weight_on_the_input(tmp_path, rows, dtype):
    """Few pairs (streamed weights), many (slices on the tensor cores, or row tiles), one and several experts per token."""
    from purhie_b200.parts import PartProbe
    for width, f in ((64, moe(48, 5, 2)), (40, moe(24, 3, 1)), (42, moe(18, 4, 4))):
        cfg = config(width, 20, [(channel(1, 1, 4, 4, 1, 2, 2), f)])
        w = draw_weights(cfg, 9, std=0.5)
        # inputs near one direction that the routers tell apart clearly: no close calls
        x = inputs(rows, width, 2, dtype, 1.5)
        wd = f64(w)
        s = np.sort(P.sigmoid(x.astype(np.float64) @ wd["l0.mlp.router"].T), axis=-1)
        top = f["router"]["top"]
        gap = s[:, -top] - (s[:, -top - 1] if top < s.shape[1] else 0.0)
        ref = P.experts(x.astype(np.float64), wd, "l0.mlp.", f)
        folder = make_folder(tmp_path / f"{width}", cfg, w, "F32" if dtype == "float32" else "BF16")
        p = PartProbe("feed_forward", *part_of(cfg, 0, "feed_forward"), dtype=dtype)
        p.bind_folder(folder)
        clear = gap > 1e-3
        assert clear.mean() > 0.9
        got = p.feed_forward(x)
        close(got[clear], ref[clear], 2e-4 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("weight_on", ["output", "input"])
@pytest.mark.parametrize("activation", [None, {"kind": "clamped_swish", "alpha": 1.5, "limit": 1.0, "shift": 0.5}, {"kind": "gelu_tanh"}, "relu2"])
def test_experts_with_tiles_of_their_own_give_a_row_what_it_gets_alone(activation, weight_on):
    """bfloat16, hundreds of rows per expert (one launch per product over row tiles that know their expert) against the same
    rows a few at a time (streamed weights); with a shared expert, and with experts that get no row at all."""
    from purhie_b200.parts import PartProbe
    gated = activation != "relu2"
    if not gated and weight_on == "input":
        pytest.skip("experts without a gate take their weight on the output")
    # (the second case: several tiles of features, several blocks of K, more tiles than the device holds at a time)
    for E, width, ff, rows, shared in ((6, 72, 40, 700, False), (6, 72, 40, 700, True), (5, 576, 328, 4000, activation is None)):
        unit = lambda stem: dict({"up_proj": stem + "up", "down_proj": stem + "down"}, **({"gate_proj": stem + "gate"} if gated else {}))
        params = {"hidden_size": width, "intermediate_size": ff, "experts": E, "top": 2, "gated": gated, "activation": activation,
                  "scoring": {"kind": "sigmoid"}, "weight_on": weight_on, "names": {"router": "r"}, "expert_names": [unit(f"e{e}.") for e in range(E)]}
        if shared:
            params["shared"] = {"kind": "swiglu" if gated else "mlp",
                                "params": {"hidden_size": width, "intermediate_size": 24, "activation": activation, "names": unit("s.")}}
        p = PartProbe("feed_forward", "routed_glu", params, dtype="bfloat16")
        p.bind_random(7, 0.2)
        x = inputs(rows, width, 3, "bfloat16")
        x[:, :16] = bf16_round(x[:, :16] + 2.0)                     # a common direction: some experts get most rows, some none
        many = p.feed_forward(x)
        few = np.concatenate([p.feed_forward(x[at:at + 100]) for at in range(0, rows, 100)])
        close(many, few, 1.5e-2)


def test_a_norm_whose_weight_is_stored_around_zero(tmp_path):
    from purhie_b200.parts import PartProbe
    cfg = config(24, 20, [(channel(1, 1, 4, 4, 1, 2, 2), None)])
    w = draw_weights(cfg, 9)
    folder = make_folder(tmp_path, cfg, w, "F32")
    p = PartProbe("norm", *part_of(cfg, 0, "mixer_norm"))
    p.bind_folder(folder)
    x = inputs(7, 24, 1, "float32")
    close(p.norm(x)[1], P.norm(x.astype(np.float64), 1e-5, f64(w)["l0.norm1"]), 1e-5)


def test_rotation_tables_follow_the_wavelengths():
    from purhie_b200.parts import PartProbe
    for r in (rot(16, 1e4, SCALING), rot(32, 5e5, scaling(4.0, 2.0, 6.0, 300)), rot(8, 100.0, scaling(3.0, 1.0, 1.0, 50)), rot(64, 1e6)):
        params = {"theta": r["base"], "n_rot": r["dims"], "max_position": 700, "pairing": "interleaved"}
        if r["scaling"]:
            params["scaling"] = dict(r["scaling"], kind="wavelength")
        p = PartProbe("position", "rope_neox", params)
        p.bind_random(1)
        t = p.position_table()
        a = np.arange(700)[:, None] * P.frequencies(r)
        half = r["dims"] // 2
        assert np.abs(t[:, :half] - np.cos(a)).max() < 1e-6 and np.abs(t[:, half:] - np.sin(a)).max() < 1e-6


# ---- kernels' own choices inside whole models --------------------------------------------------------------------------
def test_key_splits_and_kernel_choices_agree_with_the_plain_implementation(models):
    from purhie_b200.engine import StepEntry
    for name, choices in (("C", [{}, {"tile16_splits": 3}, {"delta": "scan"}, {"experts": "slices"}]),
                          ("D", [{"decode_splits": 3, "prefill_splits": 2}, {"decode_splits": 8, "prefill_splits": 5}, {"sink_kernel": "tile"}])):
        folder, cfg, w = models[name, "bfloat16"]
        toks = tokens(300, cfg["vocab"], 6)
        ref = P.forward(cfg, w, toks)
        for options in choices:
            eng = engine_for(folder, "bfloat16", max_tokens=1024, step_options=options)
            close_logits(run_cut(eng, "whole", toks, []), ref, "bfloat16")
            close_logits(run_cut(eng, "tail", toks, [2, 250] + [1] * 48), ref, "bfloat16")
            eng.add_request("a"); eng.add_request("b")
            eng.step([StepEntry("a", toks[:200], [])])
            out = eng.step([StepEntry("a", toks[200:201], [0]), StepEntry("b", toks[:130], list(range(130)))])
            close_logits(out, np.concatenate([ref[200:201], ref[:130]]), "bfloat16")
            eng.close()


# ---- generation -----------------------------------------------------------------------------------------------------
def plain_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(P.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_greedy_generation_through_the_entry_point_and_the_scheduler(models, name):
    from purhie_b200.api import load_model
    from purhie_b200.sampling import SamplerParams
    folder, cfg, w = models[name]
    model = load_model(folder, dtype="float32")
    model.kv_cache_init(256, max_sequences=3, page_size=8, max_batch_tokens=24, prefill_chunk=11)
    prompts = [tokens(n, cfg["vocab"], 60 + i) for i, n in enumerate((1, 14, 37))]
    expected = [plain_greedy(cfg, w, p, 10) for p in prompts]
    for p, exp in zip(prompts, expected):
        assert model.generate_ex(p, 10, SamplerParams.greedy()) == exp
    assert model.generate(prompts, max_new_tokens=10) == expected        # chunked prompts beside decoding requests
    model.free()


def test_the_command_line_generates_from_a_folder_of_this_design(models):
    import subprocess
    import sys
    from helpers import ROOT
    folder, cfg, w = models["B"]
    prompt = tokens(12, cfg["vocab"], 8)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "qwen_demo"), folder, ",".join(map(str, prompt)), "5", "--dtype", "float32",
                        "--ctx", "64"], capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    lines = r.stdout.strip().splitlines()
    assert [int(x) for x in lines[2:7]] == plain_greedy(cfg, w, prompt, 5)


def test_trace_replay_reads_a_folder_of_this_design(models, tmp_path):
    from helpers import TraceRun
    folder, cfg, w = models["A"]
    toks = tokens(40, cfg["vocab"], 5)
    ref = P.forward(cfg, w, toks)
    run = TraceRun(folder, "float32", tmp_path, 128)
    run.vocab = cfg["vocab"]
    a = run.step(0, [("x", toks[:17], [0, 16])])
    b = run.step(1, [("x", toks[17:19], [1]), ("y", toks[:3], [2])])
    c = run.step(2, [("x", toks[19:], [20])], end=["x", "y"])
    run.close()
    close(np.concatenate([a.numpy(), b.numpy()[:1], c.numpy()]), ref[[0, 16, 18, 39]], TOL["float32"])
    close(b.numpy()[1:], ref[[2]], TOL["float32"])
