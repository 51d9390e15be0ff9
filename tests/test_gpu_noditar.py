"""The Noditar design in the engine against the plain implementation (GPU): every mechanism alone, whole prompts, cuts
down to two tokens, decoding, unequal batches, pages and state slots used again, keys far away and at page borders, the
first token of a sequence in a state hundreds of tokens later, other sizes than any real model's, and greedy generation
through the entry point and the scheduler."""
import os

import numpy as np
import pytest

from noditar_helpers import (CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_D, CONFIG_E, bf16_round, biased, config, dense, draw_weights, latent, make_folder,
                             mamba2, tokens)
from plain import noditar_plain as P

pytestmark = pytest.mark.gpu

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D, "E": CONFIG_E}
TOL = {"float32": 2e-4, "bfloat16": 6e-2}


def f64(w):
    return {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}


class Models:
    """Per configuration and dtype: (folder, config, weights for the plain implementation); the same values stored in 32
    bits for the float32 runs and as bfloat16 for the others."""

    def __init__(self, factory):
        self.items = {}
        for i, (name, cfg) in enumerate(CONFIGS.items()):
            w = draw_weights(cfg, 800 + i)
            self.items[name, "float32"] = (make_folder(factory.mktemp(f"nd_{name}_f32"), cfg, w, "F32"), cfg, f64(w))
            self.items[name, "bfloat16"] = (make_folder(factory.mktemp(f"nd_{name}_bf16"), cfg, w, "BF16"), cfg, f64(w))

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


def close(got, ref, tol):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape
    assert np.isfinite(got).all()
    err = np.abs(got - ref).max() / max(np.abs(ref).max(), 1e-30)
    assert err < tol, f"relative error {err:.3e} (allowed {tol:.1e})"


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
    part = spec["layers"][layer]["parts"][name] if layer is not None else spec[name]
    return part["kind"], part["params"]


def probe(cfg, layer, folder, dtype, pages=80, slots=3):
    from purhie_b200.parts import PartProbe
    p = PartProbe("mixer", *part_of(cfg, layer, "mixer"), dtype=dtype)
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
    close(whole, ref, TOL[dtype])
    # one token (the first of a sequence alone), then two, then portions of changing size, single tokens between them
    cut = run_cut(eng, "cut", toks, [1, 2, 2, 5, 1, 1, 16, 3, 17, 2, 1])
    close(cut, ref, TOL[dtype])
    # a prompt, then token by token: every decode step replays a graph
    tail = run_cut(eng, "tail", toks, [30] + [1] * 45)
    close(tail, ref, TOL[dtype])
    if dtype == "float32":                      # the 32-bit kernels add in one order however the tokens arrive
        assert np.abs(cut - whole).max() <= 1e-5 * np.abs(ref).max()
        assert np.abs(tail - whole).max() <= 1e-5 * np.abs(ref).max()
    eng.check_cache()
    eng.close()


def test_every_layer_agrees_with_the_plain_implementation(models):
    """The sum of the streams after each layer, so that a fault shows where it starts."""
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


def test_the_streams_are_mixed_from_old_to_new_and_each_weight_counts(models):
    """The comparison above can tell a mix matrix read the other way round, streams that start unequal, and a part whose
    output enters every stream alike."""
    for name in ("A", "C"):
        _, cfg, w = models[name]
        toks = tokens(20, cfg["vocab"], 2)
        ref = P.forward(cfg, w, toks)
        for end, change in ((".mix", lambda a: a.T), (".out", lambda a: np.full_like(a, a.mean())), (".in", lambda a: np.full_like(a, a.mean()))):
            other = {k: (change(v) if ".hc" in k and k.endswith(end) else v) for k, v in w.items()}
            moves(P.forward(cfg, other, toks), ref, 0.2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(models, name, dtype):
    from purhie_b200.engine import StepEntry
    folder, cfg, w = models[name, dtype]
    # room for two requests' states and about 100 tokens: five requests must take turns, pages come back poisoned
    eng = engine_for(folder, dtype, max_tokens=104, max_requests=2)
    lengths = [41, 9, 1, 56, 23]
    reqs = {f"r{i}": tokens(n, cfg["vocab"], 20 + i) for i, n in enumerate(lengths)}
    refs = {r: P.forward(cfg, w, t) for r, t in reqs.items()}
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
    for r in reqs:
        close(np.concatenate(got[r]), refs[r], TOL[dtype])
    eng.close()


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "bfloat16"), ("C", "float32"), ("D", "bfloat16")])
def test_a_long_prompt_alone_and_beside_a_decode_row_and_a_two_token_portion(models, name, dtype):
    """330 tokens: several chunks of the state-space scan, hundreds of keys."""
    from purhie_b200.engine import StepEntry
    folder, cfg, w = models[name, dtype]
    eng = engine_for(folder, dtype, max_tokens=1024)
    toks = tokens(330, cfg["vocab"], 11)
    ref = P.forward(cfg, w, toks)
    close(run_cut(eng, "whole", toks, []), ref, TOL[dtype])
    close(run_cut(eng, "cut", toks, [2, 63, 64, 65, 1, 2, 100]), ref, TOL[dtype])
    eng.add_request("a"); eng.add_request("b"); eng.add_request("c")
    eng.step([StepEntry("b", toks[:5], []), StepEntry("c", toks[:9], [])])
    out = eng.step([StepEntry("b", toks[5:6], [0]), StepEntry("a", toks[:300], list(range(300))), StepEntry("c", toks[9:11], [0, 1])])
    close(out[1:301], ref[:300], TOL[dtype])
    close(out[:1], ref[5:6], TOL[dtype])
    close(out[301:], ref[9:11], TOL[dtype])
    eng.close()


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "bfloat16")])
def test_long_decoding_keeps_its_state(models, name, dtype):
    folder, cfg, w = models[name, dtype]
    eng = engine_for(folder, dtype, max_tokens=256)
    toks = tokens(230, cfg["vocab"], 3)
    close(run_cut(eng, "long", toks, [2] + [1] * 228), P.forward(cfg, w, toks), TOL[dtype])
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


# latents of 12 to 512: every width of the tensor-core kernel, and 12 and 20, which go the plain way; one head alone
LATENTS = {
    "r12": (latent(4, 16, 20, 12, 2.0), 64), "r20": (latent(3, 24, 8, 20, 1.5), 40), "r64": (latent(8, 32, 48, 64, 1.0), 72),
    "r136": (latent(5, 48, 40, 136, 0.7), 64), "r256": (latent(1, 64, 64, 256, 0.5), 48), "r264": (latent(6, 40, 24, 264, 0.6), 64),
    "r512": (latent(2, 128, 128, 512, 0.4), 64), "r72": (latent(3, 128, 128, 72, 0.3), 40),      # long portions: keys and values of their own
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(LATENTS))
def test_attention_through_a_latent_alone(tmp_path, which, dtype):
    kind_m, width = LATENTS[which]
    cfg = config(width, 20, 2, [(kind_m, None)])
    w = draw_weights(cfg, 3, std=0.4)
    folder = make_folder(tmp_path, cfg, w, "F32" if dtype == "float32" else "BF16")
    x, wd, m, eps = inputs(260, width, 1, dtype), f64(w), kind_m[1], cfg["norm"]["eps"]
    ref = P.latent_attention(x.astype(np.float64), wd, "l0.mix.", m, eps)
    tol = 2e-4 if dtype == "float32" else 3e-2
    # a missing gate, a gate per head, a latent without its norm's weight, another scale each show
    moves(P.latent_attention(x.astype(np.float64), dict(wd, **{"l0.mix.g": 0 * wd["l0.mix.g"]}), "l0.mix.", m, eps), ref, 2 * tol)
    per_head = np.repeat(wd["l0.mix.g"][::m["vdim"]], m["vdim"], axis=0)
    moves(P.latent_attention(x.astype(np.float64), dict(wd, **{"l0.mix.g": per_head}), "l0.mix.", m, eps), ref, 2 * tol)
    moves(P.latent_attention(x.astype(np.float64), dict(wd, **{"l0.mix.dkv.norm": 1 + 0 * wd["l0.mix.dkv.norm"]}), "l0.mix.", m, eps), ref, 2 * tol)
    moves(P.latent_attention(x.astype(np.float64), wd, "l0.mix.", dict(m, scale=1.3 * m["scale"]), eps), ref, 2 * tol)
    whole_cut_decoded_and_batched(probe(cfg, 0, folder, dtype), x, ref, tol)


# groups of 1 to 6, one head alone, forty heads (more than a tile kernel takes); heads of 128 take the tcgen05 and TMA kernels,
# 16, 32, 48, 64 (with other values too) the tile kernel, the rest the plain one
BIASED = {
    "h4": (biased(4, 2, 16, 16, 0.9), 64), "h6": (biased(6, 1, 24, 40, 0.5), 48), "h1": (biased(1, 1, 40, 8, 0.6), 40), "h8": (biased(8, 2, 48, 48, 0.3), 72),
    "h3": (biased(3, 3, 64, 32, 0.3), 24), "h40": (biased(40, 8, 8, 8, 1.2), 56), "h24": (biased(24, 4, 32, 32, 0.5), 48),
    "d128": (biased(4, 1, 128, 128, 0.12), 48), "d128h8": (biased(8, 4, 128, 128, 0.2), 64), "d64": (biased(4, 1, 64, 64, 0.3), 64),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(BIASED))
def test_attention_with_a_distance_bias_a_sink_and_a_gate_alone(tmp_path, which, dtype):
    kind_m, width = BIASED[which]
    cfg = config(width, 20, 2, [(kind_m, None)])
    w = draw_weights(cfg, 4, std=0.5)
    folder = make_folder(tmp_path, cfg, w, "F32" if dtype == "float32" else "BF16")
    x, wd, m, eps = inputs(260, width, 2, dtype), f64(w), kind_m[1], cfg["norm"]["eps"]
    at = lambda **kw: P.biased_attention(x.astype(np.float64), wd, "l0.mix.", m, eps, **kw)
    ref = at()
    tol = 2e-4 if dtype == "float32" else 3e-2
    # a softmax without the sink, slopes a head off, slopes left out, norms left out (an eps that dwarfs the squares), no gate
    moves(at(sink=False), ref, 2 * tol)
    H = m["heads"]
    moves(at(slopes=2.0 ** (-8.0 * np.arange(H) / H)), ref, 2 * tol)
    moves(at(slopes=np.zeros(H)), ref, 2 * tol)
    moves(P.biased_attention(x.astype(np.float64), wd, "l0.mix.", m, 1e4), ref, 2 * tol)
    moves(P.biased_attention(x.astype(np.float64), dict(wd, **{"l0.mix.g": 0 * wd["l0.mix.g"]}), "l0.mix.", m, eps), ref, 2 * tol)
    whole_cut_decoded_and_batched(probe(cfg, 0, folder, dtype), x, ref, tol)


# states, groups, taps and norm parts of every kind; r32, r64 and r72 run long portions in chunks on the tensor cores
MAMBAS = {
    "r32": (mamba2(6, 32, 40, 2, 4, 3), 64), "r64": (mamba2(2, 64, 128, 1, 3, 4), 48), "r72": (mamba2(3, 72, 8, 3, 2, 1), 40), "r5": (mamba2(6, 5, 7, 2, 5, 10), 32),
    "r16": (mamba2(1, 16, 200, 1, 1, 1), 24), "r8": (mamba2(8, 8, 16, 8, 4, 16), 56), "r40": (mamba2(2, 40, 256, 2, 4, 2), 32),
}


def mamba_case(tmp_path, which, dtype, seed=5):
    kind_m, width = MAMBAS[which]
    cfg = config(width, 20, 2, [(kind_m, None)])
    w = draw_weights(cfg, seed, std=0.4)
    return cfg, w, make_folder(tmp_path, cfg, w, "F32" if dtype == "float32" else "BF16"), width


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(MAMBAS))
def test_the_second_mamba_form_alone(tmp_path, which, dtype):
    cfg, w, folder, width = mamba_case(tmp_path, which, dtype)
    x, wd, m, eps = inputs(260, width, 3, dtype), f64(w), cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    at = lambda weights, mixer=m: P.mamba2(x.astype(np.float64), weights, "l0.mix.", mixer, eps)
    ref = at(wd)
    tol = 2e-4 if dtype == "float32" else 3e-2
    # each of these left out, or taken the other way round, shows (the first four in 32 bits)
    zero = lambda n: dict(wd, **{"l0.mix." + n: 0 * wd["l0.mix." + n]})
    for n in ("D", "A_log", "dt_bias", "conv.b"):
        moves(at(zero(n)), ref, 6e-4)
    if m["conv"] > 1:
        moves(at(dict(wd, **{"l0.mix.conv": wd["l0.mix.conv"][:, ::-1]})), ref, 2 * tol)
    if m["norm_groups"] > 1:
        moves(at(wd, dict(m, norm_groups=1)), ref, 2 * tol)
    whole_cut_decoded_and_batched(probe(cfg, 0, folder, dtype), x, ref, tol)


def test_chunks_and_single_steps_of_the_scan_agree_wherever_a_prompt_is_cut(tmp_path):
    """bfloat16: the same rows in one portion (chunks), in portions either side of a chunk's edge, in portions short enough to
    go token by token, and one by one."""
    cfg, w, folder, width = mamba_case(tmp_path, "r64", "bfloat16")
    x = inputs(200, width, 4, "bfloat16")
    ref = P.mamba2(x.astype(np.float64), f64(w), "l0.mix.", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    p = probe(cfg, 0, folder, "bfloat16")
    for pieces in ([200], [64, 64, 72], [63, 65, 72], [32, 31, 33, 104], [31] * 6 + [14], [1] * 200, [1, 128, 1, 70], [2, 33, 2, 2, 161]):
        close(mixer_in_pieces(p, x, pieces, 1), ref, 3e-2)


def test_the_first_token_still_shows_hundreds_of_tokens_later_in_a_state_that_hardly_forgets(tmp_path):
    for dtype in ("float32", "bfloat16"):
        cfg, w, folder, width = mamba_case(tmp_path / dtype, "r32", dtype)
        w["l0.mix.A_log"] = np.full(6, -7.0, dtype=np.float32)                # a decay of about 1/1000 per unit of dt
        folder = make_folder(tmp_path / dtype, cfg, w, "F32" if dtype == "float32" else "BF16")
        m, eps, wd = cfg["layers"][0]["mixer"], cfg["norm"]["eps"], f64(w)
        x = inputs(400, width, 4, dtype)
        y = x.copy()
        y[0] = bf16_round(y[0] * 40.0)                                         # a first token that writes a state far above the others'
        at = lambda v: P.mamba2(v.astype(np.float64), wd, "l0.mix.", m, eps)
        ref_x, ref_y = at(x), at(y)
        moves(ref_y[-1], ref_x[-1], 0.3)
        p = probe(cfg, 0, folder, dtype)
        tol = 2e-4 if dtype == "float32" else 3e-2
        close(mixer_in_pieces(p, y, [1, 200] + [1] * 199, 1), ref_y, tol)
        close(mixer_in_pieces(p, y, [400], 2), ref_y, tol)
        close(mixer_in_pieces(p, x, [400], 1), ref_x, tol)                      # the slot again: nothing is left of y


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dims", [(16, 16, 40), (64, 32, 128)])
def test_a_far_key_decides_the_output_of_attention_through_a_latent(tmp_path, dims, dtype):
    """Row `at` is built so that its key is what every later query asks for: it takes nearly all their weight, however far."""
    dim, vdim, rank = dims
    T, at = 300, 39                                                            # the last slot of a page
    cfg = config(64, 20, 2, [(latent(2, dim, vdim, rank, 4.0 / dim), None)])
    w = draw_weights(cfg, 6, std=0.4)
    m, eps, wd = cfg["layers"][0]["mixer"], cfg["norm"]["eps"], f64(w)
    x = np.random.default_rng(3).normal(0, 1.0, (T, 64))
    x[at + 1:] = x[at + 1] * (1.0 + 0.01 * np.arange(T - at - 1))[:, None] / 2.0      # later queries all ask for the same key
    q = x[at + 1] @ wd["l0.mix.q"].T
    c = wd["l0.mix.uk"][:dim].T @ q[:dim]                                       # the latent whose first head's key lines up
    x[at] = 3.0 * np.linalg.lstsq(wd["l0.mix.dkv"], c / wd["l0.mix.dkv.norm"] / np.linalg.norm(c) * np.sqrt(rank), rcond=None)[0]
    x = bf16_round(x.astype(np.float32))
    ref = P.latent_attention(x.astype(np.float64), wd, "l0.mix.", m, eps)
    without = x.astype(np.float64).copy()
    without[at] = -without[at]
    moves(P.latent_attention(without, wd, "l0.mix.", m, eps)[-1], ref[-1], 0.2)
    folder = make_folder(tmp_path, cfg, w, "F32" if dtype == "float32" else "BF16")
    p = probe(cfg, 0, folder, dtype)
    tol = 2e-4 if dtype == "float32" else 4e-2
    for pieces in ([T], [at, 1, 7, T - at - 8], [at - 1, 2, T - at - 1], [T - 60] + [1] * 60, [at + 1, T - at - 1 - 2, 2]):
        close(mixer_in_pieces(p, x, pieces, 1), ref, tol)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim", [16, 24, 128])
def test_a_far_key_against_the_distance_bias(tmp_path, dim, dtype):
    """The last of eight heads loses 1/256 per position: a key that lines up wins over near ones from 250 positions away, and
    the weight it has left depends on the distance being counted right."""
    T, at = 300, 39
    cfg = config(64, 20, 2, [(biased(8, 8, dim, dim, 14.0 / dim), None)])
    w = draw_weights(cfg, 7, std=0.4)
    m, eps, wd = cfg["layers"][0]["mixer"], cfg["norm"]["eps"], f64(w)
    x = np.random.default_rng(3).normal(0, 1.0, (T, 64))
    x[at + 1:] = x[at + 1] * (1.0 + 0.01 * np.arange(T - at - 1))[:, None] / 2.0
    q = x[at + 1] @ wd["l0.mix.q"].T
    x[at] = 3.0 * np.linalg.lstsq(wd["l0.mix.k"][7 * dim:], q[7 * dim:], rcond=None)[0]      # the last head's key lines up
    x = bf16_round(x.astype(np.float32))
    ref = P.biased_attention(x.astype(np.float64), wd, "l0.mix.", m, eps)
    without = x.astype(np.float64).copy()
    without[at] = -without[at]
    moves(P.biased_attention(without, wd, "l0.mix.", m, eps)[-1], ref[-1], 0.1)
    folder = make_folder(tmp_path, cfg, w, "F32" if dtype == "float32" else "BF16")
    p = probe(cfg, 0, folder, dtype)
    tol = 2e-4 if dtype == "float32" else 4e-2
    for pieces in ([T], [at, 1, 7, T - at - 8], [at - 1, 2, T - at - 1], [T - 60] + [1] * 60):
        close(mixer_in_pieces(p, x, pieces, 1), ref, tol)


def test_the_sink_takes_its_share_of_the_first_tokens(tmp_path):
    """A request's first token sees itself and the sink: its value enters with exp(s) / (1 + exp(s)), not with 1."""
    for dtype, dim in (("float32", 12), ("bfloat16", 32), ("bfloat16", 128)):
        cfg = config(40, 20, 2, [(biased(2, 1, dim, dim, 0.5 / dim), None)])
        w = draw_weights(cfg, 8, std=0.5)
        folder = make_folder(tmp_path / f"{dtype}{dim}", cfg, w, "F32" if dtype == "float32" else "BF16")
        x, m, eps = inputs(3, 40, 6, dtype), cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
        ref = P.biased_attention(x.astype(np.float64), f64(w), "l0.mix.", m, eps)
        moves(P.biased_attention(x.astype(np.float64), f64(w), "l0.mix.", m, eps, sink=False)[:1], ref[:1], 0.4)
        p = probe(cfg, 0, folder, dtype)
        for pieces in ([3], [1, 1, 1], [2, 1], [1, 2]):
            close(mixer_in_pieces(p, x, pieces, 1), ref, 2e-4 if dtype == "float32" else 3e-2)


def test_the_feed_forward_alone_with_clamps_that_bite(models):
    from purhie_b200.parts import PartProbe
    for name, layer, dtype in (("A", 0, "float32"), ("A", 1, "float32"), ("B", 3, "float32"), ("C", 4, "bfloat16"), ("C", 5, "bfloat16")):
        folder, cfg, w = models[name, dtype]
        limit = cfg["layers"][layer]["mlp"]["limit"]
        x = inputs(37, cfg["width"], layer, dtype, 2.0)
        ref = P.clamped_unit(x.astype(np.float64), w, f"l{layer}.mlp.", limit)
        moves(P.clamped_unit(x.astype(np.float64), w, f"l{layer}.mlp.", 1.2 * limit), ref, 0.03)
        p = PartProbe("feed_forward", *part_of(cfg, layer, "feed_forward"), dtype=dtype)
        p.bind_folder(folder)
        tol = 2e-4 if dtype == "float32" else 2e-2
        close(p.feed_forward(x), ref, tol)
        close(p.feed_forward(x[:1]), ref[:1], tol)


# ---- kernels' own choices inside whole models --------------------------------------------------------------------------
def test_key_splits_and_kernel_choices_agree_with_the_plain_implementation(models):
    from purhie_b200.engine import StepEntry
    for name, choices in (("C", [{}, {"tile16_splits": 3}, {"latent_splits": 4}, {"ssd": "scan"}, {"ssd_chunk_rows": 2}]),
                          ("D", [{"decode_splits": 3, "prefill_splits": 2}, {"decode_splits": 8, "prefill_splits": 5}, {"sink_kernel": "tile"}])):
        folder, cfg, w = models[name, "bfloat16"]
        toks = tokens(300, cfg["vocab"], 6)
        ref = P.forward(cfg, w, toks)
        for options in choices:
            eng = engine_for(folder, "bfloat16", max_tokens=1024, step_options=options)
            close(run_cut(eng, "whole", toks, []), ref, TOL["bfloat16"])
            close(run_cut(eng, "tail", toks, [2, 250] + [1] * 48), ref, TOL["bfloat16"])
            eng.add_request("a"); eng.add_request("b")
            eng.step([StepEntry("a", toks[:200], [])])
            out = eng.step([StepEntry("a", toks[200:201], [0]), StepEntry("b", toks[:130], list(range(130)))])
            close(out[:1], ref[200:201], TOL["bfloat16"])
            close(out[1:], ref[:130], TOL["bfloat16"])
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
