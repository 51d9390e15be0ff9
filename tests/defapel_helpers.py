"""Small Defapel configurations and model folders with weights the tests choose themselves."""
import numpy as np

from bozosun_helpers import bf16_round, make_folder, tokens, write_safetensors  # noqa: F401  (re-exported)


def channel(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return ("channel_delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank,
                              "gate_rank": gate_rank})


def rot(dims, base=1e4, scaling=None):
    return {"base": base, "dims": dims, "scaling": scaling}


def scaling(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def window(heads, kv_heads, dim, vdim, size, rot_, scale=None, softcap=4.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": rot_,
            "scale": scale if scale is not None else dim ** -0.5, "softcap": softcap}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def parallel(left, right, left_scale, right_scale):
    return ("parallel", {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale})


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Defapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [{"type": kind, "mixer": m, "mlp": mlp} for (kind, m), mlp in layers]}


SCALING = scaling(8.0, 1.0, 4.0, 64)

# Configurations that differ in every size.  Groups of 1, 2, 3 and 4 heads on both sides; heads of 6 to 128 with values narrower
# and wider than keys; convolutions of 1, 2, 3, 4 and 6 taps; low ranks of 3 to 16 that differ between decay and gate; windows
# shorter than a page, of a page, and longer than any test; rotation over a whole head, part of one and none, with and without
# stretched frequencies; caps that bite; one and several chosen experts, all of them, layers without a feed-forward; widths
# that no vector access fits.
CONFIG_A = config(48, 80, [
    (parallel(window(4, 2, 12, 20, 11, rot(8, 1e4, SCALING)), delta(6, 2, 8, 12, 3), 0.8, 1.3), moe(24, 5, 2)),
    (channel(3, 1, 10, 14, 4, 5, 3), moe(20, 3, 1)),
    (parallel(window(3, 3, 16, 8, 40, rot(16, 100.0)), delta(2, 2, 16, 20, 2), 1.2, -0.6), None),
    (channel(4, 2, 16, 8, 1, 6, 11), moe(16, 4, 4)),
], eps=1e-6)

CONFIG_B = config(42, 70, [
    (channel(2, 2, 6, 18, 6, 7, 16), None),
    (parallel(window(6, 1, 20, 10, 8, rot(0)), delta(4, 1, 24, 6, 4), 0.5, 0.5), moe(30, 7, 3)),
    (channel(6, 3, 12, 12, 2, 3, 4), moe(18, 2, 1)),
], eps=1e-3, logit_scale=2.5)

# wider layers, stored in bfloat16: what the tensor-core kernels take (chunks of the recurrence, tiles of attention)
CONFIG_C = config(128, 200, [
    (channel(4, 2, 32, 48, 4, 16, 16), moe(64, 4, 2)),
    (parallel(window(4, 2, 64, 64, 70, rot(32, 1e4, scaling(4.0, 2.0, 6.0, 128))), delta(4, 4, 64, 32, 3), 1.1, 0.7), moe(48, 6, 1)),
    (parallel(window(6, 2, 32, 32, 33, rot(32)), delta(3, 1, 48, 40, 4), 0.9, 0.9), None),
    (channel(2, 2, 128, 64, 3, 24, 8), moe(96, 3, 2)),
], eps=1e-6, logit_scale=0.5)

# heads of 128, which take the tcgen05 prompt kernel and the TMA decode kernel
CONFIG_D = config(96, 60, [
    (parallel(window(4, 2, 128, 128, 90, rot(128, 1e6, SCALING), 0.09, 3.0), delta(2, 1, 64, 64, 4), 0.7, 1.1), moe(64, 4, 2)),
    (channel(2, 1, 64, 96, 4, 8, 8), None),
    (parallel(window(2, 2, 128, 128, 500, rot(64), 0.07, 50.0), delta(2, 2, 16, 128, 2), 1.0, 1.0), moe(32, 2, 1)),
], eps=1e-5, logit_scale=1.0)


def draw_weights(cfg, seed, std=0.3):
    """Weights for every tensor the framework says the configuration reads: matrices N(0, 3 std / sqrt(fan_in)) so that
    activations stay of order one, layer norms' weights around zero, decays that forget within a few to a few hundred tokens.
    q and k of a delta rule share a part, so that a read-out S^T q is not a difference of like terms whose sign a rounding
    turns (the norm behind it keeps little but the direction)."""
    from purhie_b200.weights import expected_tensors
    rng = np.random.default_rng(seed)
    out = {}
    for name, spec in expected_tensors(cfg).items():
        shape = tuple(spec.shape)
        if name.endswith("A_log"):
            a = rng.uniform(-2.0, 1.0, shape)
        elif name.endswith("dt_bias"):
            a = rng.uniform(-4.0, 0.0, shape)
        elif name.endswith(".conv"):
            a = rng.normal(0.0, 0.5, shape)
            a[:, -1] += 0.8
        elif name.endswith(("norm1", "norm2", "final.norm")):
            a = rng.uniform(-0.5, 0.5, shape)
        elif spec.init == "scale":
            a = rng.uniform(0.5, 1.5, shape)
        elif len(shape) == 2:
            a = rng.normal(0.0, std * 3.0 / np.sqrt(shape[1]), shape)
        else:
            a = rng.normal(0.0, std, shape)
        out[name] = a
    for name in list(out):
        if name.endswith(".q.conv"):
            stem = name[:-len("q.conv")]
            out[stem + "q"] = 0.8 * out[stem + "k"] + 0.6 * out[stem + "q"]
            out[stem + "q.conv"] = out[stem + "k.conv"] + 0.2 * out[stem + "q.conv"]
    return {n: bf16_round(np.asarray(a, dtype=np.float32)) for n, a in out.items()}          # representable in either storage
