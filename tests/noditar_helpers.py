"""Small Noditar configurations and model folders with weights the tests choose themselves."""
import numpy as np

from bozosun_helpers import bf16_round, make_folder, tokens, write_safetensors  # noqa: F401  (re-exported)


def latent(heads, dim, vdim, kv_rank, scale=None):
    return ("latent_attention", {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale if scale is not None else dim ** -0.5})


def biased(heads, kv_heads, dim, vdim, scale=None):
    return ("attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5})


def mamba2(heads, vdim, state, groups, conv, norm_groups):
    return ("mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups})


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def config(width, vocab, streams, layers, eps=1e-5):
    return {"architecture": "Noditar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "layers": [{"type": kind, "mixer": m, "mlp": mlp} for (kind, m), mlp in layers]}


# Configurations that differ in every size.  Two, three, five and nine streams and one alone; layers without a feed-forward of
# every kind of mixer; heads of 8 to 128; values narrower and wider than keys; groups of 1, 2, 3 and 5 query heads; latents
# narrower and wider than a head, and of a width the tensor-core kernel does not take; states of 6 to 144 with one group for
# all heads, several, and one per head; convolutions of 1, 2, 3, 4 and 6 taps; one norm part, several, and more than heads;
# widths that no vector access fits; clamps that bite and clamps that do not.
CONFIG_A = config(48, 80, 2, [
    (latent(3, 16, 24, 40, 0.3), dense(64, 1.1)),
    (mamba2(6, 8, 12, 3, 3, 4), dense(40, 0.6)),
    (biased(4, 2, 12, 20, 0.4), None),
    (biased(5, 1, 8, 8, 0.5), dense(24, 3.0)),
    (latent(1, 24, 8, 12, 0.25), None),
], eps=1e-6)

CONFIG_B = config(42, 70, 5, [
    (mamba2(3, 10, 6, 1, 6, 1), None),
    (biased(3, 3, 20, 10, 0.25), dense(30, 0.9)),
    (latent(5, 8, 14, 30, 0.5), dense(54, 2.5)),
    (mamba2(4, 24, 33, 4, 1, 12), dense(18, 1.4)),
], eps=1e-3)

# wider layers, stored in bfloat16: what the tensor-core kernels take (chunks of the state-space scan, tiles of attention)
CONFIG_C = config(128, 200, 3, [
    (mamba2(4, 32, 64, 2, 4, 2), dense(192, 1.5)),
    (biased(6, 2, 32, 32, 0.2), dense(128, 2.0)),
    (latent(4, 32, 48, 64, 0.2), None),
    (mamba2(2, 72, 144, 1, 2, 3), None),
    (biased(4, 4, 64, 64, 0.15), dense(256, 1.0)),
    (latent(6, 48, 32, 160, 0.15), dense(96, 0.8)),
], eps=1e-6)

# heads of 128, which take the tcgen05 prompt kernel and the TMA decode kernel; one stream; a latent of 512 whose heads of
# 128 / 128 get keys and values of their own for long portions, and one of 264 whose heads do not
CONFIG_D = config(96, 60, 1, [
    (biased(4, 2, 128, 128, 0.09), dense(64, 1.3)),
    (latent(2, 128, 128, 512, 0.09), None),
    (biased(2, 2, 128, 128, 0.07), None),
    (latent(3, 64, 128, 264, 0.1), dense(48, 2.0)),
], eps=1e-5)

# nine streams: more than the vector kernel keeps in registers
CONFIG_E = config(32, 50, 9, [(latent(2, 8, 8, 16, 0.4), dense(24, 1.0)), (biased(2, 1, 16, 16, 0.3), None)], eps=1e-5)


def draw_weights(cfg, seed, std=0.3):
    """Weights for every tensor the framework says the configuration reads: matrices N(0, 3 std / sqrt(fan_in)) so that
    activations stay of order one, norm weights around 1, the streams' mixing matrices near a rotation of the identity so
    that [from, to] and [to, from] differ, step sizes and decays that forget within a few to a few hundred tokens."""
    from purhie_b200.weights import expected_tensors
    rng = np.random.default_rng(seed)
    out = {}
    for name, spec in expected_tensors(cfg).items():
        shape = tuple(spec.shape)
        if name.endswith(".mix") and ".hc" in name:
            s = shape[0]
            a = 0.7 * np.eye(s) + 0.3 * np.roll(np.eye(s), 1, axis=1) + rng.normal(0.0, 0.25 / np.sqrt(s), shape)
        elif name.endswith((".in", ".out")) and ".hc" in name:
            a = rng.normal(0.4, 0.6, shape) if name.endswith(".in") else rng.normal(0.7, 0.5, shape)
        elif name.endswith("A_log"):
            a = rng.uniform(-2.0, 1.0, shape)
        elif name.endswith("dt_bias"):
            a = rng.uniform(-3.0, 0.5, shape)
        elif name.endswith("mix.D"):
            a = rng.uniform(-1.0, 1.5, shape)
        elif name.endswith("conv"):
            a = rng.normal(0.0, 0.6, shape)
        elif name.endswith("conv.b"):
            a = rng.normal(0.0, 0.3, shape)
        elif spec.init == "scale":
            a = rng.uniform(0.5, 1.5, shape)
        elif len(shape) == 2:
            a = rng.normal(0.0, std * 3.0 / np.sqrt(shape[1]), shape)
        else:
            a = rng.normal(0.0, std, shape)
        if name.endswith("mix.conv.b"):
            # B and C mostly positive: a read-out C . B that is a difference of like terms has a sign that a bfloat16 rounding
            # can turn, and the norm behind it keeps little but the sign
            m = cfg["layers"][int(name[1:].split(".")[0])]["mixer"]
            a[m["heads"] * m["vdim"]:] += 1.5
        out[name] = bf16_round(np.asarray(a, dtype=np.float32))          # representable in either storage
    return out
