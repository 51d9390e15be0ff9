"""The kernels the Noditar design added, each alone against a plain PyTorch reference in float64 (GPU)."""
import math

import pytest
import torch

from test_gpu_kernels import DEV, paged_case, rel, rnd

pytestmark = pytest.mark.gpu


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ---- the residual of several lanes -----------------------------------------------------------------------------------
# clusters for few rows, a block per row for many; one to nine lanes; widths that no vector access fits
@pytest.mark.parametrize("S,E,T,splits", [(3, 320, 5, 1), (4, 4096, 8, 9), (4, 4096, 200, 1), (2, 2048, 70, 3), (1, 512, 3, 2), (5, 1000, 66, 1),
                                          (8, 8192, 2, 4), (7, 50, 9, 3), (9, 128, 4, 2), (3, 12000, 3, 1), (3, 4, 65, 1)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_lanes_rmsnorm(S, E, T, splits, out_dtype):
    from purhie_b200.csrc import ops
    X, add = rnd(T, S, E, seed=1), rnd(splits, T, E, seed=2)
    mix, out, in_, w = rnd(S, S, seed=3), rnd(S, seed=4), rnd(S, seed=5), rnd(E, seed=6) + 1.0
    tol = 3e-6 if out_dtype == torch.float32 else 8e-3
    d = lambda t: t.double().cpu()
    new = torch.einsum("st,nse->nte", d(mix), d(X)) + d(out)[None, :, None] * d(add).sum(0)[:, None, :]

    def normed(lanes, a, weight):
        u = torch.einsum("s,nse->ne", a, lanes)
        return u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-5) * weight
    y = torch.full((T, E), float("nan"), dtype=out_dtype, device=DEV)
    lanes = X.clone()
    ops.lanes_rmsnorm(lanes, S, lanes, add, mix, out, in_, w, 1e-5, y)                        # in place
    assert rel(lanes.cpu(), new) < 3e-6 and rel(y.cpu(), normed(new, d(in_), d(w))) < tol
    # gathered rows, the plain sum, nothing written back
    rows = i32([T - 1, 0, T // 2])
    part = torch.full((3, E), float("nan"), dtype=out_dtype, device=DEV)
    lanes = X.clone()
    ops.lanes_rmsnorm(lanes, S, None, add, mix, out, None, w, 1e-5, part, rows=rows)
    assert torch.equal(lanes, X) and rel(part.cpu(), normed(new, torch.ones(S).double(), d(w))[[T - 1, 0, T // 2]]) < tol
    # no addend; no norm (the sum itself)
    ops.lanes_rmsnorm(lanes, S, None, None, None, None, in_, w, 1e-5, y)
    assert rel(y.cpu(), normed(d(X), d(in_), d(w))) < tol
    ops.lanes_rmsnorm(lanes, S, None, add, mix, out, in_, None, 0.0, y)
    assert rel(y.cpu(), torch.einsum("s,nse->ne", d(in_), new)) < tol
    # the first update: every lane is one row
    x = X[:, 0].contiguous()
    fresh = torch.full((T, S, E), float("nan"), dtype=torch.float32, device=DEV)
    ops.lanes_rmsnorm(x, S, fresh, add, mix, out, in_, w, 1e-5, y)
    first = d(mix).sum(0)[None, :, None] * d(x)[:, None, :] + d(out)[None, :, None] * d(add).sum(0)[:, None, :]
    assert rel(fresh.cpu(), first) < 3e-6 and rel(y.cpu(), normed(first, d(in_), d(w))) < tol


def test_lanes_rmsnorm_of_a_bfloat16_addend():
    from purhie_b200.csrc import ops
    S, E, T = 3, 192, 6
    X, add = rnd(T, S, E, seed=1), rnd(2, T, E, dtype=torch.bfloat16, seed=2)
    mix, out, in_, w = rnd(S, S, seed=3), rnd(S, seed=4), rnd(S, seed=5), rnd(E, seed=6) + 1.0
    new = torch.einsum("st,nse->nte", mix.double(), X.double()) + out.double()[None, :, None] * add.double().sum(0)[:, None, :]
    u = torch.einsum("s,nse->ne", in_.double(), new)
    y = torch.empty(T, E, dtype=torch.float32, device=DEV)
    ops.lanes_rmsnorm(X, S, X, add, mix, out, in_, w, 1e-5, y)
    assert rel(X, new) < 3e-6 and rel(y, u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-5) * w.double()) < 3e-6


# ---- the second Mamba form -----------------------------------------------------------------------------------------------
def ssd_case(H, P, N, G, K, lens, dtype, seed, fast_decay=False):
    T, inner = sum(lens), H * P
    CH = inner + 2 * G * N
    xbc = rnd(T, CH, dtype=dtype, seed=seed)
    rows = rnd(T, inner + CH + H, dtype=dtype, seed=seed + 1)
    dt_bias = rnd(H, seed=seed + 2, scale=0.5) - 1.5
    a = -torch.exp(rnd(H, seed=seed + 3)) * (20.0 if fast_decay else 1.0)
    d = rnd(H, seed=seed + 4)
    slots = list(range(len(lens)))[::-1]
    floats = (inner * N + (K - 1) * CH + 3) // 4 * 4
    state = rnd(len(lens) + 1, floats, seed=seed + 5)
    seg_start = i32([0] + torch.tensor(lens).cumsum(0).tolist())
    # float64, token by token
    y = torch.zeros(T, H, P, dtype=torch.float64)
    after = state.double().cpu().clone()
    f = lambda t: t.double().cpu()
    X, B, C = f(xbc)[:, :inner].view(T, H, P), f(xbc)[:, inner:inner + G * N].view(T, G, N), f(xbc)[:, inner + G * N:].view(T, G, N)
    group = torch.arange(H) // (H // G)
    at = 0
    for n, slot in zip(lens, slots):
        S = after[slot, :inner * N].view(H, P, N).clone()
        past = after[slot, inner * N:inner * N + (K - 1) * CH].view(K - 1, CH).clone()
        for t in range(at, at + n):
            dt = torch.nn.functional.softplus(f(rows)[t, inner + CH:] + f(dt_bias), threshold=100.0)
            S = torch.exp(f(a) * dt)[:, None, None] * S + (dt[:, None] * X[t])[:, :, None] * B[t][group][:, None, :]
            y[t] = torch.einsum("hpn,hn->hp", S, C[t][group]) + f(d)[:, None] * X[t]
        past = torch.cat([past, f(rows)[at:at + n, inner:inner + CH]])[n:]
        after[slot, :inner * N] = S.reshape(-1)
        after[slot, inner * N:inner * N + (K - 1) * CH] = past.reshape(-1)
        at += n
    used = inner * N + (K - 1) * CH
    return dict(xbc=xbc, rows=rows, dt_bias=dt_bias, a=a, d=d, state=state, seg_start=seg_start, seg_slot=i32(slots), y=y.view(T, inner),
                after=after[:, :used], used=used, inner=inner, CH=CH, dims=dict(heads=H, value_dim=P, states=N, groups=G, taps=K))


def run_ssd(case, kind, **limits):
    from purhie_b200.csrc import ops
    state = case["state"].clone()
    y = torch.full(case["y"].shape, float("nan"), dtype=torch.float32, device=DEV)
    ops.ssd(kind, case["xbc"], case["rows"], case["inner"] + case["CH"], case["inner"], case["dt_bias"], case["a"], case["d"], state,
            case["seg_start"], case["seg_slot"], y, **case["dims"], **limits)
    return y.cpu(), state.cpu()


# states of 1 to 300 with and without whole quads, one lane group and several per lane; values that end inside a block
@pytest.mark.parametrize("H,P,N,G,K", [(6, 32, 40, 2, 4), (6, 10, 6, 3, 1), (2, 64, 128, 1, 4), (3, 5, 33, 3, 6), (2, 72, 300, 2, 3), (1, 7, 1, 1, 2),
                                       (2, 16, 250, 1, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_ssd_scan_token_by_token(H, P, N, G, K, dtype):
    case = ssd_case(H, P, N, G, K, [1, 37, 2, 3, 1], dtype, 10)
    y, state = run_ssd(case, "scan")
    assert rel(y, case["y"]) < 5e-6 and rel(state[:, :case["used"]], case["after"]) < 5e-6


# chunks full and cut, states of 8 to 256, values that end inside a block of 32 and beyond it; decays of a few tokens' reach
@pytest.mark.parametrize("H,P,N,G,K,fast", [(6, 32, 40, 2, 4, False), (2, 64, 128, 1, 4, False), (2, 64, 128, 2, 4, True), (3, 40, 8, 3, 2, False),
                                            (2, 72, 144, 1, 1, False), (1, 8, 256, 1, 3, False), (2, 96, 64, 2, 4, True)])
def test_ssd_chunks_on_the_tensor_cores(H, P, N, G, K, fast):
    from purhie_b200.csrc import ops
    assert ops.ssd_chunk_supports(P, N, G) and not ops.ssd_chunk_supports(P + 1, N, G) and not ops.ssd_chunk_supports(P, 264, G)
    case = ssd_case(H, P, N, G, K, [1, 200, 64, 65, 3, 33], torch.bfloat16, 20, fast)
    y, state = run_ssd(case, "chunk")
    # every float32 factor keeps 16 bits through the tensor cores
    assert rel(y, case["y"]) < 6e-5 and rel(state[:, :case["used"]], case["after"]) < 6e-5
    # the two forms share a step: short portions token by token, long ones in chunks, nobody's state touched twice
    y1, s1 = run_ssd(case, "chunk", rows_from=33)
    long_rows = torch.zeros(case["y"].shape[0], dtype=torch.bool)
    for s, n in enumerate([1, 200, 64, 65, 3, 33]):
        if n >= 33:
            long_rows[int(case["seg_start"][s]):int(case["seg_start"][s + 1])] = True
    assert torch.isnan(y1[~long_rows]).all() and rel(y1[long_rows], case["y"][long_rows]) < 6e-5
    y2, s2 = run_ssd(case, "scan", rows_to=32)
    assert torch.isnan(y2[long_rows]).all() and rel(y2[~long_rows], case["y"][~long_rows]) < 5e-6
    for s, n in enumerate([1, 200, 64, 65, 3, 33]):
        slot = int(case["seg_slot"][s])
        done, kept = (s1, s2) if n >= 33 else (s2, s1)
        assert torch.equal(kept[slot], case["state"][slot].cpu()) and rel(done[slot, :case["used"]], case["after"][slot]) < 6e-5


@pytest.mark.parametrize("T,inner,parts,extra", [(3, 64, 2, 10), (300, 4096, 8, 40), (2, 8192, 1, 0), (5, 60, 4, 7), (4, 30, 30, 2), (260, 12288, 1, 8)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gate_rms_in_parts(T, inner, parts, extra, dtype):
    from purhie_b200.csrc import ops
    y, z, w = rnd(T, inner, seed=1), rnd(T, inner + extra, dtype=dtype, seed=2), rnd(inner, seed=3) + 1.0
    out = torch.full((T, inner), float("nan"), dtype=dtype, device=DEV)
    ops.gate_rms(y, z, w, 1e-4, out, parts=parts)
    g = z.double().cpu()[:, :inner]
    v = (y.double().cpu() * g * torch.sigmoid(g)).view(T, parts, -1)
    ref = (v / torch.sqrt((v * v).mean(-1, keepdim=True) + 1e-4)).view(T, inner) * w.double().cpu()
    assert rel(out.cpu(), ref) < (3e-6 if dtype == torch.float32 else 8e-3)


# ---- a bias linear in the distance -----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype,HQ,HKV,D", [(torch.float32, 5, 1, 24), (torch.bfloat16, 6, 2, 48), (torch.bfloat16, 20, 4, 32)])
def test_a_bias_linear_in_the_distance_in_the_plain_and_the_tile_kernel(dtype, HQ, HKV, D):
    from purhie_b200.csrc import ops
    segs = [(1, 1), (64, 64), (200, 130), (300, 1), (65, 2)]
    case = paged_case(segs, HQ, HKV, D, 16, dtype, seed=4)
    slope = torch.tensor([2.0 ** (-8.0 * (h + 1) / HQ) for h in range(HQ)], dtype=torch.float32, device=DEV)
    sink, scale = torch.zeros(HQ, device=DEV), 1.5 / math.sqrt(D)
    ref, row = torch.zeros(case["T"], HQ, D, dtype=torch.float64), 0
    for (ctx, ql), (k, v) in zip(case["segs"], case["dense"]):
        kk, vv = (t.double().cpu().repeat_interleave(HQ // HKV, dim=1) for t in (k, v))
        for i in range(ql):
            z = ctx - ql + i
            s = torch.einsum("hd,nhd->hn", case["q"][row].double().cpu(), kk[:z + 1]) * scale
            s = s - slope.double().cpu()[:, None] * (z - torch.arange(z + 1)).double()[None]
            e = torch.exp(s)
            ref[row] = torch.einsum("hn,nhd->hd", e / (1.0 + e.sum(1, keepdim=True)), vv[:z + 1])
            row += 1
    ref = ref.view(case["T"], -1)
    kw = dict(num_heads=HQ, num_kv_heads=HKV, head_dim=D, window=None, scale=scale)
    out = torch.full((case["T"], HQ * D), float("nan"), dtype=dtype, device=DEV)
    ops.attention_talking(case["q"], case["k_base"], case["v_base"], case["page_stride"], 16, case["table"], case["row_seg"], case["positions"],
                          out, slope=slope, sink=sink, **kw)
    assert rel(out.cpu(), ref) < (3e-6 if dtype == torch.float32 else 8e-3)
    if dtype == torch.float32:
        return
    tiles = [(s, f) for s, (ctx, ql) in enumerate(segs) for f in range(0, ql, 16)]
    for splits in (1, 3):
        out = torch.full((case["T"], HQ * D), float("nan"), dtype=dtype, device=DEV)
        ops.attention_talking_mma(case["q"], case["k_base"], case["v_base"], case["page_stride"], 16, case["table"], case["seg_start"],
                                  case["seg_ctx"], i32([t[0] for t in tiles]), i32([t[1] for t in tiles]), out, splits=splits, slope=slope,
                                  sink=sink, **kw)
        assert rel(out.cpu(), ref) < 1.2e-2
