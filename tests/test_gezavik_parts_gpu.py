"""The mechanisms of the Gezavik decoder one by one: each part alone against its function of the plain implementation
(`plain_gezavik`), whole, cut into portions down to two tokens, token by token, in batches of unequal requests, and after
slots and pages were freed and taken again.  Where random weights would hide a fault, the weights or inputs are made so that
it shows."""
import numpy as np
import pytest
import torch

import plain_gezavik as P
from test_kedanex_parts_gpu import close
from test_mifolorn_parts_gpu import Harness, under_every_cut
from test_parts_gpu import DTYPES, IDS, bind_random

pytestmark = pytest.mark.gpu
NAMES = {"gate": "gate", "up": "up", "down": "down"}


def to_bfloat16(x):
    return torch.from_numpy(np.ascontiguousarray(x)).to(torch.bfloat16).double().numpy()


# ------------------------------------------------------------------------------------ the state-space mixer

def state_space(d, H, dv, N, G, taps, parts, dtype, std=0.3):
    """The part with random weights whose decays live for tens of tokens; returns (part, precision, weights, mixer config)."""
    from hk_b200.parts import StateSpace
    part = StateSpace(d, H, dv, N, G, taps, "m.", 1e-5, norm_groups=parts)
    prec, w = bind_random(part, dtype, std=std)
    with torch.no_grad():
        part.a_log.sub_(2.0)
        part.dt_bias.sub_(0.5)
    w["m.A_log"] = part.a_log.double().cpu().numpy()
    w["m.dt_bias"] = part.dt_bias.double().cpu().numpy()
    return part, prec, w, {"heads": H, "vdim": dv, "state": N, "groups": G, "conv": taps, "norm_groups": parts}


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d,H,dv,N,G,taps,parts", [
    (40, 6, 8, 16, 3, 3, 4),         # the norm's parts cut across heads
    (48, 4, 64, 128, 2, 4, 2),       # the chunked walk's common sizes
    (32, 3, 40, 64, 1, 2, 3),        # value columns that end inside a block of the chunked walk
    (32, 2, 72, 32, 2, 5, 1),        # more value columns than a block
    (24, 2, 16, 200, 1, 3, 2),       # states that end inside a tile, above 128
    (24, 2, 8, 24, 1, 1, 8),         # one tap
    (40, 3, 5, 10, 3, 6, 5),         # sizes no vector load divides: token by token
    (24, 1, 12, 264, 1, 4, 1),       # a state larger than the chunked walk takes
])
def test_state_space_under_every_cut(dtype, d, H, dv, N, G, taps, parts):
    part, prec, w, m = state_space(d, H, dv, N, G, taps, parts, dtype)
    under_every_cut(part, prec, dtype, {"a": 37, "b": 9, "c": 150}, lambda x: P.mamba2(x, w, "m.", m, 1e-5))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_state_space_long_portions_beside_single_tokens(dtype):
    """Portions around the length from which a request is walked in chunks and around a chunk's edge, in one batch with
    requests that bring a token or two; slots are taken again by the second run."""
    part, prec, w, m = state_space(40, 4, 24, 48, 2, 4, 2, dtype)
    lengths = {"a": 260, "b": 150, "c": 40}
    x = {r: torch.randn(n, 40, device="cuda").to(dtype) for r, n in lengths.items()}
    want = {r: P.mamba2(v.double().cpu().numpy(), w, "m.", m, 1e-5) for r, v in x.items()}
    hs = Harness(part, prec, dtype, x)
    steps = [[("a", 31), ("b", 1)], [("b", 32), ("a", 1), ("c", 2)], [("a", 64), ("c", 1), ("b", 2)], [("b", 65), ("a", 63)],
             [("a", 66), ("b", 33), ("c", 35)], [("a", 2), ("b", 1), ("c", 2)], [("a", 33)], [("b", 16)]]
    for _ in range(2):
        got = hs.run(steps)
        for r in lengths:
            close(got[r], want[r], dtype, r)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("N,dv", [(16, 8), (10, 5)])
def test_state_space_keeps_what_a_token_wrote_300_tokens_back(dtype, N, dv):
    """B and C read input dims one to one: position 3 writes into the state's first half and the last token reads there,
    every other token writes into the second half.  Nothing decays (A_log = -30), the skip is zero and the gate's logit is
    read from one input that is 4 for every token: the last token's result is what position 3 wrote and its own value.  A
    state that is lost, cleared or taken from another slot gives its own value alone."""
    d, H, G, taps, T = 40, 2, 1, 2, 301
    part, prec, w, m = state_space(d, H, dv, N, G, taps, 1, dtype, std=0.2)
    inner, half = H * dv, N // 2
    with torch.no_grad():
        rows = part.w_in[:2 * inner + 2 * N + H]
        rows[:inner] = 0
        rows[:inner, d - 1] = 1.0                                             # z = 4
        rows[inner:2 * inner, :N] = 0                                         # x does not see the key's dims
        rows[2 * inner:2 * inner + N] = 0
        rows[2 * inner + N:2 * inner + 2 * N] = 0
        for i in range(N):
            rows[2 * inner + i, i] = rows[2 * inner + N + i, i] = 1.0         # B = C = the first N inputs (then silu)
        rows[2 * inner + 2 * N:] = 0                                          # dt = softplus(dt_bias)
        w["m.in"] = rows.double().cpu().numpy()
        part.conv.weight.zero_()
        part.conv.weight[:, -1] = 1.0
        part.conv.bias.zero_()
        part.a_log.fill_(-30.0)
        part.skip.zero_()
    w["m.conv"] = part.conv.weight.double().cpu().numpy()
    w["m.conv.b"] = np.zeros_like(w["m.conv.b"])
    w["m.A_log"] = np.full(H, -30.0)
    w["m.D"] = np.zeros(H)
    x = torch.randn(T, d, device="cuda")
    x[:, d - 1] = 4.0
    x[:, :half] = 0
    x[3, :N] = 0
    x[3, :half] = 2.0 + torch.rand(half, device="cuda")
    x[300, :N] = x[3, :N]
    x = x.to(dtype)
    want = P.mamba2(x.double().cpu().numpy(), w, "m.", m, 1e-5)
    lost = P.mamba2(x[4:].double().cpu().numpy(), w, "m.", m, 1e-5)
    assert np.abs(want[-1] - lost[-1]).max() > 0.1 * np.abs(want[-1]).max()
    hs = Harness(part, prec, dtype, {"a": x})
    for steps in ([[("a", T)]], [[("a", 290)]] + [[("a", 1)]] * 11, [[("a", 2)], [("a", 150)], [("a", 147)], [("a", 2)]]):
        close(hs.run(steps)["a"][-3:], want[-3:], dtype, "far write")


def walk_in_double(xbc, dt, dt_bias, a_log, skip, S, H, G, N, dv):
    """The recurrence over one request's rows in float64 on the device, all heads at once; S [H, dv, N]."""
    T, inner = xbc.shape[0], H * dv
    x = xbc[:, :inner].double().view(T, H, dv)
    B, C = (xbc[:, inner + k * G * N:inner + (k + 1) * G * N].double().view(T, G, N).repeat_interleave(H // G, 1) for k in (0, 1))
    step = torch.nn.functional.softplus(dt.double() + dt_bias.double())
    decay = torch.exp(-torch.exp(a_log.double()) * step)
    S, out = S.double().clone(), []
    for t in range(T):
        S = decay[t][:, None, None] * S + x[t][:, :, None] * (step[t][:, None] * B[t])[:, None, :]
        out.append((S @ C[t][:, :, None])[:, :, 0] + skip.double()[:, None] * x[t])
    return torch.stack(out).view(T, inner), S


@pytest.mark.parametrize("H,G,N,dv", [(4, 2, 128, 64), (4, 1, 32, 32), (6, 3, 64, 24), (2, 1, 256, 64), (2, 2, 16, 8), (3, 1, 40, 72), (150, 1, 128, 64)])
@pytest.mark.parametrize("step_shift", [-5.0, -1.0, 2.0], ids=["slow", "middle", "fast"])
def test_chunked_walk_is_the_token_walk_in_32_bit(H, G, N, dv, step_shift):
    """The two forms over the same bfloat16 rows from a state that is not zero, requests whose lengths end inside, at and
    just behind a chunk's edge, in slots of another order: both within float32 rounding of the float64 recurrence, outputs
    and states, with decays that forget within a token and with decays that last."""
    from hk_b200.csrc import ops
    lens = [100, 64, 33, 5, 1, 129]
    n, inner = sum(lens), H * dv
    C = inner + 2 * G * N
    wide = (torch.randn(n, C + 8, device="cuda") * 0.7).bfloat16()
    xbc = wide[:, :C]
    dt = torch.randn(n, H + 3, device="cuda")[:, 1:1 + H]
    dt_bias, a_log, skip = (torch.randn(H, device="cuda") * 0.5 for _ in range(3))
    dt_bias += step_shift
    start = torch.randn(len(lens) + 1, H, dv, N, device="cuda") * 0.3
    at = np.concatenate([[0], np.cumsum(lens)])
    segs = torch.tensor([[len(lens) - i, int(at[i]), l] for i, l in enumerate(lens)], dtype=torch.int32, device="cuda")
    for chunked in (True, False):
        state, y = start.clone(), torch.full((n, inner), float("nan"), device="cuda")
        ops.state_space_scan(xbc, dt, dt_bias, a_log, skip, segs[:0] if chunked else segs, state, y, H, G, N, dv,
                             long_segments=segs if chunked else None)
        for slot, r0, l in segs.tolist():
            want, S = walk_in_double(xbc[r0:r0 + l], dt[r0:r0 + l], dt_bias, a_log, skip, start[slot], H, G, N, dv)
            limit = 3e-5 if chunked else 3e-6      # a chunk's cumulative log decay is a float32 number of its own size
            assert (y[r0:r0 + l] - want).abs().max() <= limit * want.abs().max(), (chunked, l)
            assert (state[slot] - S).abs().max() <= limit * S.abs().max(), (chunked, l)
        assert torch.equal(state[0], start[0])     # the slot of no request


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("H,G,N,dv", [(4, 2, 128, 64), (3, 1, 32, 20), (2, 2, 64, 5), (2, 1, 200, 8), (1, 1, 300, 12), (1, 1, 516, 8), (100, 1, 16, 64)])
def test_single_token_steps_equal_the_walk_bit_for_bit(dtype, H, G, N, dv):
    """A step of single tokens runs a kernel of its own; beside one portion of two tokens the same requests go through the
    ring.  Logits may not depend on which."""
    from hk_b200.csrc import ops
    reqs, inner = 5, H * dv
    C = inner + 2 * G * N
    xbc = (torch.randn(reqs + 2, C, device="cuda") * 0.7).to(dtype)
    dt = torch.randn(reqs + 2, H, device="cuda")
    dt_bias, a_log, skip = (torch.randn(H, device="cuda") * 0.5 for _ in range(3))
    start = torch.randn(reqs + 1, H, dv, N, device="cuda")
    segs = torch.tensor([[reqs - i, i, 1] for i in range(reqs)] + [[0, reqs, 2]], dtype=torch.int32, device="cuda")
    alone, beside = start.clone(), start.clone()
    y1, y2 = torch.full((reqs, inner), float("nan"), device="cuda"), torch.full((reqs + 2, inner), float("nan"), device="cuda")
    ops.state_space_scan(xbc[:reqs], dt[:reqs], dt_bias, a_log, skip, segs[:reqs].contiguous(), alone, y1, H, G, N, dv)
    ops.state_space_scan(xbc, dt, dt_bias, a_log, skip, segs, beside, y2, H, G, N, dv)
    assert torch.equal(y1, y2[:reqs]) and torch.equal(alone[1:], beside[1:]) and torch.equal(alone[0], start[0])
    for slot, r0, l in segs.tolist():
        want, S = walk_in_double(xbc[r0:r0 + l], dt[r0:r0 + l], dt_bias, a_log, skip, start[slot], H, G, N, dv)
        assert (y2[r0:r0 + l] - want).abs().max() <= 3e-6 * want.abs().max() and (beside[slot] - S).abs().max() <= 3e-6 * S.abs().max()


# ------------------------------------------------------------------------------------ latent attention

def latent_part(d, H, dn, dr, vd, qr, r, rot, window, scale, positions=512):
    from hk_b200.parts import LatentAttention, RotaryEmbedding
    pos = RotaryEmbedding(rot["base"], rot["dims"], positions, pairing="adjacent")
    part = LatentAttention(d, H, dn, dr, vd, r, "m.", 1e-5, scale, position=pos, gate="head", window=window, q_rank=qr)
    m = {"heads": H, "dim": dn, "rot_dim": dr, "vdim": vd, "q_rank": qr, "kv_rank": r, "scale": scale, "rot": rot}
    if window:
        m["mask"] = {"size": window}
    return part, m


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d,H,dn,dr,vd,qr,r,window", [
    (40, 3, 8, 4, 12, 20, 12, 7), (64, 8, 32, 16, 48, 72, 48, 37), (48, 2, 16, 6, 24, 32, 20, 33), (40, 5, 6, 2, 10, 11, 10, None),
    (64, 4, 16, 16, 40, 56, 128, 21), (32, 1, 8, 8, 5, 16, 24, 2), (48, 6, 24, 32, 16, 40, 64, 50)])
def test_latent_attention_with_a_query_latent_and_head_gates(dtype, d, H, dn, dr, vd, qr, r, window):
    """Sharp scores, so that a token's result hangs on few keys: a window that is one token off shows at every token whose
    strongest key lies at the window's edge, which the test first makes sure of."""
    part, m = latent_part(d, H, dn, dr, vd, qr, r, {"base": 500.0, "dims": dr}, window, 5.0 / (dn + dr))
    prec, w = bind_random(part, dtype, std=0.35)
    if window:
        x = np.random.default_rng(0).standard_normal((90, d))
        base = P.latent_attention(x, w, "m.", m, 1e-5)
        for other in (window - 1, window + 1):
            off = P.latent_attention(x, w, "m.", dict(m, mask={"size": max(other, 1)}), 1e-5)
            assert (np.abs(off - base).max(axis=1) > 0.05 * np.abs(base).max()).sum() >= 3
    under_every_cut(part, prec, dtype, {"a": 37, "b": 9, "c": 90}, lambda x: P.latent_attention(x, w, "m.", m, 1e-5))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("r,dr", [(48, 16), (12, 4), (20, 6)])
def test_latent_attention_finds_keys_at_the_edges_of_pages_and_of_the_window(dtype, r, dr):
    """The query latent of a marked token is ten times as large as the others' key parts make it: input dim 0 marks.  Keys at
    positions that are a page's last and first row and just inside the window stand out for the last tokens; without them,
    or with the one just outside, the result is another one."""
    d, H, dn, vd, qr, T, window = 32, 2, 16, 12, 24, 420, 200
    part, m = latent_part(d, H, dn, dr, vd, qr, r, {"base": 1e6, "dims": 2}, window, 1.0 / dn)
    prec, w = bind_random(part, dtype, std=0.3)
    x = torch.randn(T, d, device="cuda") * 0.5
    marks = (T - window, T - window + 1, 239, 240)                # just outside and just inside for the last token; a page's edge
    with torch.no_grad():                                          # every query and the marked keys point the same way
        x[:, 0] = 1.0
        x[list(marks), 1] = 6.0
    x = x.to(dtype)
    xs = x.double().cpu().numpy()
    want = P.latent_attention(xs, w, "m.", m, 1e-5)
    moved = 0
    for p in marks[1:]:
        other = xs.copy()
        other[p] = np.random.default_rng(p).standard_normal(d)
        moved += np.abs(P.latent_attention(other, w, "m.", m, 1e-5)[-1] - want[-1]).max() > 0.004 * np.abs(want[-1]).max()
    assert moved >= 2
    other = xs.copy()
    other[T - window - 1] += 50.0                                  # outside the last token's window
    np.testing.assert_allclose(P.latent_attention(other, w, "m.", m, 1e-5)[-1], want[-1])
    hs = Harness(part, prec, dtype, {"a": x}, page_tokens=16)
    for steps in ([[("a", T)]], [[("a", T - 11)]] + [[("a", 1)]] * 11, [[("a", 2)], [("a", 250)], [("a", 165)], [("a", 2)], [("a", 1)]]):
        close(hs.run(steps)["a"][-12:], want[-12:], dtype, "far keys")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_out_scale_rides_on_each_sublayer(dtype):
    """A factor on the result of every sublayer that a parallel block may give one to."""
    from hk_b200.parts import RoutedFeedForward, SquaredReLUFeedForward, SwiGLUFeedForward
    d, rows, s = 48, 20, 0.3
    x = torch.randn(rows, d, device="cuda").to(dtype)
    xs = x.double().cpu().numpy()

    def check(make, run, plain):
        part = make()
        part.out_scale = s
        prec, w = bind_random(part, dtype, std=0.25)
        close(run(part, prec), s * plain(w), dtype, type(part).__name__)

    mix = lambda part, prec: Harness(part, prec, dtype, {"a": x}).run([[("a", rows)]])["a"]

    def ff(part, prec):
        y = torch.full((rows, d), 0.5, device="cuda")
        part.forward(x, y, None, accumulate=True)
        return y.double().cpu().numpy() - 0.5

    from hk_b200.parts import StateSpace
    m = {"heads": 3, "vdim": 8, "state": 16, "groups": 1, "conv": 2, "norm_groups": 2}
    check(lambda: StateSpace(d, 3, 8, 16, 1, 2, "m.", 1e-5, norm_groups=2), mix, lambda w: P.mamba2(xs, w, "m.", m, 1e-5))
    made = {}

    def latent():
        part, made["m"] = latent_part(d, 2, 8, 4, 12, 20, 12, {"base": 100.0, "dims": 4}, 9, 0.3)
        return part

    check(latent, mix, lambda w: P.latent_attention(xs, w, "m.", made["m"], 1e-5))
    check(lambda: SquaredReLUFeedForward(d, 40, "f."), ff, lambda w: P.squared_relu_feed_forward(xs, w, "f."))
    mlp = {"kind": "moe", "expert": {"ff": 24, "limit": 0.9}, "router": {"experts": 3, "identity": 1, "top": 4}, "shared": {"ff": 16, "limit": 0.7}}
    check(lambda: RoutedFeedForward(d, 24, 3, 4, "f.", scores="softmax_all", correction=True, identity=1, act="swish_clamped", limit=0.9,
                                    slope=1.702, shared=SwiGLUFeedForward(d, 16, "f.shared.", act="swish_clamped", names=NAMES, limit=0.7, slope=1.702)),
          ff, lambda w: P.routed_feed_forward(xs, w, "f.", mlp))


# ------------------------------------------------------------------------------------ the block

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("scale", [0.4, 1.0, -0.7])
@pytest.mark.parametrize("carried", [True, False])
def test_parallel_block(dtype, scale, carried):
    """One norm, both sublayers on its output, their sum times a factor onto the stream: carried by the sublayers, and
    through a buffer where one of them cannot carry it."""
    from hk_b200.cache.device import PagedCache
    from hk_b200.parts import ParallelBlock, RMSNorm, SquaredReLUFeedForward, StateSpace, SwiGLUFeedForward
    from test_parts_gpu import make_ctx
    d, rows = 40, 50
    mixer = StateSpace(d, 2, 8, 16, 1, 3, "m.", 1e-5)
    ffn = SquaredReLUFeedForward(d, 56, "f.") if carried else SwiGLUFeedForward(d, 56, "f.", act="swish_clamped", names=NAMES, limit=0.8, slope=1.702)
    block = ParallelBlock(RMSNorm(d, 1e-5, "n"), mixer, ffn, scale)
    assert block._carried == (carried or scale == 1.0)
    prec, w = bind_random(block, dtype, std=0.25)
    cache = PagedCache([block.cache_specs()], prec, 8, 16, 2, 128)
    x = torch.randn(rows, d, device="cuda")
    ctx = make_ctx(prec, [(cache.open(), 0, rows)], cache, part=block)
    got = x.clone()
    block.forward(got, ctx, cache.layers[0])
    xs = x.double().cpu().numpy()
    h = P.rms(xs, 1e-5) * w["n"]
    if dtype == torch.bfloat16:
        h = to_bfloat16(h)
    ff = P.squared_relu_feed_forward(h, w, "f.") if carried else P.clamped_feed_forward(h, w, "f.", 0.8)
    m = {"heads": 2, "vdim": 8, "state": 16, "groups": 1, "conv": 3, "norm_groups": 1}
    close(got.double().cpu().numpy() - xs, scale * (P.mamba2(h, w, "m.", m, 1e-5) + ff), dtype, "block")


# ------------------------------------------------------------------------------------ short convolution with a bias

@pytest.mark.parametrize("taps", [1, 2, 4, 5, 9])
@pytest.mark.parametrize("out", [torch.float32, torch.bfloat16], ids=IDS)
def test_short_convolution_with_a_bias_across_the_edges_of_portions(taps, out):
    from hk_b200.csrc import ops
    C = 37
    wt, bias = torch.randn(C, taps, device="cuda"), torch.randn(C, device="cuda")
    counts = (1, 2, 1, 6, 2, 70, 1, 1, 33)
    x = torch.randn(sum(counts), C + 3, device="cuda")
    tail = torch.zeros(2, max(taps - 1, 1), C, device="cuda")
    got, p = [], 0
    for c in counts:
        y = torch.full((c, C + 2), float("nan"), dtype=out, device="cuda")
        ops.short_conv(x[p:p + c, 1:1 + C], wt, torch.tensor([[1, 0, c]], dtype=torch.int32, device="cuda"), tail, y[:, :C], act="silu", bias=bias)
        assert torch.isnan(y[:, C:]).all()
        got.append(y[:, :C])
        p += c
    want = P.silu(P.short_conv(x[:, 1:1 + C].double().cpu().numpy(), wt.double().cpu().numpy(), bias.double().cpu().numpy()))
    tol = 1e-5 if out == torch.float32 else 5e-3
    np.testing.assert_allclose(torch.cat(got).double().cpu().numpy(), want, rtol=tol, atol=tol)
    assert torch.all(tail[0] == 0.0)


# ------------------------------------------------------------------------------------ feed-forwards

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d,F,rows", [(40, 52, 9), (64, 160, 70), (128, 320, 300), (128, 320, 12), (192, 256, 5), (256, 1024, 2048), (44, 30, 33)])
def test_squared_relu_feed_forward(dtype, d, F, rows):
    """Rows and sizes that reach every kernel with the activation in its epilogue (the streaming products, the tcgen05 product
    with and without K slices) and the activation's own kernel."""
    from hk_b200.parts import SquaredReLUFeedForward
    part = SquaredReLUFeedForward(d, F, "f.")
    prec, w = bind_random(part, dtype, std=0.2)
    x = (torch.randn(rows, d, device="cuda") * 1.2).to(dtype)
    y = torch.zeros(rows, d, device="cuda")
    part.forward(x, y, None, accumulate=False)
    close(y.double().cpu().numpy(), P.squared_relu_feed_forward(x.double().cpu().numpy(), w, "f."), dtype, "squared relu")


@pytest.mark.parametrize("gemm", ["tc", "stream", "smallm", "generic"])
def test_squared_relu_epilogues_one_by_one(gemm):
    from hk_b200.csrc import ops
    sizes = [(5, 200, 128), (16, 96, 320)]
    sizes += {"stream": [(30, 5000, 192)], "smallm": [(30, 333, 192), (60, 77, 136)]}.get(gemm, [(30, 333, 192), (300, 520, 136)])
    for M, N, K in sizes:
        a, w = (torch.randn(M, K, device="cuda")).bfloat16(), (torch.randn(N, K, device="cuda") * 0.1).bfloat16()
        out = torch.full((M, N), float("nan"), dtype=torch.bfloat16, device="cuda")
        with ops.force(gemm=gemm):
            ops.gemm_squared_relu(a, w, out, 0.5)
        want = 0.5 * torch.relu(a.double() @ w.double().T) ** 2
        assert (out.double() - want).abs().max() <= 6e-3 * want.abs().max(), (gemm, M, N, K)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d,F,E,ident,top,limit,shared,rows", [
    (40, 12, 5, 1, 2, 0.7, (20, 1.1), 33),
    (48, 24, 3, 4, 4, 0.9, None, 57),              # more identities than experts
    (64, 32, 9, 0, 3, 1.5, (48, 0.5), 300),        # no identities; prompt-sized rows
    (32, 16, 2, 2, 4, 0.6, (24, 0.8), 20),         # everything chosen
    (128, 64, 8, 2, 2, 0.8, (96, 1.3), 600),       # the grouped tcgen05 product's sizes
    (44, 10, 40, 9, 6, 1.0, None, 90),             # more outputs than a warp has lanes
    (32, 8, 1, 1, 1, 0.5, (8, 0.5), 65),           # one expert, one identity, one choice
])
def test_softmax_router_with_identities_and_clamped_experts(dtype, d, F, E, ident, top, limit, shared, rows):
    from hk_b200.parts import RoutedFeedForward, SwiGLUFeedForward
    sh = SwiGLUFeedForward(d, shared[0], "f.shared.", act="swish_clamped", names=NAMES, limit=shared[1], slope=1.702) if shared else None
    part = RoutedFeedForward(d, F, E, top, "f.", scores="softmax_all", correction=True, identity=ident, act="swish_clamped", limit=limit,
                             slope=1.702, shared=sh)
    prec, w = bind_random(part, dtype, std=0.2)
    x = torch.randn(rows, d, device="cuda").to(dtype)
    xs = x.double().cpu().numpy()
    mlp = {"kind": "moe", "expert": {"ff": F, "limit": limit}, "router": {"experts": E, "identity": ident, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared[0], "limit": shared[1]}
    RoutedFeedForward.route_log = log = []
    try:
        y = torch.zeros(rows, d, device="cuda")
        part.forward(x, y, None, accumulate=False)
    finally:
        RoutedFeedForward.route_log = None
    ids = log[0].cpu().numpy()
    free = [P.route(xs[t] @ w["f.router"].T, w["f.correction"], top) for t in range(rows)]
    own, margins = np.asarray([f[0] for f in free]), np.asarray([f[2] for f in free])
    clear = margins >= (1e-5 if dtype == torch.float32 else 5e-3)
    assert clear.mean() > 0.5
    assert (np.sort(own[clear], axis=1) == np.sort(ids[clear], axis=1)).all()
    if ident and top < E + ident:
        plain_choice = np.asarray([P.route(xs[t] @ w["f.router"].T, np.zeros(E + ident), top)[0] for t in range(rows)])
        assert (np.sort(plain_choice, axis=1) != np.sort(own, axis=1)).any()          # the correction matters
    if ident:
        assert (own >= E).any() and (own < E).any()
    P.route_choices = {"f.": ids}
    try:
        want = P.routed_feed_forward(xs, w, "f.", mlp)
    finally:
        P.route_choices = None
    close(y.double().cpu().numpy(), want, dtype, "routed")


def test_routed_feed_forward_whose_tokens_all_choose_identities():
    """No expert has a row: the grouped products run over nothing, in the decode-sized and in the prompt-sized form."""
    from hk_b200.parts import RoutedFeedForward
    d, E, ident, top = 64, 4, 3, 2
    part = RoutedFeedForward(d, 32, E, top, "f.", scores="softmax_all", correction=True, identity=ident, act="swish_clamped", limit=1.0, slope=1.702)
    prec, w = bind_random(part, torch.bfloat16, std=0.2)
    with torch.no_grad():
        part.w_correction[:E] = -5.0
    for rows in (7, 700):
        x = torch.randn(rows, d, device="cuda").bfloat16()
        y = torch.zeros(rows, d, device="cuda")
        part.forward(x, y, None, accumulate=False)
        z = x.double() @ torch.from_numpy(w["f.router"]).cuda().T
        s = torch.softmax(z, dim=1)
        choice = (s + part.w_correction.double()).topk(top, dim=1).indices
        assert (choice >= E).all()
        want = s.gather(1, choice).sum(dim=1, keepdim=True) * x.double()
        assert (y - want).abs().max() <= 1e-3 * want.abs().max()
