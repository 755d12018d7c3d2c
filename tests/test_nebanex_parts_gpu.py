"""The mechanisms of the Nebanex decoder one by one: each part alone against its function of the plain implementation
(`plain_nebanex`), whole, cut into portions down to two tokens, token by token, in batches of unequal requests, and after
slots and pages were freed and taken again.  Where random weights would hide a fault, the weights or inputs are made so that
it shows."""
import numpy as np
import pytest
import torch

import plain_nebanex as P
from test_kedanex_parts_gpu import close
from test_mifolorn_parts_gpu import Harness, under_every_cut
from test_parts_gpu import DTYPES, IDS, bind_random

pytestmark = pytest.mark.gpu
NAMES = {"gate": "gate", "up": "up", "down": "down"}
ATTENTION = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g", "rel": "rel",
             "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b"}


def attention(d, H, G, dk, dv, rows, reach, temp, dtype, scale=None, std=0.25, rel=10.0, prefix="m."):
    """The part with random weights and a distance bias that is not flat; returns (part, precision, weights, mixer config)."""
    from hk_b200.parts import GQAAttention
    from hk_b200.parts.attention import distance_table, padded_head
    scale = dk ** -0.5 if scale is None else scale
    part = GQAAttention(d, H, G, dk, prefix, qk_norm_eps=1e-5, scale=scale, qkv_bias=True, o_bias=True, v_head_dim=dv, gate=True,
                        names=ATTENTION, qk_norm_rows=True, q_factor=temp, bias_max=reach, bias_rows=rows, pad_to=padded_head(dk, dv))
    prec, w = bind_random(part, dtype, std=std)
    w[prefix + "rel"] = w[prefix + "rel"] * rel
    part.dist = distance_table(torch.from_numpy(w[prefix + "rel"]).float().cuda(), reach)
    part.dist_log2 = part.dist * float(np.log2(np.e))
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": scale, "bias_max": reach}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return part, prec, w, m


def gated_linear(d, H, dk, dv, tau, rank, dtype, std=0.3, prefix="m."):
    """The part with random weights whose decays live for tens of tokens, some for one; (part, precision, weights, config)."""
    from hk_b200.parts import GatedLinearAttention
    part = GatedLinearAttention(d, H, dk, dv, tau, prefix, norm_eps=1e-5, decay_rank=rank)
    prec, w = bind_random(part, dtype, std=std)
    with torch.no_grad():
        part.a_bias.mul_(8.0).add_(1.0)
    w[prefix + "a2.b"] = part.a_bias.double().cpu().numpy()
    return part, prec, w, {"heads": H, "dim": dk, "vdim": dv, "tau": tau}


# ------------------------------------------------------------------------------------ attention

SIZES = [
    (40, 6, 2, 10, 6, 6, 20, (0.7, 9)),        # heads filled up to 64
    (48, 4, 4, 24, 72, 10, 50, None),          # values wider than keys, filled up to 128; no factor on the queries
    (32, 4, 2, 16, 16, 8, 40, (0.4, 16)),      # the mma.sync kernels' sizes as they are
    (64, 6, 6, 32, 32, 12, 17, (0.5, 25)),
    (64, 8, 2, 64, 64, 16, 100, (0.5, 40)),    # the tcgen05 and TMA kernels' sizes
    (48, 3, 1, 128, 128, 32, 70, (0.3, 64)),
    (42, 2, 1, 130, 7, 5, 12, (0.2, 1)),       # a head above 128: the generic kernel; a factor that changes at every position
    (32, 1, 1, 5, 13, 2, 3, (-0.3, 7)),
    (32, 20, 1, 16, 16, 1, 3, (0.4, 30)),      # more heads a group than the decode kernels' rows; one row of bias
]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d,H,G,dk,dv,rows,reach,temp", SIZES)
def test_attention_under_every_cut(dtype, d, H, G, dk, dv, rows, reach, temp):
    part, prec, w, m = attention(d, H, G, dk, dv, rows, reach, temp, dtype)
    under_every_cut(part, prec, dtype, {"a": 37, "b": 9, "c": 150}, lambda x: P.attention(x, w, "m.", m, 1e-5))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d,H,G,dk,dv,rows,reach,temp", SIZES)
def test_distance_bias_alone_decides_the_weights(dtype, d, H, G, dk, dv, rows, reach, temp):
    """With scores scaled to nothing the softmax is of the biases alone: every distance up to beyond the table's reach, in
    prompts and in decoding, by its own row (rows of up to several units apart; the gates and biases of the values are off)."""
    part, prec, w, m = attention(d, H, G, dk, dv, rows, reach, temp, dtype, scale=1e-7, rel=12.0)
    under_every_cut(part, prec, dtype, {"a": 130, "b": 21, "c": 2}, lambda x: P.attention(x, w, "m.", m, 1e-5))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("dk,dv", [(64, 64), (128, 128), (16, 16), (12, 20), (130, 8)])
def test_a_far_key_under_the_bias(dtype, dk, dv):
    """One key far back answers the last queries alone (q and k see one input dim that only it and they have), against the
    last row of the bias, which speaks for nearer keys: without the key, or with its bias off by a row, the result moves."""
    d, H, G, T, at = 48, 4, 2, 330, 5
    part, prec, w, m = attention(d, H, G, dk, dv, 8, 60, (0.3, 50), dtype, rel=0.0)
    rel = np.zeros((8, H))
    rel[7] = -1.5 - np.arange(H)                       # the far rows count against the key
    w["m.rel"] = rel
    from hk_b200.parts.attention import distance_table
    part.dist = distance_table(torch.from_numpy(rel).float().cuda(), 60)
    part.dist_log2 = part.dist * float(np.log2(np.e))
    x = torch.randn(T, d, device="cuda") * 0.3
    x[:, 0] = 0
    x[at, 0] = 9.0
    x[T - 40:, 0] = 9.0
    x = x.to(dtype)
    want = P.attention(x.double().cpu().numpy(), w, "m.", m, 1e-5)
    hs = Harness(part, prec, dtype, {"a": x})
    for steps in ([[("a", T)]], [[("a", T - 40)]] + [[("a", 1)]] * 40, [[("a", 7)]] * 47 + [[("a", 1)]]):
        close(hs.run(steps)["a"], want, dtype, str(steps[0]))


@pytest.mark.parametrize("dk,H,G", [(64, 16, 8), (128, 16, 8)])
def test_attention_on_the_tensor_cores_at_length(dk, H, G):
    """2,048 tokens of one request (the tcgen05 kernel with two query tiles per block), with a rest behind a first portion
    (one query tile), and single tokens far in."""
    part, prec, w, m = attention(64, H, G, dk, dk, 32, 700, (0.3, 500), torch.bfloat16)
    x = torch.randn(2048, 64, device="cuda").to(torch.bfloat16)
    want = P.attention(x.double().cpu().numpy(), w, "m.", m, 1e-5)
    hs = Harness(part, prec, torch.bfloat16, {"a": x}, page_tokens=16, pages=200)
    for steps in ([[("a", 2048)]], [[("a", 1024)], [("a", 333)], [("a", 600)]] + [[("a", 1)]] * 20):
        got = hs.run(steps)["a"]
        close(got, want[:len(got)], torch.bfloat16, str(steps[0]))


def test_query_factor_of_the_kernel_with_a_norm_per_head():
    """The same factor behind the per-head norm and rotation kernel, both of its forms."""
    from hk_b200.csrc import ops
    for hd, dtype in ((64, torch.float32), (64, torch.bfloat16), (10, torch.float32), (10, torch.bfloat16)):
        n, H, G = 37, 3, 1
        qkv = torch.randn(n, (H + 2 * G) * hd, device="cuda")
        pos = torch.arange(5, 5 + n, dtype=torch.int32, device="cuda")
        slot = torch.zeros(n, dtype=torch.int32, device="cuda")
        table = torch.arange(16, dtype=torch.int32, device="cuda")[None].contiguous()
        outs = []
        for factor in (None, (0.6, 8)):
            kp, vp = (torch.zeros(16, G, 4, hd, dtype=dtype, device="cuda") for _ in range(2))
            q = torch.empty(n, H * hd, dtype=dtype, device="cuda")
            ops.qk_norm_rope_kv_write(qkv, q, None, None, 0.0, None, None, 0, pos, slot, table, kp, vp, H, G, hd, 4, q_factor=factor)
            outs.append((q.double().cpu().numpy(), kp.double().cpu().numpy()))
        f = P.query_factor(np.arange(5, 5 + n), 0.6, 8)[:, None]
        np.testing.assert_allclose(outs[1][0], outs[0][0] * f, rtol=1e-2 if dtype == torch.bfloat16 else 1e-6, atol=1e-6)
        np.testing.assert_array_equal(outs[0][1], outs[1][1])


# ------------------------------------------------------------------------------------ gated linear attention

LINEAR = [
    (40, 3, 8, 12, 4.0, 5),
    (48, 2, 64, 48, 16.0, 16),
    (32, 1, 128, 72, 5.0, 12),
    (32, 4, 32, 32, 16.0, 16),
    (24, 3, 10, 5, 8.0, 4),          # sizes no vector load divides
    (24, 1, 21, 34, 1.0, 1),         # tau of 1: decays that forget at once
    (24, 2, 200, 6, 2.0, 9),         # keys that end inside a lane's share, above 128
    (24, 1, 264, 3, 3.0, 2),
    (32, 2, 24, 136, 2.0, 3),        # more value columns than a block of the chunked walk; keys that end inside a tile
    (40, 1, 96, 64, 6.0, 4),
]


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d,H,dk,dv,tau,rank", LINEAR)
def test_gated_linear_under_every_cut(dtype, d, H, dk, dv, tau, rank):
    part, prec, w, m = gated_linear(d, H, dk, dv, tau, rank, dtype)
    under_every_cut(part, prec, dtype, {"a": 37, "b": 9, "c": 150}, lambda x: P.gated_linear(x, w, "m.", m, 1e-5))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("dk,dv,tau", [(64, 64, 16.0), (40, 24, 1.0), (128, 40, 0.5)])
def test_gated_linear_long_portions_beside_single_tokens(dtype, dk, dv, tau):
    """Portions of many lengths in one batch with requests that bring a token or two; slots are taken again by the second
    run.  The decays reach from almost none to a channel that is gone after one token."""
    part, prec, w, m = gated_linear(40, 3, dk, dv, tau, 7, dtype)
    with torch.no_grad():
        part.a_bias.copy_(torch.linspace(-60.0, 40.0, part.a_bias.numel(), device="cuda")[torch.randperm(part.a_bias.numel(), device="cuda")])
    w["m.a2.b"] = part.a_bias.double().cpu().numpy()
    lengths = {"a": 260, "b": 150, "c": 40}
    x = {r: torch.randn(n, 40, device="cuda").to(dtype) for r, n in lengths.items()}
    want = {r: P.gated_linear(v.double().cpu().numpy(), w, "m.", m, 1e-5) for r, v in x.items()}
    hs = Harness(part, prec, dtype, x)
    steps = [[("a", 31), ("b", 1)], [("b", 32), ("a", 1), ("c", 2)], [("a", 64), ("c", 1), ("b", 2)], [("b", 65), ("a", 63)],
             [("a", 66), ("b", 33), ("c", 35)], [("a", 2), ("b", 1), ("c", 2)], [("a", 33)], [("b", 16)]]
    long = [[("a", 129), ("c", 1)], [("b", 150), ("a", 131), ("c", 39)]]
    for st in (steps, long, steps):
        got = hs.run(st)
        for r in lengths:
            close(got[r], want[r], dtype, r)


@pytest.mark.parametrize("dk,dv", [(64, 128), (32, 48), (128, 16)])
def test_gated_linear_chunks_of_several_long_requests(dk, dv):
    """Portions of many chunks (more than the carry asks for at once) of three requests in one batch, beside a short one, against
    the walk token by token of the same part."""
    part, prec, w, m = gated_linear(40, 2, dk, dv, 8.0, 6, torch.bfloat16)
    lengths = {"a": 1290, "b": 640, "c": 700}
    x = {r: torch.randn(n, 40, device="cuda").to(torch.bfloat16) for r, n in lengths.items()}
    hs = Harness(part, prec, torch.bfloat16, x)
    steps = [[("a", 1088), ("b", 3), ("c", 65)], [("c", 571), ("a", 1), ("b", 637)], [("a", 201), ("c", 64)]]
    assert part._chunks
    got = hs.run(steps)
    part._chunks = False
    want = hs.run(steps)
    for r in lengths:
        close(got[r], want[r], torch.bfloat16, r)
    plain = P.gated_linear(x["b"].double().cpu().numpy(), w, "m.", m, 1e-5)
    close(got["b"], plain, torch.bfloat16, "plain")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("dk,dv", [(16, 8), (10, 5), (64, 64)])
def test_gated_linear_keeps_what_a_token_wrote_300_tokens_back(dtype, dk, dv):
    """k and q read input dims one to one: position 3 writes into the keys' first half and the last token reads there, every
    other token writes into the second half.  The first half does not decay (its logits stand at 40), the second does: the
    last token's result is what position 3 wrote and its own value.  A state that is lost, cleared or taken from another slot
    gives its own value alone; decays laid out by value channel, or one per head, would forget it."""
    d, H, T, half = max(40, dk + 8), 2, 301, dk // 2
    part, prec, w, m = gated_linear(d, H, dk, dv, 16.0, 3, dtype, std=0.2)
    K, V = H * dk, H * dv
    with torch.no_grad():
        rows = part.in_weight
        rows[:2 * K] = 0
        for h in range(H):
            for i in range(dk):
                rows[h * dk + i, i] = rows[K + h * dk + i, i] = 1.0        # q = k = the first dk inputs
        rows[2 * K:2 * K + V, :dk] = 0                                     # the values do not see the keys' dims
        part.w_a2.zero_()
        part.a_bias.copy_(torch.tensor([40.0] * half + [-20.0] * (dk - half), device="cuda").repeat(H))
    for name, lo, hi in (("q", 0, K), ("k", K, 2 * K), ("v", 2 * K, 2 * K + V)):
        w["m." + name] = rows[lo:hi].double().cpu().numpy()
    w["m.a2"] = np.zeros_like(w["m.a2"])
    w["m.a2.b"] = part.a_bias.double().cpu().numpy()
    x = torch.randn(T, d, device="cuda")
    x[:, :half] = 0
    x[3, :dk] = 0
    x[3, :half] = 2.0 + torch.rand(half, device="cuda")
    x[300, :dk] = x[3, :dk]
    x = x.to(dtype)
    want = P.gated_linear(x.double().cpu().numpy(), w, "m.", m, 1e-5)
    lost = P.gated_linear(x[4:].double().cpu().numpy(), w, "m.", m, 1e-5)
    assert np.abs(want[-1] - lost[-1]).max() > 0.1 * np.abs(want[-1]).max()
    hs = Harness(part, prec, dtype, {"a": x})
    for steps in ([[("a", T)]], [[("a", 290)]] + [[("a", 1)]] * 11, [[("a", 43)]] * 7, [[("a", 1)]] * T):
        got = hs.run(steps)["a"]
        close(got[-1:], want[-1:], dtype, str(steps[0]))


# ------------------------------------------------------------------------------------ the pair, norms, router, soft cap

@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d", [42, 64])
def test_pair_of_mixers_with_normed_results(dtype, d):
    """Both sides at once, with one product for both, the output bias added where the results are normed; and the pair's layer
    norm for the next sublayer beside the sum."""
    from hk_b200.parts import LayerNorm, ParallelMixer, RMSNorm
    left, prec, wl, ml = attention(d, 4, 2, 16, 16, 8, 30, (0.4, 16), dtype, prefix="m.left.")
    right, _, wr, mr = gated_linear(d, 3, 8, 12, 4.0, 5, dtype, prefix="m.right.")
    left_out, right_out = RMSNorm(d, 1e-5, "m.left.out"), RMSNorm(d, 1e-3, "m.right.out")
    norm = LayerNorm(d, 1e-5, "n")
    w = {**wl, **wr}
    for part in (left_out, right_out, norm):
        w.update(bind_random(part, dtype, seed=3, std=0.3)[1])
    pair = ParallelMixer(left, right, 0.5, 0.25, left_out, right_out)
    left.bind = right.bind = left_out.bind = right_out.bind = lambda tensors, precision: None      # bound above, and changed since
    pair.bind({}, prec)

    def plain(x):
        a = P.rms(P.attention(x, w, "m.left.", ml, 1e-5), 1e-5) * w["m.left.out"]
        b = P.rms(P.gated_linear(x, w, "m.right.", mr, 1e-5), 1e-3) * w["m.right.out"]
        return 0.5 * a + 0.25 * b

    assert pair.takes_next_norm(norm) and not pair.takes_next_norm(left_out)
    under_every_cut(pair, prec, dtype, {"a": 33, "b": 8, "c": 70}, plain)
    # a residual stream that is there already, and the next layer norm of the sum
    x = torch.randn(33, d, device="cuda").to(dtype)
    hs = Harness(pair, prec, dtype, {"a": x})
    forward, seen = pair.forward, {}

    def with_next(xb, y, ctx, cache, accumulate):
        y.copy_(torch.arange(y.numel(), device="cuda").reshape(y.shape) % 7 - 3.0)
        seen["out"] = torch.empty_like(xb)
        forward(xb, y, ctx, cache, accumulate=True, next_norm=norm, next_out=seen["out"])

    pair.forward = with_next
    got = hs.run([[("a", 33)]])["a"]
    want = plain(x.double().cpu().numpy()) + np.arange(33 * d).reshape(33, d) % 7 - 3.0
    close(got, want, dtype, "sum")
    close(seen["out"].double().cpu().numpy(), P.layer_norm(want, w["n"], w["n.b"], 1e-5), dtype, "next norm")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("d", [42, 336, 1000, 2050, 4096, 8192, 9000])
def test_layer_norm(dtype, d):
    """Rows far from zero (a mean square less the square of the mean would lose the deviations), with and without a row list."""
    from hk_b200.parts import LayerNorm
    part = LayerNorm(d, 1e-5, "n")
    _, w = bind_random(part, dtype, std=0.5)
    x = torch.randn(9, d, device="cuda") + 300.0 * torch.arange(9, device="cuda")[:, None]
    rows = torch.tensor([4, 0, 8, 8], dtype=torch.int32, device="cuda")
    for r in (None, rows):
        out = torch.empty((9 if r is None else 4, d), dtype=dtype, device="cuda")
        part.forward(x, out, r)
        xs = x.double().cpu().numpy() if r is None else x.double().cpu().numpy()[rows.cpu().numpy()]
        got, want = out.double().cpu().numpy(), P.layer_norm(xs, w["n"], w["n.b"], 1e-5)
        limit = 3e-3 if dtype == torch.float32 else 2e-2        # x itself holds 2400 + deviation to 24 bits
        assert np.abs(got - want).max() <= limit * np.abs(want).max()


@pytest.mark.parametrize("d", [42, 336, 2050, 3072, 8192, 8200])
@pytest.mark.parametrize("bias", [False, True])
def test_pair_norm_add(d, bias):
    from hk_b200.csrc import ops
    g = lambda *s: torch.randn(*s, device="cuda")                            # noqa: E731
    a, b, res, wa, wb, ab, lw, lb = g(5, d), 0.01 * g(5, d), g(5, d), g(d), g(d), 2.0 * g(d), g(d), g(d)
    f = lambda t: t.double().cpu().numpy()                                   # noqa: E731
    want = f(res) + 0.5 * P.rms(f(a) + (f(ab) if bias else 0.0), 1e-3) * f(wa) - 2.0 * P.rms(f(b), 1e-6) * f(wb)
    for dtype in DTYPES:
        r, out = res.clone(), torch.empty(5, d, dtype=dtype, device="cuda")
        ops.pair_norm_add(a, wa, 1e-3, 0.5, b, wb, 1e-6, -2.0, r, a_bias=ab if bias else None, next_norm=(lw, lb, 1e-5), next_out=out)
        close(f(r), want, torch.float32, "sum")
        close(f(out), P.layer_norm(want, f(lw), f(lb), 1e-5), dtype, "norm")
    r = res.clone()
    ops.pair_norm_add(a, wa, 1e-3, 0.5, b, wb, 1e-6, -2.0, r, a_bias=ab if bias else None, accumulate=False)
    close(f(r), want - f(res), torch.float32, "stored")


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("n", [1, 7, 700])
def test_routed_feed_forward_with_a_bias_on_the_router(dtype, n):
    """Biases that turn the choice around, in the weights as well; with and without a shared part; 700 rows take the grouped
    tcgen05 product in bfloat16."""
    from hk_b200.parts import RoutedFeedForward, SwiGLUFeedForward
    d, E, top = 64, 5, 2
    part = RoutedFeedForward(d, 48, E, top, "f.", router_bias=True, shared=SwiGLUFeedForward(d, 72, "f.shared.", names=NAMES))
    prec, w = bind_random(part, dtype, std=0.2)
    with torch.no_grad():
        part.b_router.copy_(torch.tensor([3.0, -3.0, 0.5, 0.0, -9.0], device="cuda"))
    w["f.router.b"] = part.b_router.double().cpu().numpy()
    x = (0.7 * torch.randn(n, d, device="cuda")).to(dtype)
    y = torch.zeros(n, d, device="cuda")
    RoutedFeedForward.route_log = log = []
    try:
        part.forward(x, y, None)
    finally:
        RoutedFeedForward.route_log = None
    xs = x.double().cpu().numpy()
    z = xs @ w["f.router"].T + w["f.router.b"]
    chosen = log[0].cpu().numpy()
    own = [P.route(zz, top) for zz in z]
    clear = np.array([r[2] > 1e-3 for r in own])
    assert (np.sort(chosen, axis=1) == np.sort([r[0] for r in own], axis=1))[clear].all()
    assert (np.sort(chosen, axis=1) != np.sort([P.route(zz - w["f.router.b"], top)[0] for zz in z], axis=1)).any()
    P.route_choices = {"f.": chosen}
    try:
        want = P.routed_feed_forward(xs, w, "f.", {"kind": "moe", "router": {"experts": E, "top": top}, "shared": {"ff": 72}})
    finally:
        P.route_choices = None
    close(y.double().cpu().numpy(), want, dtype, "routed")


def test_soft_cap_of_the_logits():
    from hk_b200.csrc import ops
    x = torch.randn(3, 1001, device="cuda") * 20
    want = P.soft_cap(x.double().cpu().numpy(), 7.5)
    ops.soft_cap(x, 7.5)
    np.testing.assert_allclose(x.double().cpu().numpy(), want, rtol=2e-6, atol=1e-6)
