"""The kernels of the recurrent layers, the experts, the windowed attention and the two-sided norm (include/l3ci_mixers.h), each
against the plain float64 restatement in oracle/rupotar.py."""
import pytest
import torch

from oracle import rupotar as ref

pytestmark = pytest.mark.gpu
BF16, F32, F64 = torch.bfloat16, torch.float32, torch.float64
DTYPES = (BF16, F32)


def rand(*shape, seed=0, scale=1.0, dtype=BF16):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def close(got, want, dtype, what="", bound=None):
    """Relative L2 per row of the last axis, rounding of the type only."""
    got, want = got.double().cpu(), want.double()
    assert torch.isfinite(got).all(), what
    rel = (got - want).norm(dim=-1) / (want.norm(dim=-1) + 1e-3 * want.abs().max() + 1e-30)
    bound = bound or (1.2e-2 if dtype == BF16 else 2e-5)
    assert rel.max().item() < bound, f"{what}: {rel.max().item()} at {rel.argmax().item()} of {tuple(rel.shape)}"


def at(device, *positions):
    return torch.tensor(positions, dtype=torch.int32, device=device)


# ---- windowed attention with a distance bias and a sink ------------------------------------------------------------------
def attend(pkg, device, dtype, variant, T, pos, H, G, D, V, window, keep, bias, sink, seed=0, fill=float("nan"), boost=()):
    """T queries per sequence behind positions `pos`; `boost`: (query token, key position) pairs whose score stands out."""
    B, L = len(pos), max(pos) + T + 3
    q, k, v = rand(B, T, H, D, seed=seed, dtype=dtype), rand(B, L, G, D, seed=seed + 1, dtype=dtype), rand(B, L, G, V, seed=seed + 2, dtype=dtype)
    for t, j in boost:
        k[:, j] = q[:, t, ::H // G] * 2
    scale = D ** -0.5
    dk, dv = k.to(device), v.to(device)
    for b, p in enumerate(pos):
        dk[b, p + T:], dv[b, p + T:] = fill, fill                       # what an earlier request left is never read
    out = torch.empty(B, T, H, V, dtype=dtype, device=device)
    start = pos[0] if len(set(pos)) == 1 and T > 1 else -1
    pkg.mixers.attention(q.to(device), dk, dv, out, at(device, *pos), scale=scale, start_pos=start, variant=variant, window=window,
                         keep_first=keep, bias_range=bias, sink=sink)
    want = []
    for b, p in enumerate(pos):
        S = p + T
        if bias == 8.0 and sink:
            want.append(ref.attention(q[b].double(), k[b, :S].double(), v[b, :S].double(), scale, window or None, keep))
            continue
        i, j = torch.arange(p, S)[:, None], torch.arange(S)[None, :]
        seen = (j <= i) & ((i - j < window) | (j < keep) if window else True)
        o = torch.zeros(T, H, V, dtype=F64)
        for h in range(H):
            s = q[b, :, h].double() @ k[b, :S, h // (H // G)].double().T * scale
            s = s - (2.0 ** (-bias * (h + 1) / H) * (i - j) if bias else 0)
            w = ref.sink_softmax(s, seen) if sink else torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
            o[:, h] = w @ v[b, :S, h // (H // G)].double()
        want.append(o)
    return out, torch.stack(want)


SIZES = [(8, 2, 64, 96), (4, 4, 128, 128), (6, 2, 16, 24), (16, 1, 80, 64)]
WINDOWS = [(0, 0), (1, 0), (40, 6), (64, 64), (130, 1), (65, 130), (5000, 3)]


@pytest.mark.parametrize("window,keep", WINDOWS)
@pytest.mark.parametrize("H,G,D,V", SIZES)
def test_attention_variants(pkg, device, H, G, D, V, window, keep):
    for variant, T, pos in ((1, 1, (0, 5, 333)), (1, 9, (200,)), (2, 1, (0, 63, 64, 700)), (2, 7, (150,)), (2, 100, (0,)), (2, 33, (318,)),
                            (3, 128, (0,)), (3, 300, (0,)), (3, 130, (257,)), (3, 140, (55,)), (0, 1, (299,)), (0, 200, (64,))):
        got, want = attend(pkg, device, BF16, variant, T, pos, H, G, D, V, window, keep, 8.0, True, seed=T)
        close(got, want, BF16, (variant, T, pos), bound=2e-2)
    for T, pos in ((1, (0, 70, 290)), (50, (100,)), (130, (0,))):
        got, want = attend(pkg, device, F32, 0, T, pos, H, G, D, V, window, keep, 8.0, True, seed=T)
        close(got, want, F32, (T, pos))


@pytest.mark.parametrize("bias,sink", [(0.0, False), (0.0, True), (8.0, False), (3.5, True)])
def test_bias_and_sink_are_separate(pkg, device, bias, sink):
    for variant, T, pos in ((1, 3, (50,)), (2, 1, (0, 200)), (2, 20, (100,)), (3, 150, (70,))):
        got, want = attend(pkg, device, BF16, variant, T, pos, 4, 2, 64, 64, 90, 4, bias, sink)
        close(got, want, BF16, (variant, T), bound=2e-2)


def test_single_keys_at_the_window_borders(pkg, device):
    """A key that carries the row's weight, moved over every border of window, kept tokens and tiles."""
    for variant, T, p in ((1, 1, 300), (2, 1, 300), (2, 40, 261), (3, 172, 129)):
        t = T - 1
        for window, keep in ((70, 20), (128, 64), (129, 0)):
            i = p + t
            for j in sorted({0, keep - 1, keep, keep + 1, i - window - 1, i - window, i - window + 1, i - 64, i - 1, i, 127, 128, 255, 256}):
                if 0 <= j <= i:
                    got, want = attend(pkg, device, BF16, variant, T, (p,), 4, 2, 64, 64, window, keep, 8.0, True, seed=j, boost=[(t, j)])
                    close(got, want, BF16, (variant, window, keep, j), bound=2e-2)


def test_a_sink_swallows_rows_of_low_scores(pkg, device):
    B, T, H, D = 1, 140, 2, 64
    for dtype, variant in ((F32, 1), (BF16, 1), (BF16, 2), (BF16, 3)):
        q = torch.full((B, T, H, D), 4.0, dtype=dtype, device=device)
        out = torch.full((B, T, H, D), 9.0, dtype=dtype, device=device)
        v = torch.ones(B, T, H, D, dtype=dtype, device=device)
        pkg.mixers.attention(q, -q, v, out, at(device, 0), scale=1.0, start_pos=0, variant=variant, sink=True)
        assert out.abs().max().item() == 0.0
        pkg.mixers.attention(q, q * 0, v, out, at(device, 0), scale=1.0, start_pos=0, variant=variant, sink=True)
        n = torch.arange(1, T + 1, device=device).float()
        assert (out[0, :, 0, 0].float() - n / (n + 1)).abs().max() < 5e-3


# ---- residual stream --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 8), (3, 60), (5, 33), (2, 2048), (700, 320), (4, 9000), (3, 1030), (400, 2048)])
def test_residual_norm(pkg, device, dtype, rows, width):
    x, y = rand(rows, width, seed=1, scale=3, dtype=F32) + 5, rand(rows, width, seed=2, dtype=dtype) - 2
    pw, pb, nw, nb, step = (rand(width, seed=s, dtype=F32) for s in range(3, 8))
    d = [t.to(device) for t in (y, x, pw, pb, nw, nb, step)]
    out = pkg.mixers.residual_norm(d[0], d[1], dtype=dtype, post=(d[2], d[3]), pre=(d[4], d[5]), eps=1e-3)
    want = x.double() + ref.layer_norm(y.double(), pw.double(), pb.double(), 1e-3)
    close(d[1], want, F32)
    close(out, ref.layer_norm(want, nw.double(), nb.double(), 1e-3), dtype)
    # the stream starts anew from a fp32 product, a step is added, and the plain stream goes into a strided place
    y32, wide = rand(rows, width, seed=9, dtype=F32).to(device), torch.zeros(rows, 2 * width, dtype=dtype, device=device)
    got = pkg.mixers.residual_norm(y32, d[1], dtype=dtype, reset=True, step=d[6], out=wide[:, :width])
    want = y32.double().cpu() + step.double()
    close(d[1], want, F32)
    close(got, want, dtype)
    assert wide[:, width:].abs().max() == 0
    # nothing added: only the norm
    before = d[1].clone()
    out = pkg.mixers.residual_norm(None, d[1], dtype=dtype, pre=(d[4], d[5]), eps=1e-3)
    assert torch.equal(before, d[1])
    close(out, ref.layer_norm(want, nw.double(), nb.double(), 1e-3), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_norm_keeps_small_deviations_of_a_large_mean(pkg, device, dtype):
    """Rows of 3000 with deviations near 0.1: sums of squares would lose them."""
    x = (3000 + 0.1 * rand(4, 1500, seed=1, dtype=F32))
    one, zero = torch.ones(1500, device=device), torch.zeros(1500, device=device)
    out = pkg.mixers.residual_norm(None, x.to(device), dtype=dtype, pre=(one, zero), eps=1e-9)
    close(out, ref.layer_norm(x.double(), torch.ones(1500, dtype=F64), torch.zeros(1500, dtype=F64), 1e-9), dtype, bound=1.5e-2 if dtype == BF16 else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 51])
def test_embedding_with_positions(pkg, device, dtype, width):
    B, T, pos = 2, 3, (0, 70001)
    table, tokens = rand(50, width, seed=5, dtype=dtype), torch.tensor([[3, 49, 0], [7, 7, 12]])
    freqs = (10000.0 ** (-2.0 * torch.arange((width + 1) // 2, dtype=F64) / width)).to(device)
    w, b = rand(width, seed=6, dtype=F32), rand(width, seed=7, dtype=F32)
    cat = torch.zeros(B, T, 2 * width, dtype=dtype, device=device)
    x, h = pkg.mixers.embed_residual(tokens.to(device), table.to(device), 1.7, freqs, at(device, *pos), x0=cat[..., width:],
                                     norm=(w.to(device), b.to(device)), eps=1e-5)
    want = table[tokens].double() * 1.7 + torch.stack([ref.sinusoid(torch.arange(p, p + T), width) for p in pos])
    assert (x.double().cpu() - want).abs().max() < 2e-6
    assert torch.equal(cat[..., width:], x.to(dtype)) and cat[..., :width].abs().max() == 0
    close(h, ref.layer_norm(want, w.double(), b.double(), 1e-5), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,ff", [(1, 8), (5, 33), (300, 256)])
def test_activations(pkg, device, dtype, rows, ff):
    gu = rand(rows, 2 * ff, seed=1, scale=3, dtype=dtype)
    g, u = gu.double()[:, :ff], gu.double()[:, ff:]
    close(pkg.mixers.gated_act(gu.to(device)), ref.silu(g) * u, dtype)
    g, u = g.clamp(max=0.9), u.clamp(-0.9, 0.9)
    close(pkg.mixers.gated_act(gu.to(device), limit=0.9), g / (1 + torch.exp(-1.702 * g)) * (u + 1), dtype)
    close(pkg.mixers.tanh_(gu.to(device)), torch.tanh(gu.double()), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", [(8, 2, 64, 96), (3, 1, 5, 9), (1, 1, 8, 8), (16, 4, 128, 128)])
def test_qk_norm_cache(pkg, device, dtype, H, G, D, V):
    """Whole-row norms; positions differ per sequence; rows of other positions stay; a position beyond the cache is skipped."""
    B, T, L, eps = 2, 3, 40, 1e-3
    qkv = rand(B, T, H * D + G * (D + V), seed=1, dtype=dtype)
    qw, kw = rand(H * D, seed=2, dtype=F32), rand(G * D, seed=3, dtype=F32)
    ck, cv = (torch.full((B, L, G, n), 7.0, dtype=dtype, device=device) for n in (D, V))
    d = qkv.to(device)
    pkg.mixers.qk_norm_cache(d, H * D, G * D, qw.to(device), kw.to(device), eps, ck, cv, at(device, 5, L - 2))
    q, k, v = qkv.double().split([H * D, G * D, G * V], dim=-1)
    close(d[..., :H * D], ref.rms(q, eps) * qw.double(), dtype)
    k = ref.rms(k, eps) * kw.double()
    for b, p, n in ((0, 5, 3), (1, L - 2, 2)):
        close(ck[b, p:p + n].reshape(n, -1), k[b, :n], dtype)
        assert torch.equal(cv[b, p:p + n].reshape(n, -1).cpu(), v[b, :n].to(dtype))
        ck[b, p:p + n], cv[b, p:p + n] = 7.0, 7.0
    assert (ck == 7).all() and (cv == 7).all()


# ---- recurrences ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 37])
def test_token_shift(pkg, device, dtype, width):
    B, n = 3, 5
    h, mu = rand(B, 10, width, seed=1, dtype=dtype), rand(n, width, seed=2, dtype=F32)
    last = torch.full((B, width), float("nan"), dtype=dtype, device=device)
    want = torch.stack([torch.stack([ref.token_shift(h[b].double(), mu[s].double()) for b in range(B)]) for s in range(n)])
    start = 0
    for T in (1, 1, 2, 5, 1):
        part = h[:, start:start + T].contiguous().to(device)
        out = pkg.mixers.token_shift(part, mu.to(device), last, at(device, *[start] * B))
        close(out, want[:, :, start:start + T], dtype, T)
        start += T
        assert torch.equal(last.cpu(), h[:, start - 1])


def delta_case(H, G, D, V, taps, B, T, dtype, seed=0):
    C_ = 2 * G * D + H * V
    p, b, a = rand(B, T, C_, seed=seed, dtype=dtype), rand(B, T, H, seed=seed + 1, dtype=dtype), rand(B, T, H * D, seed=seed + 2, dtype=dtype)
    conv = rand(taps, C_, seed=seed + 3, dtype=F32) * taps ** -0.5
    a_log, dt_bias = rand(H, seed=seed + 4, dtype=F32) - 1, rand(H * D, seed=seed + 5, dtype=F32)
    return p, b, a, conv, a_log, dt_bias


def delta_want(p, b, a, conv, a_log, dt_bias, H, G, D, V):
    """The oracle's inputs of the scan for one sequence, from projections (float64)."""
    x = ref.silu(ref.short_conv(p, conv.t()))
    T = x.shape[0]
    q, k, v = x.split([G * D, G * D, H * V], dim=-1)
    q, k = ref.unit(q.view(T, G, D)) * D ** -0.5, ref.unit(k.view(T, G, D))
    g = torch.exp(-torch.exp(a_log)[None, :, None] * ref.softplus(a + dt_bias).view(T, H, D))
    return q, k, v.view(T, H, V), 1 / (1 + torch.exp(-b)), g


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,taps", [(4, 2, 64, 32, 4), (3, 3, 5, 7, 1), (2, 1, 128, 128, 3), (2, 2, 200, 24, 6), (1, 1, 8, 8, 2)])
def test_delta_rule_in_portions(pkg, device, dtype, H, G, D, V, taps):
    """Inputs and scan over portions of every kind, two sequences: the outputs, the carried state and the carried inputs are
    those of the whole."""
    B, T, eps = 2, 60, 1e-4
    args = delta_case(H, G, D, V, taps, B, T, dtype)
    p, b, a, conv, a_log, dt_bias = args
    norm, gate = rand(V, seed=7, dtype=F32), rand(B, T, H, V, seed=8, dtype=dtype)
    want, states, inputs = [], [], []
    for s in range(B):
        q, k, v, beta, g = delta_want(*(t[s].double() for t in (p, b, a)), *(t.double() for t in (conv, a_log, dt_bias)), H, G, D, V)
        of = [i // (H // G) for i in range(H)]
        o, S = ref.delta_scan(q[:, of], k[:, of], v, g, beta)
        want.append((ref.rms(o, eps) * norm.double() / (1 + torch.exp(-gate[s].double()))).reshape(T, H * V))
        states.append(S)
        inputs.append((q, k, v, beta, g))
    want = torch.stack(want)
    for cuts in ([60], [1] * 60, [2] * 30, [16, 17, 1, 15, 3, 8], [33, 1, 26], [1, 2, 3, 54]):
        state = torch.full((B, H, D, V), float("nan"), device=device)
        tail = torch.full((B, taps - 1, p.shape[2]), float("nan"), dtype=dtype, device=device)
        start = 0
        for n in cuts:
            sl = slice(start, start + n)
            dp, db, da, dg = (t[:, sl].contiguous().to(device) for t in (p, b, a, gate))
            pos = at(device, *[start] * B)
            qk, v, beta, decay = pkg.mixers.delta_inputs(dp, db, da, conv.to(device), a_log.to(device), dt_bias.to(device), tail, pos, H, G, D, V)
            if len(cuts) < 7:
                for s in range(B):
                    for got, w in zip((qk[s, :, 0], qk[s, :, 1], beta[s], decay[s]), (inputs[s][0], inputs[s][1], inputs[s][3], inputs[s][4])):
                        close(got, w[sl], F32, cuts, bound=1e-4)
                    close(v[s], inputs[s][2][sl], dtype, cuts)
            out = pkg.mixers.recurrent_scan(qk[:, :, 0], qk[:, :, 1], v, decay, state, pos, norm.to(device), dg, act=pkg.mixers.SIGMOID, eps=eps,
                                            beta=beta, conv_in=dp, tail=tail, taps=taps)
            close(out.view(B, n, H, V), want[:, sl].view(B, n, H, V), dtype, cuts, bound=2.5e-2 if dtype == BF16 else 3e-5)
            start += n
        close(state.view(B, -1), torch.stack(states).view(B, -1), dtype, cuts)
        if taps > 1:
            assert torch.equal(tail.cpu(), p[:, T - taps + 1:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D", [(4, 64), (3, 7), (2, 128), (1, 8), (2, 180), (40, 32)])
def test_time_mixing_in_portions(pkg, device, dtype, H, D):
    B, T, eps = 2, 50, 1e-4
    r, k, v, g = (rand(B, T, H, D, seed=s, dtype=dtype) for s in range(4))
    x = rand(B, T, H, D, seed=5, dtype=dtype)
    w0, u, norm = rand(H * D, seed=6, dtype=F32) - 2, rand(H, D, seed=7, dtype=F32), rand(H, D, seed=8, dtype=F32)
    want, states = [], []
    for s in range(B):
        w = torch.exp(-torch.exp(x[s].double() + w0.double().view(H, D)))
        o, S = ref.wkv_scan(*(t[s].double() for t in (r, k, v)), w, u.double())
        want.append(ref.rms(o, eps) * norm.double() * ref.silu(g[s].double()))
        states.append(S)
    want = torch.stack(want)
    for cuts in ([50], [1] * 50, [2] * 25, [17, 1, 15, 17], [48, 2]):
        state, start = torch.full((B, H, D, D), float("nan"), device=device), 0
        for n in cuts:
            sl = slice(start, start + n)
            dr, dk, dv, dg, dx = (t[:, sl].contiguous().to(device) for t in (r, k, v, g, x))
            out = pkg.mixers.recurrent_scan(dr, dk, dv, dx, state, at(device, *[start] * B), norm.to(device), dg, act=pkg.mixers.SILU, eps=eps,
                                            bonus=u.to(device), g_bias=w0.to(device))
            close(out.view(B, n, H, D), want[:, sl], dtype, cuts, bound=2e-2 if dtype == BF16 else 3e-5)
            start += n
        close(state.view(B, -1), torch.stack(states).view(B, -1), F32, cuts)


def test_scan_of_sequences_at_different_places(pkg, device):
    """One step of a batch in which some sequences start: these begin at zero, the others go on."""
    H, D, V, B = 2, 16, 24, 4
    q, k, g = (rand(B, 1, H, D, seed=s, dtype=F32) for s in range(3))
    v, gate, beta = rand(B, 1, H, V, seed=3, dtype=F32), rand(B, 1, H, V, seed=4, dtype=F32), rand(B, 1, H, seed=5, dtype=F32)
    held = rand(B, H, D, V, seed=6, dtype=F32)
    state, norm = held.to(device), torch.ones(V)
    out = pkg.mixers.recurrent_scan(q.to(device), k.to(device), v.to(device), g.to(device), state, at(device, 0, 9, 0, 1), norm.to(device),
                                    gate.to(device), act=pkg.mixers.SIGMOID, eps=1e-5, beta=beta.to(device))
    for b in range(B):
        start = torch.zeros(H, D, V, dtype=F64) if b in (0, 2) else held[b].double()
        o, S = ref.delta_scan(*(t[b].double() for t in (q, k, v, g, beta)), state=start)
        close(out[b].view(1, H, V), ref.rms(o, 1e-5) / (1 + torch.exp(-gate[b].double())), F32)
        close(state[b].reshape(1, -1), S.reshape(1, -1), F32)


# ---- experts ----------------------------------------------------------------------------------------------------
def route(pkg, device, rows, width, E, top, dtype, seed=0, skew=0.0):
    h, logits, bias = rand(rows, width, seed=seed, dtype=dtype), rand(rows, E, seed=seed + 1, scale=5, dtype=F32), rand(E, seed=seed + 2, dtype=F32)
    bias[0] += skew
    return h, logits.double() + bias.double(), pkg.mixers.moe_route(logits.to(device), bias.to(device), top)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,E,top,skew", [(1, 64, 8, 2, 0), (5, 33, 3, 3, 0), (700, 64, 9, 4, 0), (700, 40, 64, 1, 0), (33, 96, 1, 1, 0),
                                                   (2000, 32, 6, 2, 100.0), (601, 48, 200, 7, 0)])
def test_routing_and_sorting(pkg, device, dtype, rows, width, E, top, skew):
    h, z, (experts, ranks, weights, counts) = route(pkg, device, rows, width, E, top, dtype, skew=skew)
    chosen, w = ref.route(z, top)
    clear = torch.ones(rows, dtype=torch.bool)
    if top < E:
        s = z.sort(dim=-1, descending=True).values
        clear = s[:, top - 1] - s[:, top] > 1e-5
    e = experts.cpu().long()
    assert torch.equal(e.sort(-1).values[clear], chosen.sort(-1).values[clear]) and clear.float().mean() > 0.9
    assert (weights.cpu().double() - w)[clear].abs().max() < 2e-4
    assert torch.equal(counts.cpu().long(), torch.bincount(e.flatten(), minlength=E))
    x, part_rows = pkg.mixers.moe_gather(h.to(device), experts, ranks, counts)
    at_ = part_rows.cpu().long().flatten()
    assert torch.equal(at_.sort().values, torch.arange(rows * top))                               # a permutation
    by_place = torch.empty(rows * top, dtype=torch.long)
    by_place[at_] = e.flatten()
    assert (by_place.diff() >= 0).all()                                                           # expert by expert
    assert torch.equal(x.cpu()[at_], h.repeat_interleave(top, 0))


def test_equal_logits_take_the_smaller_index(pkg, device):
    for E in (5, 33, 100):
        experts, _, weights, _ = pkg.mixers.moe_route(torch.zeros(40, E, device=device), torch.zeros(E, device=device), 3)
        assert (experts.cpu() == torch.arange(3)).all() and (weights - 1 / 3).abs().max() < 1e-6
    z = torch.full((40, 50), -1e30, device=device)
    z[:, 41], z[:, 7], z[:, 20] = float("inf"), float("nan"), -5.0
    assert (pkg.mixers.moe_route(z, torch.zeros(50, device=device), 3)[0].cpu() == torch.tensor([41, 20, 0])).all()


@pytest.mark.parametrize("E,counts_kind", [(4, "even"), (7, "one"), (40, "random")])
@pytest.mark.parametrize("rows,K,N", [(1, 64, 64), (100, 72, 40), (700, 256, 304), (37, 13, 21), (3000, 128, 1032)])
def test_expert_products(pkg, device, E, counts_kind, rows, K, N):
    """Gated and plain, both variants, both types: empty experts, runs that end inside a tile, columns behind the last one."""
    g = torch.Generator().manual_seed(rows)
    if counts_kind == "one":
        counts = torch.zeros(E, dtype=torch.int32)
        counts[E - 2] = rows
    else:
        p = torch.ones(E) if counts_kind == "even" else torch.rand(E, generator=g) ** 3
        counts = torch.bincount(torch.multinomial(p, rows, True, generator=g), minlength=E).int()
    of = torch.repeat_interleave(torch.arange(E), counts.long())
    for dtype in DTYPES:
        x, w, w2 = rand(rows, K, seed=1, dtype=dtype), rand(E, 2, N, K, seed=2, scale=2 * K ** -0.5, dtype=dtype), rand(E, N, K, seed=3, dtype=dtype)
        want = torch.zeros(rows, N, dtype=F64)
        plain = torch.zeros(rows, N, dtype=F64)
        eye = torch.eye(N, dtype=F64)
        for e in range(E):
            if (of == e).any():
                want[of == e] = ref.clamped_expert(w[e, 0].double(), w[e, 1].double(), eye, x[of == e].double(), 0.8)
                plain[of == e] = x[of == e].double() @ w2[e].double().T
        for variant in ((0, 1, 2) if dtype == BF16 and K % 8 == 0 and N % 8 == 0 else (0, 1)):
            status = torch.zeros(1, dtype=torch.int32, device=device)
            d = [t.to(device) for t in (x, w, w2, counts)]
            got = pkg.mixers.moe_gemm(d[0], d[1], d[3], limit=0.8, variant=variant, status=status)
            close(got, want, dtype, (variant, "gated"))
            close(pkg.mixers.moe_gemm(d[0], d[2], d[3], variant=variant, status=status), plain, dtype, (variant, "plain"))
            assert status.item() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_tokens_experts_are_combined(pkg, device, dtype):
    rows, width, E, top, ff, limit = 50, 64, 6, 3, 40, 0.7
    h, z, (experts, ranks, weights, counts) = route(pkg, device, rows, width, E, top, dtype)
    w = {f"e{e}.{n}": rand(*s, seed=10 * e + i, scale=s[1] ** -0.5, dtype=dtype) for e in range(E)
         for i, (n, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))}
    gate_up = torch.stack([torch.stack([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)]).to(device)
    down = torch.stack([w[f"e{e}.down"] for e in range(E)]).to(device)
    x, part_rows = pkg.mixers.moe_gather(h.to(device), experts, ranks, counts)
    y = pkg.mixers.moe_gemm(pkg.mixers.moe_gemm(x, gate_up, counts, limit=limit), down, counts)
    stream = torch.zeros(rows, width, device=device)
    pkg.mixers.residual_norm(y, stream, dtype=dtype, part_rows=part_rows, part_weights=weights)
    want = torch.zeros(rows, width, dtype=F64)
    chosen, p = ref.route(z, top)
    for t in range(rows):
        for e, q in zip(chosen[t].tolist(), p[t]):
            want[t] += q * ref.clamped_expert(*(w[f"e{e}.{n}"].double() for n in ("gate", "up", "down")), h[t].double(), limit)
    close(stream, want, dtype, bound=2e-2 if dtype == BF16 else 2e-5)
