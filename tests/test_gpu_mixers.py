"""The mixer kernels (include/l3ci_mixers.h), each against the plain float64 restatement in oracle/nibelorn.py: every
variant of the attention kernel over sizes that are not multiples of its tiles, keys that stand out at tile borders,
device-side positions, and the steps around the mixers."""
import math

import pytest
import torch

from oracle import nibelorn as ref

pytestmark = pytest.mark.gpu
BF16, F32 = torch.bfloat16, torch.float32


def rand(*shape, seed=0, scale=1.0, dtype=BF16):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def close(got, want, dtype, what=""):
    """Relative L2 per row of the last axis, rounding of the type only."""
    got, want = got.double().cpu(), want.double()
    rel = (got - want).norm(dim=-1) / (want.norm(dim=-1) + 1e-3 * want.abs().max())
    bound = 1.2e-2 if dtype == BF16 else 2e-5
    assert rel.max().item() < bound, f"{what}: {rel.max().item()} at {rel.argmax().item()} of {tuple(rel.shape)}"


def run_variants(pkg, device, dtype, variants, make):
    """`make(variant)` -> (out tensor, reference) for every variant that takes the sizes."""
    for v in variants:
        got, want = make(v)
        torch.cuda.synchronize()
        close(got, want, dtype, f"variant {v}")


# ---- elementwise steps --------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("rows,width", [(1, 8), (3, 60), (5, 33), (7, 2048), (300, 320)])
def test_add_dyn_tanh(pkg, device, dtype, rows, width):
    x, y = rand(rows, width, seed=1, scale=3, dtype=F32), rand(rows, width, seed=2, dtype=dtype)
    w, b = rand(width, seed=3, dtype=F32), rand(width, seed=4, dtype=F32)
    alpha = torch.tensor(0.37)
    dx = x.to(device)
    out = pkg.mixers.add_dyn_tanh(y.to(device), dx, w.to(device), b.to(device), float(alpha))
    want_x = x.double() + y.double()
    assert torch.equal(dx.cpu(), (x + y.float()))
    want = ref.dyn_tanh(want_x, w, b, alpha)
    assert (out.double().cpu() - want).abs().max() < (2e-2 if dtype == BF16 else 1e-5)
    close(out, want, dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [64, 100])
def test_embedding_starts_the_residual(pkg, device, dtype, width):
    table, tokens = rand(50, width, seed=5, dtype=dtype), torch.tensor([[3, 49, 0], [7, 7, 12]])
    w, b = rand(width, seed=6, dtype=F32), rand(width, seed=7, dtype=F32)
    x, h = pkg.mixers.embed_dyn_tanh(tokens.to(device), table.to(device), w.to(device), b.to(device), 1.5)
    assert x.dtype == F32 and torch.equal(x.cpu(), table[tokens].float())
    close(h, ref.dyn_tanh(table[tokens].double(), w, b, torch.tensor(1.5)), dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("n", [1, 7, 4096, 4099])
def test_gelu(pkg, device, dtype, n):
    z = rand(n, seed=8, scale=3, dtype=dtype)
    out = pkg.mixers.gelu_(z.to(device).clone())
    want = ref.gelu(z.double())
    assert (out.double().cpu() - want).abs().max() < (3e-2 if dtype == BF16 else 2e-6)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,D,R,C", [(3, 24, 8, 40), (2, 10, 6, 33), (16, 128, 64, 512), (1, 16, 2, 16)])
def test_latent_cache_rows(pkg, device, dtype, H, D, R, C):
    """Positions differ per sequence; rows of other positions stay as they were; a position beyond the cache is skipped."""
    B, T, L, base, eps = 2, 3, 900, 1234.5, 1e-5
    W = H * (D + R) + C + R
    qd, nw = rand(B, T, W, seed=9, dtype=dtype), rand(C, seed=10, dtype=F32)
    table = pkg.rope_table.rotation_table(R, L, base)
    width = (C + R + 7) // 8 * 8
    cache = torch.full((B, L, width), 7.0, dtype=dtype, device=device)
    positions = torch.tensor([5, L - 2], dtype=torch.int32, device=device)   # the second sequence's last token does not fit
    dq = qd.to(device).clone()
    pkg.mixers.latent_cache(dq, table.to(device), nw.to(device), eps, cache, positions, H, D, R, C)
    torch.cuda.synchronize()
    for b, p0 in enumerate((5, L - 2)):
        for t in range(T):
            if p0 + t >= L:
                continue
            pos, row = torch.tensor([p0 + t]), qd[b, t].double()
            q = row[:H * (D + R)].view(1, H, D + R)
            got_q = dq[b, t, :H * (D + R)].view(H, D + R).cpu()
            assert torch.equal(got_q[:, :D], qd[b, t, :H * (D + R)].view(H, D + R)[:, :D])
            close(got_q[:, D:], ref.rotate_half(q[..., D:], pos, base)[0], dtype, "q")
            c = row[H * (D + R):H * (D + R) + C]
            close(cache[b, p0 + t, :C], ref.rms(c, eps) * nw.double(), dtype, "latent")
            close(cache[b, p0 + t, C:C + R], ref.rotate_half(row[None, H * (D + R) + C:], pos, base)[0], dtype, "k")
    untouched = cache.clone()
    untouched[0, 5:8] = 7.0
    untouched[1, L - 2:] = 7.0
    assert bool((untouched == 7.0).all()) and bool((cache[..., C + R:] == 7.0).all())


@pytest.mark.parametrize("H,D,R,C", [(3, 24, 16, 40), (16, 128, 64, 512), (20, 32, 96, 768)])
def test_latent_cache_rows_of_many_tokens(pkg, device, H, D, R, C):
    """The warp-per-token form: enough tokens to take it, the last ones beyond the cache."""
    B, T, L, base, eps = 2, 1500, 1600, 500.0, 1e-5
    W = H * (D + R) + C + R
    qd, nw = rand(B, T, W, seed=9), rand(C, seed=10, dtype=F32)
    cache = torch.full((B, L, C + R), 7.0, dtype=BF16, device=device)
    positions = torch.tensor([0, 150], dtype=torch.int32, device=device)
    dq = qd.to(device).clone()
    pkg.mixers.latent_cache(dq, pkg.rope_table.rotation_table(R, L, base).to(device), nw.to(device), eps, cache, positions, H, D, R, C)
    for b, p0, n in ((0, 0, T), (1, 150, L - 150)):
        pos, rows = torch.arange(p0, p0 + n), qd[b, :n].double()
        q, down = rows[:, :H * (D + R)].view(n, H, D + R), rows[:, H * (D + R):]
        got = dq[b, :, :H * (D + R)].view(T, H, D + R)
        assert torch.equal(got[..., :D].cpu(), qd[b, :, :H * (D + R)].view(T, H, D + R)[..., :D])
        close(got[:n, :, D:], ref.rotate_half(q[..., D:], pos, base), BF16, "q")
        assert torch.equal(got[n:, :, D:].cpu(), qd[b, n:, :H * (D + R)].view(T - n, H, D + R)[..., D:])
        close(cache[b, p0:p0 + n, :C], ref.rms(down[:, :C], eps) * nw.double(), BF16, "latent")
        close(cache[b, p0:p0 + n, C:], ref.rotate_half(down[:, C:], pos, base), BF16, "k")
    assert bool((cache[0, T:] == 7.0).all()) and bool((cache[1, :150] == 7.0).all())


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("G,D,V", [(2, 8, 24), (3, 5, 7)])
@pytest.mark.parametrize("T", [4, 700])
def test_kv_cache_write(pkg, device, dtype, G, D, V, T):
    B, L = 2, T + 16
    src = rand(B, T, 16 + G * (2 * D + V) + 8, seed=11, dtype=dtype).to(device)
    k = torch.zeros(B, L, G, 2 * D, dtype=dtype, device=device)
    v = torch.zeros(B, L, G, V, dtype=dtype, device=device)
    positions = torch.tensor([0, 13], dtype=torch.int32, device=device)
    pkg.mixers.kv_cache_write(src, 16, 16 + G * 2 * D, k, v, positions)
    for b, p in enumerate((0, 13)):
        assert torch.equal(k[b, p:p + T].flatten(1), src[b, :, 16:16 + G * 2 * D])
        assert torch.equal(v[b, p:p + T].flatten(1), src[b, :, 16 + G * 2 * D:16 + G * (2 * D + V)])
        k[b, p:p + T] = 0
        v[b, p:p + T] = 0
    assert not k.any() and not v.any()


# ---- attention ------------------------------------------------------------------------------------------------
def latent_case(pkg, device, dtype, B, T, H, C, R, starts, L, seed=0, variant=0, boost=None):
    """Absorbed form: one key row per token (C latent + R rotated), values are its first C columns."""
    width = (C + R + 7) // 8 * 8
    q, rows = rand(B, T, H, C + R, seed=seed, dtype=dtype), rand(B, L, width, seed=seed + 1, dtype=dtype)
    scale = 1.7 / math.sqrt(C + R)
    if boost is not None:   # one key stands out for every query of sequence 0
        rows[0, boost, :C + R] = (4.0 * q[0, :, 0].double().mean(0)).to(dtype)
    positions = torch.tensor(starts, dtype=torch.int32, device=device)
    dq, dc = q.to(device), rows.to(device)
    out = torch.empty(H, B, T, C, dtype=dtype, device=device).permute(1, 2, 0, 3)
    same = starts[0] if len(set(starts)) == 1 and T > 1 else -1
    pkg.mixers.attention(dq[..., :C], dc[:, :, None, :C], dc[:, :, None, :C], out, positions, qb=dq[..., C:],
                         kb=dc[:, :, None, C:C + R], scale=scale, start_pos=same, variant=variant)
    want = torch.stack([ref.cached_attention(q[b], rows[b, :, None, :C + R], rows[b, :, None, :C], starts[b], scale)
                        for b in range(B)])
    return out, want


@pytest.mark.parametrize("H,C,R", [(1, 16, 8), (5, 40, 24), (10, 112, 24), (16, 512, 64), (20, 96, 32), (3, 200, 8)])
@pytest.mark.parametrize("T,starts", [(1, (0, 70)), (1, (63, 64)), (1, (127, 300)), (2, (62, 62)), (7, (0, 0)), (67, (129, 129))])
def test_latent_attention_over_the_cache(pkg, device, H, C, R, T, starts):
    run_variants(pkg, device, BF16, (1, 2), lambda v: latent_case(pkg, device, BF16, 2, T, H, C, R, starts, 384, variant=v))


@pytest.mark.parametrize("C,R,starts", [(33, 6, (0, 200)), (112, 24, (130, 129))])
def test_latent_attention_fp32(pkg, device, C, R, starts):
    run_variants(pkg, device, F32, (0, 1), lambda v: latent_case(pkg, device, F32, 2, 1, 3, C, R, starts, 256, variant=v))


@pytest.mark.parametrize("key", [0, 1, 62, 63, 64, 65, 127, 128, 191, 192, 1023, 1024, 2046, 2047])
def test_latent_attention_finds_a_single_key(pkg, device, key):
    """A far key that carries almost all the weight, at tile and split borders; the query is at 2047."""
    run_variants(pkg, device, BF16, (1, 2), lambda v: latent_case(pkg, device, BF16, 1, 1, 4, 64, 16, (2047,), 2304, variant=v, boost=key))


def differential_case(pkg, device, dtype, B, T, H, G, D, V, starts, L, cap=20.0, temp=(0.4, 50.0), gated=True, variant=0,
                      q_scale=1.0, boost=None, seed=0):
    q, k, v = (rand(B, T, H, 2 * D, seed=seed, scale=q_scale, dtype=dtype), rand(B, L, G, 2 * D, seed=seed + 1, dtype=dtype),
               rand(B, L, G, V, seed=seed + 2, dtype=dtype))
    gate = rand(B, T, H + 3, seed=seed + 3, dtype=dtype)[..., :H] if gated else None
    scale, lam, diff, eps = 1.3 / math.sqrt(D), 0.61, 0.35, 1e-5
    if boost is not None:
        m, key = boost
        k[0, key, :, m * D:(m + 1) * D] = (6.0 * q[0, 0].view(G, H // G, 2 * D)[:, 0, m * D:(m + 1) * D].double()).to(dtype)
    positions = torch.tensor(starts, dtype=torch.int32, device=device)
    out = torch.empty(B, T, H, V, dtype=dtype, device=device)
    same = starts[0] if len(set(starts)) == 1 and T > 1 else -1
    dg = rand(B, T, H + 3, seed=seed + 3, dtype=dtype).to(device)[..., :H] if gated else None
    pkg.mixers.attention(q.to(device), k.to(device), v.to(device), out, positions, maps=2, scale=scale, softcap=cap,
                         temp_coef=temp[0], temp_every=temp[1], gate=dg, lambda_=lam, post=1 - diff, eps=eps,
                         start_pos=same, variant=variant)
    want = []
    for b in range(B):
        a = [ref.cached_attention(q[b, ..., m * D:(m + 1) * D], k[b, ..., m * D:(m + 1) * D], v[b], starts[b], scale, cap,
                                  temp if temp[1] else None) for m in range(2)]
        want.append(ref.differential_combine(a[0], a[1], lam, diff, eps, gate[b] if gated else None))
    return out, torch.stack(want)


@pytest.mark.parametrize("H,G,D,V", [(4, 1, 40, 56), (6, 2, 24, 40), (8, 8, 64, 128), (16, 4, 64, 128), (12, 1, 16, 8), (5, 5, 128, 256)])
@pytest.mark.parametrize("T,starts", [(1, (0, 90)), (1, (63, 64)), (2, (126, 126)), (9, (0, 0)), (67, (100, 100))])
def test_differential_attention_over_the_cache(pkg, device, H, G, D, V, T, starts):
    run_variants(pkg, device, BF16, (1, 2), lambda v: differential_case(pkg, device, BF16, 2, T, H, G, D, V, starts, 320, variant=v))


@pytest.mark.parametrize("cap,temp,gated", [(0.0, (0.0, 0.0), False), (2.0, (0.0, 0.0), True), (0.0, (1.5, 7.0), True), (5.0, (0.3, 1.0), False)])
def test_differential_attention_options(pkg, device, cap, temp, gated):
    """No cap, a cap that bites, temperatures that change from token to token, no gate."""
    for dtype, variants in ((BF16, (1, 2)), (F32, (1,))):
        run_variants(pkg, device, dtype, variants, lambda v: differential_case(
            pkg, device, dtype, 2, 5, 4, 2, 16, 24, (140, 140), 160, cap=cap, temp=temp, gated=gated, variant=v, q_scale=2.0))


@pytest.mark.parametrize("m", [0, 1])
@pytest.mark.parametrize("key", [0, 63, 64, 127, 128, 1023, 1024, 1500])
def test_differential_attention_finds_a_single_key(pkg, device, m, key):
    """One map's weight sits on one key."""
    run_variants(pkg, device, BF16, (1, 2), lambda v: differential_case(pkg, device, BF16, 1, 1, 4, 2, 32, 64, (1500,), 1600,
                                                                        boost=(m, key), variant=v))


@pytest.mark.parametrize("H,G,D,V", [(4, 1, 40, 56), (6, 2, 24, 40), (3, 3, 64, 128), (16, 4, 64, 128), (2, 1, 8, 8)])
@pytest.mark.parametrize("T,start", [(128, 0), (129, 0), (300, 0), (130, 77), (128, 128), (5, 260)])
def test_differential_attention_of_a_prompt(pkg, device, H, G, D, V, T, start):
    """The tcgen05 kernel: whole prompts and later portions, more items than SMs and fewer."""
    for cap in (0.0, 20.0):
        run_variants(pkg, device, BF16, (3,), lambda v: differential_case(pkg, device, BF16, 2, T, H, G, D, V, (start, start),
                                                                          start + T + 10, cap=cap, variant=v))


def test_differential_attention_of_a_long_prompt(pkg, device):
    run_variants(pkg, device, BF16, (3,), lambda v: differential_case(pkg, device, BF16, 1, 1500, 16, 4, 32, 64, (0,), 1500, variant=v))


@pytest.mark.parametrize("cap", [0.0, 1.0, 6.0])
@pytest.mark.parametrize("temp", [(0.0, 0.0), (1.5, 7.0), (-0.9, 3.0)])
def test_prompt_scores_beyond_the_cap(pkg, device, cap, temp):
    """Scores far outside the cap's near-linear range; temperatures that grow, and that turn negative."""
    run_variants(pkg, device, BF16, (2, 3), lambda v: differential_case(pkg, device, BF16, 1, 200, 4, 2, 32, 64, (40,), 240, cap=cap,
                                                                        temp=temp, variant=v, q_scale=2.0))


@pytest.mark.parametrize("m", [0, 1])
@pytest.mark.parametrize("key", [0, 1, 127, 128, 255, 256, 700])
def test_prompt_differential_attention_finds_a_single_key(pkg, device, m, key):
    def make(v):
        B, T, start, H, G, D, V = 1, 140, 700, 2, 1, 32, 64
        q, k, val = rand(B, T, H, 2 * D, seed=1), rand(B, 840, G, 2 * D, seed=2), rand(B, 840, G, V, seed=3)
        k[0, key, 0, m * D:(m + 1) * D] = (40.0 * q[0, 139, 1, m * D:(m + 1) * D].double() / q[0, 139, 1, m * D:(m + 1) * D].double().norm()).to(BF16)
        out = torch.empty(B, T, H, V, dtype=BF16, device=device)
        pkg.mixers.attention(q.to(device), k.to(device), val.to(device), out, torch.full((1,), start, dtype=torch.int32, device=device),
                             maps=2, scale=0.2, softcap=30.0, lambda_=0.4, post=0.6, eps=1e-5, start_pos=start, variant=v)
        a = [ref.cached_attention(q[0, ..., i * D:(i + 1) * D], k[0, ..., i * D:(i + 1) * D], val[0], start, 0.2, 30.0) for i in range(2)]
        return out[0], ref.differential_combine(a[0], a[1], 0.4, 0.4, 1e-5)

    run_variants(pkg, device, BF16, (1, 2, 3), make)


@pytest.mark.parametrize("H,D,R,V", [(3, 64, 24, 56), (5, 128, 64, 128), (2, 24, 8, 40), (4, 72, 64, 64), (1, 128, 32, 72), (7, 64, 64, 128)])
@pytest.mark.parametrize("T,start", [(128, 0), (257, 0), (700, 0), (130, 77), (128, 128), (40, 260)])
def test_expanded_latent_attention_of_a_prompt(pkg, device, H, D, R, V, T, start):
    """Keys and values per head, the rotated key part shared by the heads and lying in other rows than the rest."""
    B, S, scale = 2, start + T, 1.4 / math.sqrt(D + R)
    q, kv, rows = rand(B, T, H, D + R, seed=1), rand(B, S, H * (D + V), seed=2), rand(B, S + 5, 16 + R, seed=3)
    out = torch.empty(B, T, H, V, dtype=BF16, device=device)
    dq, dkv, drows = q.to(device), kv.to(device), rows.to(device)
    positions = torch.full((B,), start, dtype=torch.int32, device=device)
    for variant in (1, 3):
        out.zero_()
        pkg.mixers.attention(dq[..., :D], dkv[..., :H * D].view(B, S, H, D), dkv[..., H * D:].view(B, S, H, V), out, positions,
                             qb=dq[..., D:], kb=drows[:, :S, None, 16:].expand(B, S, H, R), scale=scale, start_pos=start,
                             variant=variant)
        torch.cuda.synchronize()
        for b in range(B):
            k = torch.cat([kv[b, :, :H * D].view(S, H, D), rows[b, :S, None, 16:].expand(S, H, R)], dim=-1)
            close(out[b], ref.cached_attention(q[b], k, kv[b, :, H * D:].view(S, H, V), start, scale), BF16, f"variant {variant}")


def test_one_map_without_a_second_part(pkg, device):
    B, T, S, H, G, D, V = 1, 200, 230, 6, 2, 96, 56
    q, k, v = rand(B, T, H, D, seed=1), rand(B, S, G, D, seed=2), rand(B, S, G, V, seed=3)
    for variant in (1, 2, 3):
        out = torch.empty(B, T, H, V, dtype=BF16, device=device)
        pkg.mixers.attention(q.to(device), k.to(device), v.to(device), out, torch.full((1,), 30, dtype=torch.int32, device=device),
                             scale=0.15, start_pos=30, variant=variant)
        close(out[0], ref.cached_attention(q[0], k[0], v[0], 30, 0.15), BF16, f"variant {variant}")


def test_attention_reads_nothing_beyond_the_position(pkg, device):
    """What lies in the cache after a query's position (an earlier holder's rows, even NaN) does not enter."""
    B, T, H, C, R, L = 1, 1, 4, 64, 16, 512
    q, rows = rand(B, T, H, C + R, seed=1).to(device), rand(B, L, C + R, seed=2).to(device)
    k, v, qd = rand(B, L, 2, 64, seed=3).to(device), rand(B, L, 2, 64, seed=4).to(device), rand(B, T, H, 64, seed=5).to(device)
    for pos in (0, 1, 62, 63, 64, 200, 510):
        positions = torch.tensor([pos], dtype=torch.int32, device=device)
        for variant in (1, 2):
            outs = []
            for fill in (0.0, float("nan")):
                c, kk, vv = rows.clone(), k.clone(), v.clone()
                for t in (c, kk, vv):
                    t[:, pos + 1:] = fill
                o = torch.empty(B, T, H, C, dtype=BF16, device=device)
                pkg.mixers.attention(q[..., :C], c[:, :, None, :C], c[:, :, None, :C], o, positions, qb=q[..., C:],
                                     kb=c[:, :, None, C:], scale=0.2, variant=variant)
                d = torch.empty(B, T, H, 64, dtype=BF16, device=device)
                pkg.mixers.attention(qd, kk, vv, d, positions, maps=2, scale=0.2, lambda_=0.5, post=0.5, eps=1e-5, variant=variant)
                outs += [o, d]
            assert torch.equal(outs[0], outs[2]) and torch.equal(outs[1], outs[3]), (pos, variant)


def test_refuses_what_it_cannot_run(pkg, device):
    q = rand(1, 1, 3, 16).to(device)
    with pytest.raises(RuntimeError):   # 3 query heads over 2 key heads
        pkg.mixers.attention(q, rand(1, 8, 2, 16).to(device), rand(1, 8, 2, 16).to(device), torch.empty_like(q),
                             torch.zeros(1, dtype=torch.int32, device=device), scale=1.0)
    f = q.float()
    with pytest.raises(RuntimeError):   # the tensor-core variants are bf16
        pkg.mixers.attention(f, f, f, torch.empty_like(f), torch.zeros(1, dtype=torch.int32, device=device), scale=1.0, variant=2)
    with pytest.raises(ValueError):
        pkg.mixers.gelu_(torch.zeros(4))
