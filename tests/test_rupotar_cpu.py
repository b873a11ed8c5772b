"""What needs no GPU of the Rupotar decoder and the framework around it: configuration, registry, tensor names, state planes of
the cache, argument checks of the kernels' C ABI, and the oracle against closed forms and itself."""
import ctypes as C
import math
import re
from pathlib import Path

import pytest
import torch

from oracle import rupotar as ref
from tests.rupotar_cases import NAMES, case, weights, write_model


def test_configuration_reads_every_key(pkg):
    ru = pkg.rupotar
    cfg = ru.config_from_json(case("mixed"))
    assert (cfg.vocab_size, cfg.width, cfg.eps, cfg.embed_scale) == (211, 104, 1e-4, 2.5)
    assert cfg.loop == ru.Loop(1, 3, 2)
    assert cfg.layers[0].mixer == ru.Attention(6, 2, 16, 24, 16 ** -0.5, 13, 5)
    assert cfg.layers[1].mixer == ru.ChannelDelta(6, 3, 24, 16, 4)
    assert cfg.layers[2].mixer == ru.TimeMix(3, 24) and cfg.layers[2].ff is None
    assert cfg.layers[3].mixer == ru.Attention(4, 4, 8, 16, 8 ** -0.5, 0, 0)
    assert cfg.layers[1].ff == ru.Experts(40, 0.8, 6, 3) and cfg.layers[0].ff == ru.Dense(72)


def test_runs_follow_the_loop(pkg):
    runs = [(r.layer, r.step) for r in pkg.rupotar.config_from_json(case("mixed")).runs]
    assert runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert [(r.layer, r.step) for r in pkg.rupotar.config_from_json(case("thin")).runs] == [(0, 0), (1, None), (2, None)]
    assert [(r.layer, r.step) for r in pkg.rupotar.config_from_json(case("odd")).runs] == [(i, None) for i in range(4)]
    for name in NAMES:
        want = [(i, t if opens else None) for i, t, opens in ref.layer_runs(case(name))]
        assert [(r.layer, r.step) for r in pkg.rupotar.config_from_json(case(name)).runs] == want


def test_configuration_refuses_what_it_does_not_know(pkg):
    for change in (lambda c: c["layers"][0].update(type="latent_attention"), lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
                   lambda c: c["loop"].update(stop=9), lambda c: c["loop"].update(times=0)):
        c = case("mixed")
        change(c)
        with pytest.raises(ValueError):
            pkg.rupotar.config_from_json(c)


@pytest.mark.parametrize("name", NAMES)
def test_a_checkpoint_has_exactly_the_named_tensors(pkg, tmp_path, name):
    c = case(name)
    w = weights(pkg, c)
    shapes = pkg.rupotar.tensor_shapes(pkg.rupotar.config_from_json(c))
    assert w.keys() == shapes.keys()
    assert all(len(w[n].shape) == len(s) and all(x in (None, y) for x, y in zip(s, w[n].shape)) for n, s in shapes.items())
    assert ("loop.in" in w) == ("loop" in c)
    write_model(tmp_path, c, w)
    got = pkg.checkpoint.read_weights(tmp_path)
    assert all(torch.equal(got[n], w[n]) for n in w)
    assert pkg.models.architecture_of(pkg.checkpoint.read_config(tmp_path)).decoder is pkg.rupotar.RupotarDecoder


def test_state_planes_hold_one_value_per_sequence(pkg):
    planes = [pkg.rupotar.ChannelDelta(6, 3, 24, 16, 4).planes(104), pkg.rupotar.TimeMix(3, 24).planes(104),
              pkg.rupotar.Attention(6, 2, 16, 24, 1.0).planes(104)]
    cache = pkg.kv_cache.StaticCache(planes, 2, 9, torch.bfloat16, "cpu")
    shapes = [{n: (tuple(t.shape), t.dtype) for n, t in l.items()} for l in cache.layers]
    bf, f = torch.bfloat16, torch.float32
    assert shapes == [{"state": ((2, 6, 24, 16), f), "tail": ((2, 3, 2 * 72 + 96), bf)}, {"state": ((2, 3, 24, 24), f), "last": ((2, 104), bf)},
                      {"k": ((2, 9, 2, 16), bf), "v": ((2, 9, 2, 24), bf)}]


def test_struct_layouts(pkg):
    m = pkg.mixers
    text = (Path(__file__).resolve().parents[1] / "include" / "l3ci_mixers.h").read_text()
    for name, struct in (("residual_norm", m.ResidualNormArgs), ("delta_inputs", m.DeltaInputsArgs), ("recurrent_scan", m.RecurrentScanArgs),
                         ("moe_gemm", m.MoeGemmArgs)):
        body = text[text.index(f"typedef struct l3ci_{name}_args"):text.index("} l3ci_" + name + "_args")]
        body = re.sub(r"/\*.*?\*/", "", body, flags=re.S).replace("*", " ")
        assert re.findall(r"\b(\w+)(?=[,;])", body) == [n for n, _ in struct._fields_], name   # same members, same order
    assert C.sizeof(m.ResidualNormArgs) == 15 * 8 + 5 * 8 + 5 * 4 + 2 * 4 + 4 + 8
    assert C.sizeof(m.DeltaInputsArgs) == 12 * 8 + 4 * 8 + 8 * 4 + 4 + 4 + 8
    assert C.sizeof(m.RecurrentScanArgs) == 15 * 8 + 14 * 8 + 10 * 4 + 4 + 4 + 8
    assert C.sizeof(m.MoeGemmArgs) == 5 * 8 + 8 + 6 * 4 + 2 * 4 + 8


def test_argument_validation_happens_before_cuda(pkg):
    m = pkg.mixers
    lib, fake = m.load(), 0x1000   # never dereferenced: validation fails first
    bad, unsupported, ok = pkg.capi.ERR_INVALID, pkg.capi.ERR_UNSUPPORTED, pkg.capi.OK

    def scan(**kw):
        a = m.RecurrentScanArgs(**{**dict(B=1, T=1, H=4, G=2, D=8, V=8), **kw})
        return lib.l3ci_recurrent_scan(C.byref(a))

    assert scan(H=3) == bad and scan(kind=2) == bad and scan(kind=1) == bad and scan(D=257) == unsupported and scan() == bad and scan(B=0) == ok
    a = m.DeltaInputsArgs(B=1, T=1, H=2, G=2, D=8, V=8, taps=0, p_st=48, a_st=16)
    assert lib.l3ci_delta_inputs(C.byref(a)) == bad
    a.taps, a.p_st = 2, 47
    assert lib.l3ci_delta_inputs(C.byref(a)) == bad
    a.p_st, a.T = 48, 0
    assert lib.l3ci_delta_inputs(C.byref(a)) == ok
    r = m.ResidualNormArgs(x=fake, rows=2, width=8, reset=1)
    assert lib.l3ci_residual_norm(C.byref(r)) == bad
    r = m.ResidualNormArgs(x=fake, rows=2, width=8, y=fake, parts=0)
    assert lib.l3ci_residual_norm(C.byref(r)) == bad
    assert lib.l3ci_moe_route(fake, fake, fake, fake, fake, fake, 4, 3, 4, None) == bad       # four of three experts
    assert lib.l3ci_moe_route(fake, fake, fake, fake, fake, fake, 4, 5000, 4, None) == bad
    assert lib.l3ci_moe_gather(fake, fake, fake, fake, fake, fake, 0, 8, 4, 2, 0, None) == ok
    g = m.MoeGemmArgs(x=fake, w=fake, out=fake, counts=fake, rows=4, K=12, N=8, n_experts=2, variant=2)
    assert lib.l3ci_moe_gemm_variant(C.byref(g)) == -1 and lib.l3ci_moe_gemm(C.byref(g)) == unsupported     # rows of 24 bytes
    g.variant = 0
    assert lib.l3ci_moe_gemm_variant(C.byref(g)) == 1
    g.K = 16
    assert lib.l3ci_moe_gemm_variant(C.byref(g)) == 2
    g.dtype = 1
    assert lib.l3ci_moe_gemm_variant(C.byref(g)) == 1
    assert lib.l3ci_gated_act(fake, fake, 2, 0, 0.0, 1.0, 0, None) == bad and lib.l3ci_tanh(None, fake, 3, 0, None) == bad
    assert lib.l3ci_token_shift(fake, fake, fake, 4, fake, fake, 5, 2, 1, 8, 0, None) == bad
    assert lib.l3ci_qk_norm_cache(fake, 23, 8, 8, 8, fake, fake, 1e-5, fake, 8, 8, fake, 8, 8, 4, fake, 1, 1, 0, None) == bad
    t = m.AttnArgs(qa=fake, ka=fake, v=fake, out=fake, positions=fake, B=1, T=1, H=2, G=1, maps=2, Da=8, Dv=8, n_keys=4, window=3)
    assert lib.l3ci_mixer_attention_variant(C.byref(t)) == -1
    t.maps, t.window = 1, -1
    assert lib.l3ci_mixer_attention_variant(C.byref(t)) == -1


# ---- the oracle ------------------------------------------------------------------------------------------------
def test_oracle_sink_softmax_and_window():
    z = torch.tensor([[1.0, -2.0, 300.0], [-400.0, -500.0, 0.0]], dtype=torch.float64)
    seen = torch.tensor([[True, True, False], [True, True, False]])
    p = ref.sink_softmax(z, seen)
    assert torch.allclose(p[0, :2], torch.exp(z[0, :2]) / (1 + torch.exp(z[0, :2]).sum())) and p[0, 2] == 0
    assert p[1].sum() < 1e-100                                                       # all of it goes to the sink
    q = k = torch.zeros(12, 2, 4, dtype=torch.float64)
    v = torch.eye(12, dtype=torch.float64)[:, None].expand(12, 2, 12)
    o = ref.attention(q, k, v, 1.0, 4, 2)
    for h in range(2):
        s = 2.0 ** (-8.0 * (h + 1) / 2)
        for i in range(12):
            e = {j: math.exp(-s * (i - j)) for j in range(i + 1) if i - j < 4 or j < 2}
            for j in range(12):
                assert abs(o[i, h, j] - e.get(j, 0.0) / (1 + sum(e.values()))) < 1e-12


def test_oracle_scans_reduce_to_closed_forms():
    g = torch.Generator().manual_seed(0)
    T, H, D, V = 9, 2, 4, 3
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    decay = torch.rand(T, H, D, generator=g, dtype=torch.float64)
    # orthonormal keys, step size 1, no decay: the state answers every key with its value
    eye = torch.eye(D, dtype=torch.float64)[:, None].expand(D, H, D)
    o, S = ref.delta_scan(eye, eye, v[:D], torch.ones(D, H, D, dtype=torch.float64), torch.ones(D, H, dtype=torch.float64))
    assert torch.allclose(o, v[:D]) and torch.allclose(S.transpose(0, 1), v[:D].clone())
    # step size 0: nothing is ever written
    o, S = ref.delta_scan(q, k, v, decay, torch.zeros(T, H, dtype=torch.float64))
    assert o.abs().max() == 0 and S.abs().max() == 0
    # time mixing with the sum written out
    r, u = q, torch.randn(H, D, generator=g, dtype=torch.float64)
    vv = torch.randn(T, H, D, generator=g, dtype=torch.float64)
    o, _ = ref.wkv_scan(r, k, vv, decay, u)
    for t in range(T):
        for h in range(H):
            want = (r[t, h] * u[h] * k[t, h]).sum() * vv[t, h]
            for s in range(t):
                reach = decay[s + 1:t, h].prod(0) if s + 1 < t else torch.ones(D, dtype=torch.float64)
                want = want + (r[t, h] * reach * k[s, h]).sum() * vv[s, h]
            assert torch.allclose(o[t, h], want)


def test_oracle_convolution_and_router():
    x = torch.arange(8.0, dtype=torch.float64).view(4, 2)
    taps = torch.tensor([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]], dtype=torch.float64)
    y = ref.short_conv(x, taps)
    assert y[:, 1].tolist() == x[:, 1].tolist() and y[3, 0] == 100 * 6 + 10 * 4 + 2 and y[0, 0] == 0 and y[1, 0] == 200
    chosen, w = ref.route(torch.tensor([[0.0, 3.0, 1.0, 3.5]], dtype=torch.float64), 2)
    assert chosen.tolist() == [[3, 1]] and abs(w[0, 0] - 1 / (1 + math.exp(-0.5))) < 1e-12


@pytest.mark.parametrize("name", NAMES)
def test_oracle_is_causal(pkg, name):
    c = case(name)
    w = weights(pkg, c)
    toks = torch.randint(0, c["vocab"], (30,), generator=torch.Generator().manual_seed(1)).tolist()
    assert torch.allclose(ref.forward(c, w, toks)[:17], ref.forward(c, w, toks[:17]), atol=1e-9)
