"""What needs no GPU of the Nibelorn decoder and the framework around it: configuration, registry, checkpoint reading, the
cache's slots, the rotation table, the C ABI of the mixer kernels, and the oracle against itself."""
import ctypes as C
import math
import re
from pathlib import Path

import pytest
import torch

from oracle import nibelorn as ref
from tests.nibelorn_cases import NAMES, case, weights, write_model

REPO = Path(__file__).resolve().parents[1]


def test_configuration_reads_every_key(pkg):
    nb = pkg.nibelorn
    cfg = nb.config_from_json(case("mixed"))
    assert (cfg.vocab_size, cfg.width, cfg.eps) == (211, 104, 1e-4)
    assert [l.weights for l in cfg.layers] == [0, 1, 2, 1, 0, 2]
    assert [l.ff for l in cfg.layers] == [72, 128, None, 128, 72, None]
    a, m = cfg.layers[2].mixer, cfg.layers[1].mixer
    assert a == nb.DifferentialAttention(heads=4, kv_heads=4, dim=8, vdim=16, scale=8 ** -0.5, diff=0.7, softcap=4.0, temp_coef=1.1,
                                         temp_every=3.0)
    assert m == nb.LatentAttention(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=56, scale=32 ** -0.5, rot_base=500.0)
    assert m.planes == {"latent": (64,)} and a.planes == {"k": (4, 16), "v": (4, 16)}


def test_configuration_refuses_what_it_does_not_know(pkg):
    read = pkg.nibelorn.config_from_json
    for change in (lambda c: c["layers"][0].update(type="recurrence"), lambda c: c["layers"][0]["mlp"].update(kind="experts"),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), lambda c: c["layers"][0].update(weights_of=4)):
        c = case("mixed")
        change(c)
        with pytest.raises(ValueError):
            read(c)


def test_weights_follow_chains_of_borrowed_layers(pkg):
    c = case("thin")
    c["layers"][1]["weights_of"] = 2          # layer 1 borrows from layer 2, which now owns the tensors
    del c["layers"][2]["weights_of"]
    c["layers"].append(dict(c["layers"][1], weights_of=1))
    assert [l.weights for l in pkg.nibelorn.config_from_json(c).layers] == [0, 2, 2, 2]


def test_borrowed_layers_have_no_tensors(pkg):
    shapes = pkg.nibelorn.tensor_shapes(pkg.nibelorn.config_from_json(case("mixed")))
    assert {n.split(".")[0] for n in shapes} == {"embed", "head", "final", "l0", "l1", "l2"}
    assert "l2.norm2" not in shapes and "l2.mlp.up" not in shapes and shapes["l1.mix.dkv"] == (64, 104)


def test_registry(pkg, tmp_path):
    models = pkg.models
    assert models.architecture_of({"architecture": "Nibelorn"}).decoder is pkg.nibelorn.NibelornDecoder
    assert models.architecture_of({"architectures": ["LlamaForCausalLM"]}).decoder is pkg.decode_loop.Llama3Decoder
    with pytest.raises(ValueError, match="no decoder"):
        models.architecture_of({"architectures": ["Other"]})
    (tmp_path / "config.json").write_text('{"architectures": ["LlamaForCausalLM"]}')
    with pytest.raises(NotImplementedError):
        models.load_model(tmp_path, "cpu", 1, 16, dtype=torch.float32)
    llama = {"vocab_size": 100, "num_hidden_layers": 2, "num_attention_heads": 4, "num_key_value_heads": 2, "hidden_size": 256,
             "intermediate_size": 512, "rms_norm_eps": 1e-5, "rope_theta": 1e6}
    cfg = models.ARCHITECTURES["LlamaForCausalLM"].read_config(llama)
    assert (cfg.n_layer, cfg.n_kv_head, cfg.rope_theta, cfg.rope_scaled) == (2, 2, 1e6, False)


@pytest.mark.parametrize("name", NAMES)
def test_model_folder_round_trip(pkg, tmp_path, name):
    c = case(name)
    w = dict(weights(pkg, c), extra=torch.arange(5, dtype=torch.int32), more=torch.randn(3, 2), empty=torch.empty(0, 4))
    write_model(tmp_path, c, w)
    assert pkg.checkpoint.read_config(tmp_path) == c
    got = pkg.checkpoint.read_weights(tmp_path)
    assert got.keys() == w.keys()
    for k in w:
        assert got[k].dtype == w[k].dtype and got[k].shape == w[k].shape and torch.equal(got[k], w[k]), k
    try:
        from safetensors.torch import load_file
    except ImportError:
        return
    theirs = load_file(tmp_path / "model.safetensors")
    assert all(torch.equal(theirs[k], w[k]) for k in w)


def test_a_broken_checkpoint_is_refused(pkg, tmp_path):
    write_model(tmp_path, {}, {"a": torch.zeros(4, 4)})
    raw = (tmp_path / "model.safetensors").read_bytes()
    (tmp_path / "model.safetensors").write_bytes(raw[:-8])
    with pytest.raises(ValueError):
        pkg.checkpoint.read_weights(tmp_path)


def test_cache_slots(pkg):
    cache = pkg.kv_cache.StaticCache([{"k": (2, 4), "v": (2, 6)}, {"latent": (8,)}], 2, 5, torch.float32, "cpu")
    assert [{n: tuple(t.shape) for n, t in l.items()} for l in cache.layers] == [
        {"k": (2, 5, 2, 4), "v": (2, 5, 2, 6)}, {"latent": (2, 5, 8)}]
    assert cache.slot("a") == 0 and cache.slot("b") == 1 and cache.slot("a") == 0
    cache.advance("a", 3)
    assert cache.length("a") == 3 and cache.length("b") == 0 and cache.length("nobody") == 0
    with pytest.raises(RuntimeError):
        cache.slot("c")
    cache.release("a")
    cache.release("nobody")
    assert cache.slot("c") == 0 and cache.length("c") == 0


def test_rotation_table_rotates_like_the_oracle(pkg):
    for dims, base in ((2, 10000.0), (6, 77.0), (64, 5e5)):
        table = pkg.rope_table.rotation_table(dims, 3000, base).double().view(3000, dims // 2, 2)
        pos = torch.tensor([0, 1, 511, 2999])
        x = torch.randn(4, dims, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
        c, s = table[pos, :, 0], table[pos, :, 1]
        u, v = x[:, :dims // 2], x[:, dims // 2:]
        got = torch.cat([u * c - v * s, v * c + u * s], dim=-1)
        assert (got - ref.rotate_half(x, pos, base)).abs().max() < 1e-6


# ---- the C ABI --------------------------------------------------------------------------------------------------
def test_mixer_header_and_binding_agree(pkg):
    text = (REPO / "include" / "l3ci_mixers.h").read_text()
    declared = set(re.findall(r"L3CI_API\s+[\w\s\*]+?\b(l3ci_\w+)\s*\(", text))
    assert declared == set(pkg.mixers.EXPORTS)
    lib = pkg.mixers.load()
    assert all(hasattr(lib, n) for n in declared)
    names = re.findall(r"\b(\w+)(?=[,;])", text[text.index("typedef struct l3ci_mixer_attn_args"):text.index("} l3ci_mixer_attn_args")].replace("*", " "))
    fields = [n.rstrip("_") for n, _ in pkg.mixers.AttnArgs._fields_]
    assert [n for n in names if n in fields] == fields   # same members, same order
    assert C.sizeof(pkg.mixers.AttnArgs) == 11 * 8 + 20 * 8 + 15 * 4 + 8 * 4 + 4 + 8


def test_mixer_arguments_are_validated_before_cuda(pkg):
    lib, capi = pkg.mixers.load(), pkg.capi
    fake = C.c_void_p(0x1000)   # never dereferenced
    assert lib.l3ci_gelu(fake, fake, -1, 0, None) == capi.ERR_INVALID
    assert lib.l3ci_gelu(fake, fake, 8, 7, None) == capi.ERR_INVALID
    assert lib.l3ci_gelu(None, None, 0, 0, None) == capi.OK
    assert lib.l3ci_add_dyn_tanh(None, None, None, 0, None, fake, fake, 1.0, fake, 2, 8, 0, None) == capi.ERR_INVALID
    assert lib.l3ci_latent_cache(fake, 10, fake, 4, fake, 1e-5, fake, 64, 8, 8, fake, 1, 1, 2, 8, 3, 4, 0, None) == capi.ERR_INVALID
    a = pkg.mixers.AttnArgs()
    a.qa = a.ka = a.v = a.out = a.positions = 0x1000
    a.B, a.T, a.H, a.G, a.maps, a.Da, a.Dv, a.n_keys, a.start_pos = 1, 1, 6, 4, 1, 16, 16, 8, -1
    assert lib.l3ci_mixer_attention(C.byref(a)) == capi.ERR_INVALID      # 6 heads over 4
    a.G, a.maps, a.Db = 2, 2, 8
    assert lib.l3ci_mixer_attention(C.byref(a)) == capi.ERR_UNSUPPORTED  # two maps have one key part
    a.maps, a.Db, a.B = 1, 0, 0
    assert lib.l3ci_mixer_attention(C.byref(a)) == capi.OK               # empty batch
    assert lib.l3ci_mixer_attention(None) == capi.ERR_INVALID


def attn_args(pkg, **kw):
    a = pkg.mixers.AttnArgs()
    a.qa = a.ka = a.v = a.out = a.positions = a.qb = a.kb = 0x10000
    a.B, a.T, a.H, a.G, a.maps, a.Da, a.Db, a.Dv, a.n_keys, a.start_pos, a.scale = 1, 1, 6, 1, 1, 72, 24, 56, 4096, -1, 0.1
    for n in ("qa", "qb", "ka", "kb", "v", "o"):
        for ax in ("sb", "st", "sh"):
            setattr(a, f"{n}_{ax}", 1024)
    a.kb = a.ka + 2 * a.Da
    for k, v in kw.items():
        setattr(a, k, v)
    return a


def test_which_attention_kernel_runs(pkg):
    lib = pkg.mixers.load()
    choice = lambda **kw: lib.l3ci_mixer_attention_variant(C.byref(attn_args(pkg, **kw)))  # noqa: E731
    M = pkg.mixers
    assert choice() == M.MMA
    assert choice(dtype=1) == M.ROWS                                  # 32-bit: the plain kernel
    assert choice(Da=60, kb=0x10000 + 120) == M.ROWS                  # rows of 120 bytes
    assert choice(qa_st=1020) == M.ROWS
    assert choice(kb=0x20000) == M.ROWS                               # two key rows: only a prompt's kernel reads those
    assert choice(kb=0x20000, T=128, start_pos=0) == M.TC
    assert choice(T=128, start_pos=0) == M.TC and choice(T=127, start_pos=0) == M.MMA
    assert choice(T=128, start_pos=4000) == M.MMA                     # does not fit the keys given
    assert choice(maps=2, Db=0, Da=48, T=200, start_pos=0, softcap=5.0) == M.TC
    assert choice(maps=2, Db=0, Da=72, T=200, start_pos=0) == M.MMA   # the prompt kernel's tile of a map is 64 columns
    assert choice(variant=M.TC, dtype=1) == -1


# ---- the oracle against itself -----------------------------------------------------------------------------------
def test_oracle_latent_attention_equals_its_absorbed_form():
    """Keys and values folded into the query and the output give the same numbers."""
    g = torch.Generator().manual_seed(0)
    H, D, R, V, Cn, E, T, eps = 3, 8, 4, 6, 10, 12, 9, 1e-5
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    w = {"q": r(H * (D + R), E), "dkv": r(Cn + R, E), "dkv.norm": r(Cn), "uk": r(H * D, Cn), "uv": r(H * V, Cn), "o": r(E, H * V)}
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": V, "kv_rank": Cn, "scale": 0.3, "rot": {"base": 100.0}}
    h, pos = r(T, E), torch.arange(T)
    want = ref.latent_attention(h, w, m, eps)
    q, down = (h @ w["q"].T).view(T, H, D + R), h @ w["dkv"].T
    c = ref.rms(down[:, :Cn], eps) * w["dkv.norm"]
    rows = torch.cat([c, ref.rotate_half(down[:, Cn:], pos, 100.0)], dim=-1)
    q_lat = torch.einsum("thd,hdc->thc", q[..., :D], w["uk"].view(H, D, Cn))
    full = torch.cat([q_lat, ref.rotate_half(q[..., D:], pos, 100.0)], dim=-1)
    o = ref.cached_attention(full, rows[:, None], c[:, None], 0, 0.3)
    got = torch.einsum("thc,hvc->thv", o, w["uv"].view(H, V, Cn)).reshape(T, H * V) @ w["o"].T
    assert (got - want).abs().max() < 1e-10


def test_oracle_mechanisms_by_hand():
    x = torch.tensor([3.0, -4.0], dtype=torch.float64)
    assert torch.allclose(ref.rms(x, 0.0), x / math.sqrt(12.5))
    assert ref.query_temperature(torch.tensor([0, 18, 19, 39]), 0.5, 20).tolist() == pytest.approx(
        [1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)])
    assert float(ref.softcap(torch.tensor(1e9, dtype=torch.float64), 7.0)) == 7.0
    assert float(ref.gelu(torch.tensor(1.0, dtype=torch.float64))) == pytest.approx(0.8413447460685429)
    a = ref.rotate_half(torch.tensor([[1.0, 0.0]], dtype=torch.float64), torch.tensor([1]), 10.0)[0].tolist()
    assert a == pytest.approx([math.cos(1), math.sin(1)])
    assert ref.dyn_tanh(torch.tensor([0.5], dtype=torch.float64), torch.tensor([2.0]), torch.tensor([1.0]), torch.tensor(3.0)).tolist() == \
        pytest.approx([2 * math.tanh(1.5) + 1])


@pytest.mark.parametrize("name", NAMES)
def test_oracle_is_causal(pkg, name):
    """A prefix's logits do not depend on what follows; every place depends on the first token."""
    c = case(name)
    w = weights(pkg, c)
    toks = [i * 7 % c["vocab"] for i in range(20)]
    whole = ref.forward(c, w, toks)
    assert (ref.forward(c, w, toks[:11]) - whole[:11]).abs().max() < 1e-9
    other = ref.forward(c, w, [toks[0] + 1] + toks[1:])
    assert ((other - whole).abs().amax(-1) > 1e-6).all()
