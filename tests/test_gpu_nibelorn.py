"""The Nibelorn decoder through the framework's decode loop, against the plain float64 forward pass of oracle/nibelorn.py:
whole prompts layer by layer, decoding, portions, unequal batches, slots that are used again, generation."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from oracle import nibelorn as ref
from tests.nibelorn_cases import LIMIT, NAMES, case, row_errors, weights, write_model

pytestmark = pytest.mark.gpu
REPO = Path(__file__).resolve().parents[1]
DTYPES = (torch.float32, torch.bfloat16)


def make(pkg, device, name, dtype, max_batch=1, max_len=512, seed=3, ext=None):
    c = case(name)
    w = weights(pkg, c, seed)
    return pkg.nibelorn.NibelornDecoder(ext, pkg.nibelorn.config_from_json(c), device, max_batch, max_len, weights=w, dtype=dtype), c, w


def tokens_of(c, n, seed=0):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@pytest.fixture(scope="module")
def expected(pkg):
    """Logits and residual streams of the oracle, once per case and prompt."""
    known = {}

    def get(name, n, seed=0):
        if (name, n, seed) not in known:
            c = case(name)
            keep = []
            known[name, n, seed] = (ref.forward(c, weights(pkg, c, 3), tokens_of(c, n, seed), keep), keep)
        return known[name, n, seed]

    return get


def check(got, want, dtype, what=""):
    err = row_errors(got, want)
    assert err.max().item() < LIMIT[dtype], f"{what}: {err.max().item()} at place {err.argmax().item()}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("n", [1, 2, 63, 150])
def test_whole_prompt(pkg, device, expected, name, dtype, n):
    model, c, _ = make(pkg, device, name, dtype)
    check(model.extend("a", tokens_of(c, n), range(n)), expected(name, n)[0], dtype)


@pytest.mark.parametrize("name", NAMES)
def test_residual_stream_after_every_layer(pkg, device, expected, name):
    model, c, _ = make(pkg, device, name, torch.float32)
    toks = torch.tensor([tokens_of(c, 150)], device=device)
    at = torch.zeros(1, dtype=torch.int32, device=device)
    keep = []
    with torch.inference_mode():
        model.forward(toks, at, at + 150, keep=keep)
    assert len(keep) == len(c["layers"])
    for i, (x, want) in enumerate(zip(keep, expected(name, 150)[1])):
        assert x.dtype == torch.float32
        err = (x[0].double().cpu() - want).abs().max() / want.abs().max()
        assert err < 2e-5, (i, err)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("cuts", [[150], [1] * 20, [2] * 10, [100] + [1] * 30, [64, 2, 3, 64, 1, 7], [130, 20], [1, 2, 130, 1, 1], [65, 63, 10]])
def test_portions_and_decoding(pkg, device, expected, name, dtype, cuts):
    """However a prompt is cut, the logits are those of the whole."""
    n = sum(cuts)
    model, c, _ = make(pkg, device, name, dtype)
    toks, out, at = tokens_of(c, 150)[:n], [], 0
    for k in cuts:
        out.append(model.extend("a", toks[at:at + k], range(k)))
        at += k
    check(torch.cat(out), expected(name, 150)[0][:n], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_want_picks_places(pkg, device, dtype):
    model, c, _ = make(pkg, device, "mixed", dtype)
    toks = tokens_of(c, 40)
    every = model.extend("a", toks, range(40))
    model.finish("a")
    some = model.extend("b", toks, [0, 39, 7])
    assert torch.allclose(some.float(), every[[0, 39, 7]].float(), atol=2e-2 if dtype == torch.bfloat16 else 1e-4)
    assert model.extend("b", [1, 2], []) is None and model.cache.length("b") == 42


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_decode_batch(pkg, device, expected, name, dtype):
    """One decode step over slots at different positions equals each request alone."""
    lens = [1, 64, 149, 30]
    model, c, _ = make(pkg, device, name, dtype, max_batch=len(lens))
    toks = tokens_of(c, 150)
    for i, n in enumerate(lens):
        model.extend(i, toks[:n])
    assert [model.cache.slot(i) for i in range(len(lens))] == [0, 1, 2, 3]
    positions = torch.tensor(lens, dtype=torch.int32, device=device)
    with torch.inference_mode():
        logits = model.forward(torch.tensor([[toks[n]] for n in lens], device=device), positions, positions + 1)
    check(logits, expected(name, 150)[0][lens], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_are_used_again(pkg, device, expected, dtype):
    """A request in a slot that longer ones have held before gives bit for bit what it gives in a fresh cache."""
    model, c, _ = make(pkg, device, "wide", dtype, max_batch=2, max_len=200)
    toks, other = tokens_of(c, 150), tokens_of(c, 190, seed=9)
    first = model.extend("first", toks, range(150))
    model.finish("first")
    for r in ("x", "y"):
        model.extend(r, other)
    with pytest.raises(RuntimeError, match="no free slot"):
        model.extend("z", [1])
    model.finish("x")
    again = model.extend("again", toks, range(150))
    assert torch.equal(first, again)
    with pytest.raises(RuntimeError, match="do not fit"):
        model.extend("again", toks)
    check(again, expected("wide", 150)[0], dtype)


def test_a_refused_token_changes_nothing(pkg, device):
    model, c, _ = make(pkg, device, "thin", torch.bfloat16)
    with pytest.raises(ValueError, match="vocabulary"):
        model.extend("a", [1, c["vocab"]])
    assert model.cache.length("a") == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_key_decides(pkg, device, dtype):
    """The last query's best key is the first token (made so in the weights' favour: its embedding equals the query
    token's, scaled): changing that token changes the last logits by far more than rounding, also when it lies in
    another portion and the query is decoded."""
    name, n = "wide", 140
    c = case(name)
    w = weights(pkg, c, 3, gain=6.0)
    model = pkg.nibelorn.NibelornDecoder(None, pkg.nibelorn.config_from_json(c), device, 1, 256, weights=w, dtype=dtype)
    toks = tokens_of(c, n)
    other = [(toks[0] + 1) % c["vocab"]] + toks[1:]
    outs = []
    for seq in (toks, other):
        want = ref.forward(c, w, seq)[-1:]
        whole = model.extend("w", seq, [n - 1])
        model.finish("w")
        model.extend("d", seq[:70])
        model.extend("d", seq[70:-1])
        decoded = model.extend("d", seq[-1:], [0])
        model.finish("d")
        for got in (whole, decoded):
            err = row_errors(got, want).item()
            assert err < 2 * LIMIT[dtype], err
        outs.append(want)
    assert row_errors(outs[0], outs[1]).item() > 0.02


# ---- generation through the framework's loop ---------------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_greedy_generation(pkg, ext, device, name):
    """Long decoding: graph replay equals the eager loop; every token is the oracle's choice given the tokens before it,
    wherever the oracle's logits leave a clear winner."""
    B, P, G = 3, 40, 150
    model, c, w = make(pkg, device, name, torch.bfloat16, max_batch=B, max_len=P + G, ext=ext)
    prompts = torch.tensor([tokens_of(c, P, seed=s) for s in range(B)], device=device)
    graph = model.generate(prompts, G)
    eager = model.generate(prompts, G, use_graph=False)
    torch.cuda.synchronize()
    assert torch.equal(graph, eager)
    checked = 0
    for b in range(B):
        seq = prompts[b].tolist() + graph[b].tolist()
        logits = ref.forward(c, w, seq)[P - 1:-1]
        top = logits.topk(2, dim=-1).values
        clear = (top[:, 0] - top[:, 1]) > 0.25 * logits.std()
        assert torch.equal(logits.argmax(-1)[clear], graph[b].cpu()[clear])
        checked += int(clear.sum())
    assert checked > B * G // 4


def test_prompt_and_batch_do_not_matter_to_generation(pkg, ext, device):
    """A prompt long enough for the tensor-core prefill kernels, generated alone and in a batch: fp32, so that no near
    tie is decided by rounding."""
    P, G = 160, 12
    model, c, w = make(pkg, device, "wide", torch.float32, max_batch=2, max_len=P + G, ext=ext)
    prompts = torch.tensor([tokens_of(c, P, seed=s) for s in (4, 5)], device=device)
    both = model.generate(prompts, G)
    for b in range(2):
        alone = model.generate(prompts[b:b + 1], G)
        assert torch.equal(alone[0], both[b])


def test_sampled_generation(pkg, ext, device):
    model, c, _ = make(pkg, device, "mixed", torch.bfloat16, max_batch=2, max_len=80, ext=ext)
    prompts = torch.tensor([tokens_of(c, 20, seed=s) for s in range(2)], device=device)
    a, b = (model.generate(prompts, 30, temperature=0.8, top_p=0.9, seed=s) for s in (1, 2))
    again = model.generate(prompts, 30, temperature=0.8, top_p=0.9, seed=1, use_graph=False)
    assert torch.equal(a, again) and not torch.equal(a, b)


# ---- the registry, a model folder and the trace runner ----------------------------------------------------------
def test_load_model_from_a_folder(pkg, device, expected, tmp_path):
    c = case("mixed")
    write_model(tmp_path, c, weights(pkg, c, 3))
    model = pkg.models.load_model(tmp_path, device, max_batch=1, max_len=200)
    assert isinstance(model, pkg.nibelorn.NibelornDecoder) and model.dtype == torch.bfloat16
    check(model.extend("a", tokens_of(c, 150), range(150)), expected("mixed", 150)[0], torch.bfloat16)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run(pkg, device, expected, tmp_path, dtype):
    import numpy as np

    c = case("wide")
    folder, out = tmp_path / "m", tmp_path / "o"
    folder.mkdir()
    out.mkdir()
    write_model(folder, c, weights(pkg, c, 3))
    toks = tokens_of(c, 150)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:140], "want": [0, 139, 5]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[140:142], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[142:143], "want": [0]}], "end": ["a"]},
             {"step": 7, "entries": [{"id": "b", "tokens": toks, "want": [149]}], "end": ["b"]}]
    res = subprocess.run([str(REPO / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                          "--max-tokens", "150"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                         text=True, timeout=300, env=dict(os.environ, PATH=str(Path(sys.executable).parent) + ":" + os.environ["PATH"]))
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32", "7.f32"]
    want = expected("wide", 150)[0]
    for step, places in ((0, [0, 139, 5]), (2, [142]), (7, [149])):
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").copy()).view(len(places), c["vocab"])
        check(got, want[places], getattr(torch, dtype), step)


def test_llama_takes_prompts_in_portions(pkg, ext, device):
    """The shared loop's portions on the Llama-3 decoder: however a prompt is cut, the logits are those of the whole, up
    to bf16 rounding."""
    cfg = pkg.decode_loop.DecoderConfig(vocab_size=500, n_layer=2, n_head=8, n_kv_head=2, n_embd=512, hidden_dim=768)
    model = pkg.decode_loop.Llama3Decoder(ext, cfg, device, max_batch=2, max_len=256, seed=2)
    toks = torch.randint(0, 500, (200,), generator=torch.Generator().manual_seed(0)).tolist()
    whole = model.extend("w", toks, range(200))
    out, at = [], 0
    for k in (64, 2, 1, 130, 1, 1, 1):
        out.append(model.extend("p", toks[at:at + k], range(k)))
        at += k
    assert row_errors(torch.cat(out), whole.cpu()).max() < 4e-2
    with pytest.raises(NotImplementedError):
        pkg.decode_loop.Llama3Decoder(ext, cfg, device, 1, 16, dtype=torch.float32)
