"""The Rupotar decoder through the framework's decode loop, against the plain float64 forward pass of oracle/rupotar.py: whole
prompts layer run by layer run, decoding, portions, unequal batches, slots that are used again, windows, generation."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from oracle import rupotar as ref
from tests.rupotar_cases import LIMIT, NAMES, attention, case, config, delta, dense, row_errors, weights, wkv, write_model

pytestmark = pytest.mark.gpu
REPO = Path(__file__).resolve().parents[1]
DTYPES = (torch.float32, torch.bfloat16)


def make(pkg, device, name, dtype, max_batch=1, max_len=512, seed=3, ext=None):
    c = case(name, smooth=dtype == torch.bfloat16)
    w = weights(pkg, c, seed)
    return pkg.rupotar.RupotarDecoder(ext, pkg.rupotar.config_from_json(c), device, max_batch, max_len, weights=w, dtype=dtype), c, w


def tokens_of(c, n, seed=0):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


@pytest.fixture(scope="module")
def expected(pkg):
    """Logits and residual streams of the oracle, once per case and prompt."""
    known = {}

    def get(name, n, dtype, seed=0):
        key = name, n, dtype == torch.bfloat16, seed
        if key not in known:
            c = case(name, smooth=key[2])
            keep = []
            known[key] = (ref.forward(c, weights(pkg, c, 3), tokens_of(c, n, seed), keep), keep)
        return known[key]

    return get


def check(got, want, dtype, what=""):
    """bf16: a recurrent head whose output nearly cancels has its rounding blown up by its norm, so single places go further."""
    err = row_errors(got, want)
    assert err.mean().item() < LIMIT[dtype], f"{what}: {err.mean().item()} on average"
    assert err.max().item() < (2.5 if dtype == torch.bfloat16 else 1) * LIMIT[dtype], f"{what}: {err.max().item()} at place {err.argmax().item()}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("n", [1, 2, 63, 170])
def test_whole_prompt(pkg, device, expected, name, dtype, n):
    model, c, _ = make(pkg, device, name, dtype)
    check(model.extend("a", tokens_of(c, 170)[:n], range(n)), expected(name, 170, dtype)[0][:n], dtype)


@pytest.mark.parametrize("name", NAMES)
def test_residual_stream_after_every_layer_run(pkg, device, expected, name):
    model, c, _ = make(pkg, device, name, torch.float32)
    toks = torch.tensor([tokens_of(c, 170)], device=device)
    at = torch.zeros(1, dtype=torch.int32, device=device)
    keep = []
    with torch.inference_mode():
        model.forward(toks, at, at + 170, keep=keep)
    assert len(keep) == len(model.runs) == len(model.cache.layers)
    for i, (x, want) in enumerate(zip(keep, expected(name, 170, torch.float32)[1])):
        assert x.dtype == torch.float32
        err = (x[0].double().cpu() - want).abs().max() / want.abs().max()
        assert err < 2e-5, (i, err)


CUTS = [[170], [1] * 24, [2] * 12, [100] + [1] * 40, [64, 2, 3, 64, 1, 7, 2, 16, 11], [130, 40], [1, 2, 130, 1, 1], [15, 1, 16, 17, 33, 2, 31],
        [3] * 20 + [1] * 30]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("cuts", CUTS, ids=lambda c: f"{len(c)}x{max(c)}")
def test_portions_and_decoding(pkg, device, expected, name, dtype, cuts):
    """However a prompt is cut, the logits are those of the whole."""
    n = sum(cuts)
    model, c, _ = make(pkg, device, name, dtype)
    toks, out, at = tokens_of(c, 170)[:n], [], 0
    for k in cuts:
        out.append(model.extend("a", toks[at:at + k], range(k)))
        at += k
    check(torch.cat(out), expected(name, 170, dtype)[0][:n], dtype)


@pytest.mark.parametrize("name", ["mixed", "wide", "order"])
def test_long_decoding(pkg, device, expected, name):
    """Token by token far past every window, in 32-bit: no drift."""
    model, c, _ = make(pkg, device, name, torch.float32)
    toks = tokens_of(c, 400)
    out = [model.extend("a", toks[:30], range(30))] + [model.extend("a", [t], [0]) for t in toks[30:]]
    check(torch.cat(out), expected(name, 400, torch.float32)[0], torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_unequal_requests_in_one_decode_batch(pkg, device, expected, name, dtype):
    """Decode steps over slots at different positions equal each request alone; a request at position 0 starts from zero
    whatever its slot holds."""
    lens = [1, 64, 149, 30, 0]
    model, c, _ = make(pkg, device, name, dtype, max_batch=len(lens))
    toks = tokens_of(c, 170)
    model.extend("old", toks[:60])                                     # leaves state behind in the slot that is taken last
    model.finish("old")
    order = [4, 0, 1, 2, 3]
    for i in order[1:]:
        model.extend(i, toks[:lens[i]])
    slots = [model.cache.slot(i) for i in range(4)]
    positions = torch.zeros(5, dtype=torch.int32, device=device)
    tokens = torch.zeros(5, 1, dtype=torch.int64, device=device)
    last = ({0, 1, 2, 3, 4} - set(slots)).pop()
    at = {s: lens[i] for i, s in enumerate(slots)}
    at[last] = 0
    model.cache.layers[1]["state"][last].fill_(float("nan")) if "state" in model.cache.layers[1] else None
    for step in range(3):
        for s, n in at.items():
            positions[s], tokens[s, 0] = n + step, toks[n + step]
        with torch.inference_mode():
            logits = model.forward(tokens, positions, positions + 1)
        want = torch.stack([expected(name, 170, dtype)[0][at[s] + step] for s in range(5)])
        check(logits, want, dtype, step)


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_chosen_experts_in_bf16(pkg, device, name):
    """The models as they are: a token whose experts are a close call may take others in bf16 (and change what follows), most
    tokens do not."""
    c = case(name)
    w = weights(pkg, c, 3)
    model = pkg.rupotar.RupotarDecoder(None, pkg.rupotar.config_from_json(c), device, 1, 200, weights=w)
    toks = tokens_of(c, 170)
    err = row_errors(torch.cat([model.extend("a", toks[:140], range(140)), *(model.extend("a", [t], [0]) for t in toks[140:])]),
                     ref.forward(c, w, toks))
    assert err.median() < LIMIT[torch.bfloat16] and err[:6].max() < 6 * LIMIT[torch.bfloat16], err


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_of_equal_prompts(pkg, device, expected, dtype):
    model, c, _ = make(pkg, device, "mixed", dtype, max_batch=3)
    toks = [tokens_of(c, 170, seed=s) for s in range(3)]
    at = torch.zeros(3, dtype=torch.int32, device=device)
    with torch.inference_mode():
        logits = model.forward(torch.tensor(toks, device=device), at, at + 170, want=list(range(170)))
    for b in range(3):
        check(logits[b], expected("mixed", 170, dtype, b)[0], dtype, b)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["wide", "mixed"])
def test_slots_are_used_again(pkg, device, expected, name, dtype):
    """A request in a slot that longer ones have held before gives what it gives in a fresh cache."""
    model, c, _ = make(pkg, device, name, dtype, max_batch=2, max_len=200)
    toks, other = tokens_of(c, 170), tokens_of(c, 190, seed=9)
    first = model.extend("first", toks, range(170))
    model.finish("first")
    for r in ("x", "y"):
        model.extend(r, other)
    with pytest.raises(RuntimeError, match="no free slot"):
        model.extend("z", [1])
    model.finish("x")
    again = model.extend("again", toks, range(170))
    assert torch.equal(first, again)
    model.finish("again")
    one = [model.extend("third", [t], [0]) for t in toks[:40]]
    check(torch.cat(one), expected(name, 170, dtype)[0][:40], dtype)
    with pytest.raises(RuntimeError, match="do not fit"):
        model.extend("third", other)


# ---- the window's edges, the first tokens, far tokens through the recurrences ---------------------------------------
def probe_config(kind):
    """One layer (and a last one without mixing to speak of): the place a token is seen from is the layer's alone."""
    layer = {"window": attention(4, 2, 32, 16, 40, 6, gain=1.5, mlp=dense(32)), "delta": delta(4, 2, 32, 16, 4, mlp=dense(32)),
             "wkv": wkv(3, 32, mlp=dense(32))}[kind]
    return config(64, 150, [layer], scale=4.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
def test_every_border_of_the_window_shows(pkg, device, dtype, decoded):
    """Query 139 of one windowed layer: a change of token j changes its logits exactly when j is in the window (100..139) or
    among the kept first tokens (0..5), prompt or decoded; otherwise they stay (in 32-bit to the bit)."""
    c = probe_config("window")
    w = weights(pkg, c, 5)
    # a query and key that match across tokens: every score is large, so that distance alone does not hide a key
    w["l0.mix.k"] = w["l0.mix.q"][:w["l0.mix.k"].shape[0]].clone()
    model = pkg.rupotar.RupotarDecoder(None, pkg.rupotar.config_from_json(c), device, 1, 256, weights=w, dtype=dtype)
    toks, n = tokens_of(c, 140), 140

    def last(seq):
        if decoded:
            model.extend("a", seq[:-1])
            out = model.extend("a", seq[-1:], [0])
        else:
            out = model.extend("a", seq, [n - 1])
        model.finish("a")
        return out

    base, want0 = last(toks), ref.forward(c, w, toks)[-1:]
    assert row_errors(base, want0).item() < LIMIT[dtype]
    for j in (0, 4, 5, 6, 7, 50, 98, 99, 100, 101, 127, 128, 138):
        seq = list(toks)
        seq[j] = (seq[j] + 75) % 150
        got, want = last(seq), ref.forward(c, w, seq)[-1:]
        seen = j < 6 or j >= 100
        assert (row_errors(want, want0).item() > 0) == seen, j
        if dtype == torch.float32:
            assert torch.equal(got, base) != seen, j
        elif not seen:
            assert row_errors(got, base.cpu()).item() < 0.2 * LIMIT[dtype], j
        assert row_errors(got, want).item() < LIMIT[dtype], j


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["delta", "wkv"])
def test_a_far_token_is_remembered(pkg, device, dtype, kind):
    """With decays near one, a change of the first token moves the last logits by more than rounding, also over portions."""
    c = probe_config(kind)
    w = weights(pkg, c, 6)
    for name in w:
        if name.endswith((".A_log", ".w0")):
            w[name] = torch.full_like(w[name], -9.0)
        elif name.endswith("mix.b"):
            w[name] = w[name] * 0.2
    model = pkg.rupotar.RupotarDecoder(None, pkg.rupotar.config_from_json(c), device, 1, 256, weights=w, dtype=dtype)
    toks = tokens_of(c, 24)
    other = [(toks[0] + 1) % 150] + toks[1:]
    wants = [ref.forward(c, w, s)[-1:] for s in (toks, other)]
    moved = row_errors(wants[0], wants[1]).item()
    assert moved > 0.02
    for seq, want in zip((toks, other), wants):
        outs = [model.extend("w", seq, [23])]
        model.finish("w")
        for cut in ([10, 13, 1], [2] * 11 + [1, 1], [1] * 24):
            at = 0
            for k in cut:
                out = model.extend("p", seq[at:at + k], [k - 1])
                at += k
            model.finish("p")
            outs.append(out)
        for out in outs:
            assert row_errors(out, want).item() < min(LIMIT[dtype], moved)


# ---- generation through the framework's loop ---------------------------------------------------------------------
@pytest.mark.parametrize("name", ["mixed", "wide", "order"])
def test_greedy_generation(pkg, ext, device, name):
    """Graph replay equals the eager loop; every token is the oracle's choice given the tokens before it, wherever the
    oracle's logits leave a clear winner; a second generation starts from zero."""
    B, P, G = 3, 40, 100
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
    assert checked > B * G // 8


def test_prompt_and_batch_do_not_matter_to_generation(pkg, ext, device):
    """fp32, so that no near tie is decided by rounding."""
    P, G = 160, 12
    model, c, w = make(pkg, device, "wide", torch.float32, max_batch=2, max_len=P + G, ext=ext)
    prompts = torch.tensor([tokens_of(c, P, seed=s) for s in (4, 5)], device=device)
    both = model.generate(prompts, G)
    for b in range(2):
        alone = model.generate(prompts[b:b + 1], G)
        assert torch.equal(alone[0], both[b])


# ---- the registry, a model folder and the trace runner ----------------------------------------------------------
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run(pkg, device, expected, tmp_path, dtype):
    import numpy as np

    c = case("mixed", smooth=dtype == "bfloat16")
    folder, out = tmp_path / "m", tmp_path / "o"
    folder.mkdir()
    out.mkdir()
    write_model(folder, c, weights(pkg, c, 3))
    toks = tokens_of(c, 170)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:140], "want": [0, 139, 5]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[140:142], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[142:143], "want": [0]}], "end": ["a"]},
             {"step": 7, "entries": [{"id": "b", "tokens": toks, "want": [149]}], "end": ["b"]}]
    res = subprocess.run([str(REPO / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                          "--max-tokens", "170"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                         text=True, timeout=300, env=dict(os.environ, PATH=str(Path(sys.executable).parent) + ":" + os.environ["PATH"]))
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    want = expected("mixed", 170, getattr(torch, dtype))[0]
    for step, places in ((0, [0, 139, 5]), (2, [142]), (7, [149])):
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").copy()).view(len(places), c["vocab"])
        check(got, want[places], getattr(torch, dtype), step)
