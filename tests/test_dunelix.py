"""Dunelix end to end against a plain float64 implementation: prompts, portions, decoding, batches, slots, generation, the
model folder, the trace runner and the command line. Every check runs on the CPU backend and, marked `gpu`, on the kernels in
32-bit and bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import dunelix_cases as C
import plain_dunelix as plain

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BACKENDS = [("cpu", "float32"), ("cpu", "bfloat16"), pytest.param(("cuda", "float32"), marks=pytest.mark.gpu),
            pytest.param(("cuda", "bfloat16"), marks=pytest.mark.gpu)]


@pytest.fixture(params=BACKENDS, ids=lambda b: "-".join(b))
def backend(request):
    return request.param


def run(gen, tokens, cuts, req="r"):
    """Logits at all positions with the tokens cut into portions of the given sizes (the last size repeats)."""
    gen.admit(req)
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(cuts[min(k, len(cuts) - 1)], len(tokens) - at)
        out.append(gen.step({req: tokens[at:at + n]}, {req: range(n)})[req])
        at, k = at + n, k + 1
    gen.release(req)
    return np.concatenate(out)


@pytest.mark.parametrize("case", sorted(C.CASES))
def test_prompt_portions_and_decoding(case, backend):
    """Whole prompts, token by token, and portions of many sizes give the same logits as the oracle; every position of the
    prompt is compared, so the edges of every chunk and the first tokens are among them. The slot is used again and again."""
    cfg = C.CASES[case]
    ckpt, tokens = C.checkpoint(cfg), C.prompt(cfg, 61)
    want = C.oracle_logits(cfg, ckpt, tokens)
    gen = C.generator(cfg, ckpt, *backend)
    for cuts in ([61], [1], [2], [40, 1], [3, 5, 17, 2, 1, 19, 8], [33, 28]):
        assert C.error(run(gen, tokens, cuts), want) < C.TOLERANCE[backend[1]], cuts


def test_long_prompt_and_long_decoding(backend):
    """Several blocks of every kernel: hundreds of positions, chunks longer than a tile, then a long decoded tail."""
    cfg = C.config([C.layer({"width": 72}, 64), C.layer(C.attention(heads=6, kv_heads=2, dim=48, vdim=64, size=150, dims=20), 64),
                    C.layer(C.attention(heads=2, kv_heads=1, dim=64, vdim=128, size=0, dims=64), 0)], width=64, loop=(0, 2, 2))
    ckpt, tokens = C.checkpoint(cfg, 3), C.prompt(cfg, 420)
    want = C.oracle_logits(cfg, ckpt, tokens)
    gen = C.generator(cfg, ckpt, *backend, max_seq=430)
    tol = C.TOLERANCE[backend[1]]
    assert C.error(run(gen, tokens, [420]), want) < tol
    if backend[0] == "cuda":
        assert C.error(run(gen, tokens, [250, 1]), want) < tol
        assert C.error(run(gen, tokens, [64, 3, 129, 16, 17, 2, 77]), want) < tol


def test_portions_longer_than_the_largest_graph(backend):
    cfg = C.CASES["mixed"]
    ckpt, tokens = C.checkpoint(cfg), C.prompt(cfg, 61)
    gen = C.generator(cfg, ckpt, *backend, max_portion=16)
    assert gen.max_portion == 16
    assert C.error(run(gen, tokens, [61]), C.oracle_logits(cfg, ckpt, tokens)) < C.TOLERANCE[backend[1]]


def test_unequal_requests_in_one_batch(backend):
    """Requests of different lengths share steps, some idle, one ends and its slot goes to a new request; every request gets
    the logits it has alone."""
    cfg = C.CASES["mixed"]
    ckpt = C.checkpoint(cfg)
    toks = {r: C.prompt(cfg, n, seed=10 + i) for i, (r, n) in enumerate((("a", 41), ("b", 17), ("c", 30), ("d", 25)))}
    want = {r: C.oracle_logits(cfg, ckpt, t) for r, t in toks.items()}
    gen = C.generator(cfg, ckpt, *backend, batch=3)
    at, got = {}, {r: [] for r in toks}
    plan = [{"a": 9, "b": 1}, {"a": 1, "b": 15, "c": 2}, {"b": 1}, {"a": 1, "c": 1, "d": 1}, {"c": 20, "d": 3},
            {"a": 30, "c": 7, "d": 20}, {"d": 1}]
    for step in plan:
        for r in step:
            if r not in at:
                gen.admit(r)
                at[r] = 0
        out = gen.step({r: toks[r][at[r]:at[r] + n] for r, n in step.items()}, {r: range(n) for r, n in step.items()})
        for r, n in step.items():
            got[r].append(out[r])
            at[r] += n
            if at[r] == len(toks[r]):
                gen.release(r)
    assert at == {r: len(t) for r, t in toks.items()} and not gen.slots
    for r in toks:
        assert C.error(np.concatenate(got[r]), want[r]) < C.TOLERANCE[backend[1]], r


def test_wanted_rows_keep_their_order_and_slots_are_checked(backend):
    cfg = C.CASES["grouped"]
    ckpt, tokens = C.checkpoint(cfg), C.prompt(cfg, 20)
    want = C.oracle_logits(cfg, ckpt, tokens)
    gen = C.generator(cfg, ckpt, *backend, max_seq=24)
    gen.admit("x")
    out = gen.step({"x": tokens}, {"x": [19, 0, 7, 7]})["x"]
    assert C.error(out, want[[19, 0, 7, 7]]) < C.TOLERANCE[backend[1]]
    assert gen.step({"x": tokens[:1]}) == {}
    with pytest.raises(ValueError, match="positions"):
        gen.step({"x": tokens[:4]})
    with pytest.raises(ValueError, match="vocabulary"):
        gen.step({"x": [cfg["vocab"]]})
    with pytest.raises(ValueError, match="outside its"):
        gen.step({"x": [1]}, {"x": [1]})
    with pytest.raises(RuntimeError, match="slots"):
        gen.admit("y")
    gen.release("x")
    gen.admit("y")


def greedy(cfg, ckpt, tokens, n):
    out = list(tokens)
    for _ in range(n):
        out.append(int(C.oracle_logits(cfg, ckpt, out)[-1].argmax()))
    return out[len(tokens):]


def test_greedy_generation(backend):
    """Unequal prompts, more of them than slots, a prompt longer than the largest portion, twice on the same generator."""
    cfg = C.CASES["mixed"]
    ckpt = C.checkpoint(cfg, 5)
    prompts = [C.prompt(cfg, n, seed=n) for n in (5, 1, 37, 12, 3)]
    want = [greedy(cfg, ckpt, p, 9) for p in prompts]
    gen = C.generator(cfg, ckpt, *backend, batch=2, max_portion=16, max_new_tokens=9)
    for _ in range(2):
        got = gen.generate(prompts, 9)
        if backend[1] == "float32":
            assert [g.tolist() for g in got] == want
        else:  # bf16 may part from the exact path at a near-tie: every choice must be (almost) the best one
            for p, g in zip(prompts, got):
                lg = C.oracle_logits(cfg, ckpt, list(p) + g.tolist()[:-1])[len(p) - 1:]
                gap = lg.max(-1) - lg[np.arange(len(g)), g]
                assert gap.max() < 0.25 * lg.std()
    assert not gen.slots and gen.prefill_ms() >= 0 and gen.decode_ms() >= 0


@pytest.mark.gpu
def test_kernels_run_on_the_gpu():
    """A bf16 model of regular sizes runs on this package's kernels, prompts and decoding alike."""
    from popxl_addons_b200.ops import native
    from popxl_addons_b200.xl.opdef import FALLBACKS

    cfg = C.config([C.layer({"width": 128}, 256), C.layer(C.attention(heads=4, kv_heads=2, dim=64, vdim=128, size=32, dims=32), 256)],
                   width=128, vocab=256)
    gen = C.generator(cfg, C.checkpoint(cfg), "cuda", "bfloat16", batch=2, max_new_tokens=4)
    before, fell = dict(native.LAUNCHES["by_kernel"]), dict(FALLBACKS)
    gen.generate([C.prompt(cfg, 50), C.prompt(cfg, 33)], 4)
    ran = {k for k, v in native.LAUNCHES["by_kernel"].items() if v > before.get(k, 0)}
    assert {"stream_dyt", "min_gru", "swiglu_packed", "linear_small_m", "linear_small_m_residual", "linear_small_m_swiglu",
            "linear_small_m_min_gru", "diff_attn_decode", "select_dyt", "argmax_rows", "advance_by"} <= ran
    assert FALLBACKS == fell


# ---- configuration, weights, folder, runner -----------------------------------------------------------------------------
def test_configuration_reader():
    from popxl_addons_b200.models.dunelix import DiffAttentionConfig, DunelixConfig, MinGRUConfig

    d = C.CASES["mixed"]
    cfg = DunelixConfig.from_dict(d)
    assert [type(L.mixer) for L in cfg.layers] == [MinGRUConfig, DiffAttentionConfig, MinGRUConfig, DiffAttentionConfig]
    assert cfg.layers[2].ff == 0 and cfg.layers[1].mixer.chunk == 13 and cfg.residual_mult == 0.8
    assert cfg.schedule() == plain.layer_schedule(4, d["loop"])
    assert DunelixConfig.from_dict({**d, "loop": None}).schedule() == [(i, False) for i in range(4)]
    bad = [{**d, "unheard_of": 1}, {k: v for k, v in d.items() if k != "norm"}, {**d, "loop": {"start": 2, "stop": 2, "times": 1}},
           {**d, "layers": [{"type": "other", "mixer": {}, "mlp": None}]},
           {**d, "layers": [C.layer(C.attention(heads=3, kv_heads=2))]}, {**d, "layers": [C.layer(C.attention(dims=18))]}]
    sparse = json.loads(json.dumps(d))
    sparse["layers"][0]["mlp"]["kind"] = "routed"
    for b in bad + [sparse]:
        with pytest.raises(ValueError):
            DunelixConfig.from_dict(b)


def test_loading_refuses_tensors_that_do_not_fit():
    cfg = C.CASES["grouped"]
    ckpt = C.checkpoint(cfg)
    with pytest.raises(ValueError, match="missing"):
        C.generator(cfg, {k: v for k, v in ckpt.items() if k != "l1.mix.g"})
    with pytest.raises(ValueError, match="unexpected"):
        C.generator(cfg, {**ckpt, "l9.mix.g": ckpt["embed"]})
    with pytest.raises(ValueError, match="shape"):
        C.generator(cfg, {**ckpt, "head": ckpt["head"][:-1]})


def test_portion_sizes():
    from popxl_addons_b200.models.sequence_generator import portion_size

    sizes = [portion_size(n) for n in range(1, 5000)]
    assert all(s >= n and portion_size(s) == s for n, s in enumerate(sizes, 1)) and sizes == sorted(sizes)
    assert sizes[:5] == [1, 2, 4, 4, 8] and len(set(sizes)) < 75
    assert max(s / n for n, s in enumerate(sizes, 1) if n > 256) < 1.13


def test_safetensors_reader(tmp_path):
    from popxl_addons_b200.utils.safetensors import read_safetensors

    want = {"a": torch.randn(3, 5), "s": torch.tensor(0.25).bfloat16(), "odd": torch.randn(3).bfloat16(), "b": torch.randn(2, 2)}
    C.write_model(tmp_path, {}, want)
    got = read_safetensors(str(tmp_path / "model.safetensors"))
    assert set(got) == set(want) and all(torch.equal(got[k], v) and got[k].shape == v.shape for k, v in want.items())
    (tmp_path / "bad").write_bytes(b"\xff" * 16)
    with pytest.raises(ValueError):
        read_safetensors(str(tmp_path / "bad"))


def test_model_folder_and_registry(tmp_path, backend):
    from popxl_addons_b200.models import load_config, load_model
    from popxl_addons_b200.models.registry import architecture

    cfg = C.CASES["grouped"]
    ckpt, tokens = C.checkpoint(cfg), C.prompt(cfg, 20)
    folder = C.write_model(tmp_path, cfg, ckpt)
    gen = load_model(folder, dtype=backend[1], device=backend[0], max_seq=32)
    assert C.error(run(gen, tokens, [20]), C.oracle_logits(cfg, ckpt, tokens)) < C.TOLERANCE[backend[1]]
    assert load_config(folder)[0].name == "Dunelix"
    assert architecture("GPT-J").config({"layers": 2}).family == "gptj"
    with pytest.raises(KeyError, match="known"):
        architecture("nothing")
    with pytest.raises(ValueError, match="runs in"):
        load_model(folder, dtype="float16", device="cpu")


def test_trace_runner_and_command_line(tmp_path, backend):
    device, dtype = backend
    cfg = C.CASES["mixed"]
    ckpt = C.checkpoint(cfg)
    folder = C.write_model(tmp_path, cfg, ckpt)
    a, b = C.prompt(cfg, 30, 1), C.prompt(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:21], "want": [20, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[21:22], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[22:], "want": [0, 7]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [8]}], "end": ["b"]}]
    res = subprocess.run([os.path.join(REPO, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(tmp_path),
                          "--max-tokens", "30", "--device", device], input="".join(json.dumps(s) + "\n" for s in steps),
                         capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = C.oracle_logits(cfg, ckpt, a), C.oracle_logits(cfg, ckpt, b)
    for step, want in ((0, wa[[20, 3]]), (2, wa[[22, 29]]), (3, wb[[8]])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert C.error(got, want) < C.TOLERANCE[dtype]
    assert not (tmp_path / "1.f32").exists()
    if dtype == "float32":
        res = subprocess.run([sys.executable, "-m", "popxl_addons_b200.generate", "--model", folder, "--dtype", dtype, "--device",
                              device, "--max-new-tokens", "4", "--prompt", " ".join(map(str, a)), "--prompt", "3,1"], cwd=REPO,
                             capture_output=True, text=True, timeout=300)
        assert res.returncode == 0, res.stderr[-2000:]
        want = [greedy(cfg, ckpt, p, 4) for p in (a, [3, 1])]
        assert [[int(x) for x in l.split()] for l in res.stdout.splitlines()] == want
