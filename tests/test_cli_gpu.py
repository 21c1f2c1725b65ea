"""The command line on the GPU, from a written model folder to tokens: the two tiny workloads of the
benchmark description (three prompts of 5, 9 and 13 tokens, 8 greedy steps; four prompts of 1, 7, 31 and 64
tokens, 16 steps at temperature 0.8 with a fixed seed), each token checked against the plain implementation."""
import json
from importlib import import_module

import pytest
import torch

import plain_qwen3 as plain

pytestmark = pytest.mark.gpu


def _run_cli(capsys, argv):
    cli = import_module("pytorch-engine_b200.cli")
    assert cli.main(argv) == 0
    lines = [json.loads(line) for line in capsys.readouterr().out.splitlines() if line.startswith("{")]
    return sorted(lines, key=lambda r: r["request"])


def _prompts(vocab, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lengths]


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_cli_greedy_tiny_a(pe, tmp_path, capsys, dtype):
    folder = str(tmp_path / "a")
    pe.write_random_model(folder, pe.preset("tiny_a"), 0)
    cfg, w = plain.load_folder(folder)
    prompts = _prompts(cfg["vocab_size"], (5, 9, 13), 0)
    argv = ["--model", folder, "--dtype", dtype, "--max-tokens", "8", "--temperature", "0", "--json"]
    for p in prompts:
        argv += ["--prompt-ids", ",".join(map(str, p))]
    out = _run_cli(capsys, argv)
    assert [r["request"] for r in out] == [0, 1, 2] and [r["prompt_tokens"] for r in out] == [5, 9, 13]
    for r, p in zip(out, prompts):
        assert r["completion_tokens"] == 8 and r["finish_reason"] == "length"
        if dtype == "fp32":
            assert r["token_ids"] == plain.generate_greedy(cfg, w, p, 8)
        else:
            # bfloat16: each token is the plain implementation's best or, in a near tie, its runner-up
            plain.check_drawn_tokens(cfg, w, p, r["token_ids"], seed=0, request=r["request"], margin=0.05, temperature=0.0)


def test_cli_seeded_temperature_tiny_b(pe, tmp_path, capsys):
    folder = str(tmp_path / "b")
    pe.write_random_model(folder, pe.preset("tiny_b"), 1)
    cfg, w = plain.load_folder(folder)
    prompts = _prompts(cfg["vocab_size"], (1, 7, 31, 64), 1)
    base = ["--model", folder, "--dtype", "fp32", "--max-tokens", "16", "--temperature", "0.8", "--sampling-seed", "11", "--json"]
    argv = list(base)
    for p in prompts:
        argv += ["--prompt-ids", ",".join(map(str, p))]
    out = _run_cli(capsys, argv)
    differed = 0
    for r, p in zip(out, prompts):
        assert r["completion_tokens"] == 16 and r["prompt_tokens"] == len(p)
        # the command line's defaults are the reference's: top-k 40, top-p 0.95, min-p 0.05
        differed += plain.check_drawn_tokens(cfg, w, p, r["token_ids"], seed=11, request=r["request"], margin=1e-3,
                                             temperature=0.8, top_k=40, top_p=0.95, min_p=0.05)
    assert differed <= 2
    again = _run_cli(capsys, argv)
    assert [r["token_ids"] for r in again] == [r["token_ids"] for r in out]
    seed_at = argv.index("--sampling-seed") + 1
    other = _run_cli(capsys, argv[:seed_at] + ["12"] + argv[seed_at + 1:])
    assert [r["token_ids"] for r in other] != [r["token_ids"] for r in out]


def test_cli_greedy_vabelorn(pe, tmp_path, capsys):
    """The second architecture through the same command line: a folder written from the preset, greedy tokens in
    float32 against the plain implementation's best token at every step."""
    import plain_vabelorn
    from safetensors.torch import load_file

    folder = str(tmp_path / "v")
    pe.write_random_model(folder, pe.preset("vabelorn_tiny"), 5)
    with open(folder + "/config.json") as fh:
        cfg = json.load(fh)
    w = {k: v.float() for k, v in load_file(folder + "/model.safetensors").items()}
    prompts = _prompts(cfg["vocab"], (3, 11, 70), 2)
    argv = ["--model", folder, "--dtype", "fp32", "--ctx", "256", "--max-tokens", "6", "--temperature", "0", "--json"]
    for p in prompts:
        argv += ["--prompt-ids", ",".join(map(str, p))]
    out = _run_cli(capsys, argv)
    for r, p in zip(out, prompts):
        assert r["completion_tokens"] == 6
        ref = plain_vabelorn.forward(cfg, w, p + r["token_ids"])
        for j, tok in enumerate(r["token_ids"]):
            row = ref[len(p) - 1 + j]
            assert float(row.max() - row[tok]) <= 1e-4 * float(ref.abs().max())


def test_cli_greedy_lunadra(pe, tmp_path, capsys):
    """The third architecture through the same command line: a folder written from the preset (pair table, window
    attention beside the gated delta rule, mlstm, routed experts), greedy tokens in float32 against the plain
    implementation's best token at every step."""
    import plain_lunadra
    from safetensors.torch import load_file

    folder = str(tmp_path / "l")
    pe.write_random_model(folder, pe.preset("lunadra_tiny"), 6)
    with open(folder + "/config.json") as fh:
        cfg = json.load(fh)
    w = {k: v.float() for k, v in load_file(folder + "/model.safetensors").items()}
    prompts = _prompts(cfg["vocab"], (3, 11, 150), 3)
    argv = ["--model", folder, "--dtype", "fp32", "--ctx", "256", "--max-tokens", "6", "--temperature", "0", "--json"]
    for p in prompts:
        argv += ["--prompt-ids", ",".join(map(str, p))]
    out = _run_cli(capsys, argv)
    for r, p in zip(out, prompts):
        assert r["completion_tokens"] == 6
        ref = plain_lunadra.forward(cfg, w, p + r["token_ids"])
        for j, tok in enumerate(r["token_ids"]):
            row = ref[len(p) - 1 + j]
            assert float(row.max() - row[tok]) <= 1e-4 * float(ref.abs().max())


def test_cli_greedy_zonevik(pe, tmp_path, capsys):
    """The fifth architecture through the same command line: a folder written from the preset (a looped range of layers,
    window attention with kept first positions beside a state-space mixer, the gated delta rule, gated attention, experts
    chosen among groups), greedy tokens in float32 against the plain implementation's best token at every step."""
    import plain_zonevik
    from safetensors.torch import load_file

    folder = str(tmp_path / "z")
    pe.write_random_model(folder, pe.preset("zonevik_tiny"), 7)
    with open(folder + "/config.json") as fh:
        cfg = json.load(fh)
    w = {k: v.float() for k, v in load_file(folder + "/model.safetensors").items()}
    prompts = _prompts(cfg["vocab"], (3, 11, 150), 3)
    argv = ["--model", folder, "--dtype", "fp32", "--ctx", "256", "--max-tokens", "6", "--temperature", "0", "--json"]
    for p in prompts:
        argv += ["--prompt-ids", ",".join(map(str, p))]
    out = _run_cli(capsys, argv)
    for r, p in zip(out, prompts):
        assert r["completion_tokens"] == 6
        ref = plain_zonevik.forward(cfg, w, p + r["token_ids"])
        for j, tok in enumerate(r["token_ids"]):
            row = ref[len(p) - 1 + j]
            assert float(row.max() - row[tok]) <= 1e-4 * float(ref.abs().max())


def test_cli_greedy_burinex(pe, tmp_path, capsys):
    """The seventh architecture through the same command line: a folder written from the preset (lightning, latent attention under
    a window, attention with one norm over all heads, experts weighted on their input), greedy tokens in float32 against the plain
    implementation's best token at every step."""
    import plain_burinex
    from safetensors.torch import load_file

    folder = str(tmp_path / "x")
    pe.write_random_model(folder, pe.preset("burinex_tiny"), 7)
    with open(folder + "/config.json") as fh:
        cfg = json.load(fh)
    w = {k: v.float() for k, v in load_file(folder + "/model.safetensors").items()}
    prompts = _prompts(cfg["vocab"], (3, 11, 150), 3)
    argv = ["--model", folder, "--dtype", "fp32", "--ctx", "256", "--max-tokens", "6", "--temperature", "0", "--json"]
    for p in prompts:
        argv += ["--prompt-ids", ",".join(map(str, p))]
    out = _run_cli(capsys, argv)
    for r, p in zip(out, prompts):
        assert r["completion_tokens"] == 6
        ref = plain_burinex.forward(cfg, w, p + r["token_ids"])
        for j, tok in enumerate(r["token_ids"]):
            row = ref[len(p) - 1 + j]
            assert float(row.max() - row[tok]) <= 1e-4 * float(ref.abs().max())
