"""The command line: option names and defaults of the reference, inspect without a GPU."""
import json
import os
import subprocess
import sys

import pytest

import helpers
from llama_rs_metal_b200 import cli

CLI = os.path.join(helpers.ROOT, "bin", "llama-cli")


def test_sampling_options_have_the_reference_defaults():
    # crates/llama-cli/src/main.rs:79-93
    args = cli.build_parser().parse_args(["generate", "-m", "x", "-p", "1,2"])
    assert (args.max_tokens, args.temperature, args.top_k, args.top_p, args.repeat_penalty, args.seed) == \
           (256, 0.8, 40, 0.95, 1.0, 42)
    assert args.context == 0 and args.memory_mib is None and args.float_weights_f32 is False
    args = cli.build_parser().parse_args(["generate", "--model", "x", "--prompt", "@f", "-n", "5", "-c", "64",
                                          "--float-weights-f32", "--memory-mib", "100"])
    assert (args.max_tokens, args.context, args.float_weights_f32, args.memory_mib) == (5, 64, True, 100)


def test_prompts_are_token_ids(tmp_path):
    assert cli._parse_prompt("1, 2,3") == [1, 2, 3]
    (tmp_path / "ids.txt").write_text("7 8\n9\n")
    assert cli._parse_prompt("@" + str(tmp_path / "ids.txt")) == [7, 8, 9]


def test_inspect_and_random_run_without_a_gpu(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(helpers.TINY["B"]["config"]))
    out = subprocess.run([sys.executable, CLI, "random", "--config", str(config), "--out", str(tmp_path / "m"),
                          "--seed", "7", "--std", "0.05"], capture_output=True, text=True,
                         env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    out = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "m"), "--tensors"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["format"] == "safetensors" and report["config"]["num_hidden_layers"] == 3
    assert report["tensor_count"] == 3 * 9 + 3
    entry = report["tensors"]["model.layers.2.mlp.down_proj.weight"]
    assert entry == {"dimensions": [96, 256], "storage_bytes": 96 * 256 * 2, "encoding": "bfloat16"}
    assert report["weight_bytes"] == sum(t["storage_bytes"] for t in report["tensors"].values())
    bad = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "nothing")], capture_output=True, text=True)
    assert bad.returncode == 1 and bad.stderr.startswith("error:")


@pytest.mark.gpu
def test_generate_prints_token_ids_and_finish_reasons(model_dirs):
    out = subprocess.run([sys.executable, CLI, "generate", "-m", model_dirs["A"], "-p", "1,2,3", "-p", "9",
                          "-n", "4", "--temperature", "0", "-c", "64", "--float-weights-f32"],
                         capture_output=True, text=True)
    assert out.returncode == 0, out.stderr
    lines = out.stdout.strip().splitlines()
    tokens = [l.split("\t") for l in lines if "\t" in l]
    finished = [json.loads(l) for l in lines if l.startswith("{")]
    assert len(tokens) == 8 and len(finished) == 2
    assert all(f["reason"] == "length" and f["tokens"] == 4 for f in finished)
    assert finished[0]["ids"] == [int(t) for r, t in tokens if r == "0"]
    assert "context 64" in out.stderr


def test_inspect_and_random_take_the_second_architecture(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(helpers.KIKALIX["K3"]["config"]))
    out = subprocess.run([sys.executable, CLI, "random", "--config", str(config), "--out", str(tmp_path / "m"),
                          "--seed", "3", "--std", "0.1", "--norm-mean", "0", "--norm-std", "0.1"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    out = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "m"), "--tensors"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["config"]["architecture"] == "Kikalix" and len(report["config"]["layers"]) == 2
    assert report["tensors"]["l0.mix.left.v.b"]["dimensions"] == [32]
    assert report["tensors"]["l0.mix.right.a2"]["dimensions"] == [8, 2]
    assert report["tensors"]["l1.mix.g"]["dimensions"] == [48, 64]
    assert "loop.step" not in report["tensors"]            # this configuration has no loop


@pytest.mark.gpu
def test_generate_runs_the_second_architecture(tmp_path):
    folder = helpers.make_kikalix_dir(str(tmp_path / "m"), "K1")
    runs = []
    for flags in (["--float-weights-f32"], []):
        out = subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "1,2,3", "-p", "9", "-n", "5",
                              "--temperature", "0", "-c", "64", *flags], capture_output=True, text=True)
        assert out.returncode == 0, out.stderr
        finished = [json.loads(l) for l in out.stdout.strip().splitlines() if l.startswith("{")]
        assert len(finished) == 2 and all(f["reason"] == "length" and f["tokens"] == 5 for f in finished)
        assert "Kikalix" in out.stderr
        runs.append([f["ids"] for f in finished])
    # sampled generation with a seed repeats itself
    sampled = [subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "4,5", "-n", "6", "--seed", "11"],
                              capture_output=True, text=True).stdout for _ in range(2)]
    assert sampled[0] == sampled[1] and sampled[0].count("\t") == 6


def test_inspect_and_random_take_the_third_architecture(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(helpers.PIBUVIK["P3"]["config"]))
    out = subprocess.run([sys.executable, CLI, "random", "--config", str(config), "--out", str(tmp_path / "m"),
                          "--seed", "3", "--std", "0.1", "--norm-mean", "1", "--norm-std", "0.1"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    out = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "m"), "--tensors"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["config"]["architecture"] == "Pibuvik" and len(report["config"]["layers"]) == 3
    assert report["tensors"]["l0.mix.ra"]["dimensions"] == [2, 32, 32]
    assert report["tensors"]["l1.mix.sink"]["dimensions"] == [2]
    assert report["tensors"]["l2.mix.dkv"]["dimensions"] == [20, 64]
    assert "l1.mix.v" not in report["tensors"] and "l0.mlp.gate" not in report["tensors"]


@pytest.mark.gpu
def test_generate_runs_the_third_architecture(tmp_path):
    folder = helpers.make_pibuvik_dir(str(tmp_path / "m"), "P1")
    runs = []
    for flags in (["--float-weights-f32"], []):
        out = subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "1,2,3", "-p", "9", "-n", "5",
                              "--temperature", "0", "-c", "64", *flags], capture_output=True, text=True)
        assert out.returncode == 0, out.stderr
        finished = [json.loads(l) for l in out.stdout.strip().splitlines() if l.startswith("{")]
        assert len(finished) == 2 and all(f["reason"] == "length" and f["tokens"] == 5 for f in finished)
        assert "Pibuvik" in out.stderr
        runs.append([f["ids"] for f in finished])
    sampled = [subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "4,5", "-n", "6", "--seed", "11"],
                              capture_output=True, text=True).stdout for _ in range(2)]
    assert sampled[0] == sampled[1] and sampled[0].count("\t") == 6


def test_inspect_and_random_take_the_fourth_architecture(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(helpers.NOREVIK["N3"]["config"]))
    out = subprocess.run([sys.executable, CLI, "random", "--config", str(config), "--out", str(tmp_path / "m"),
                          "--seed", "3", "--std", "0.1", "--norm-mean", "1", "--norm-std", "0.1"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    out = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "m"), "--tensors"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["config"]["architecture"] == "Norevik" and len(report["config"]["layers"]) == 3
    assert report["tensors"]["l0.mix.sink"]["dimensions"] == [2]
    assert report["tensors"]["l1.mix.f.b"]["dimensions"] == [1]
    assert report["tensors"]["l2.mix.in"]["dimensions"] == [2 * 48 + 2 * 36 + 3, 64]
    assert report["tensors"]["l2.mlp.router"]["dimensions"] == [3, 64]
    assert report["tensors"]["l2.norm2.b"]["dimensions"] == [64]
    assert "l0.norm2" not in report["tensors"] and "l2.mlp.e3.gate" not in report["tensors"]


@pytest.mark.gpu
def test_generate_runs_the_fourth_architecture(tmp_path):
    folder = helpers.make_norevik_dir(str(tmp_path / "m"), "N1")
    for flags in (["--float-weights-f32"], []):
        out = subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "1,2,3", "-p", "9", "-n", "5",
                              "--temperature", "0", "-c", "64", *flags], capture_output=True, text=True)
        assert out.returncode == 0, out.stderr
        finished = [json.loads(l) for l in out.stdout.strip().splitlines() if l.startswith("{")]
        assert len(finished) == 2 and all(f["reason"] == "length" and f["tokens"] == 5 for f in finished)
        assert "Norevik" in out.stderr
    sampled = [subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "4,5", "-n", "6", "--seed", "11"],
                              capture_output=True, text=True).stdout for _ in range(2)]
    assert sampled[0] == sampled[1] and sampled[0].count("\t") == 6


def test_inspect_and_random_take_the_fifth_architecture(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(helpers.TARUPEL["T3"]["config"]))
    out = subprocess.run([sys.executable, CLI, "random", "--config", str(config), "--out", str(tmp_path / "m"),
                          "--seed", "3", "--std", "0.1", "--norm-mean", "1", "--norm-std", "0.1"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    out = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "m"), "--tensors"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["config"]["architecture"] == "Tarupel" and len(report["config"]["layers"]) == 3
    assert report["tensors"]["l0.norm1"]["dimensions"] == [] and report["tensors"]["l0.shift"]["dimensions"] == [64]
    assert report["tensors"]["l0.mix.q.conv"]["dimensions"] == [32, 5]
    assert report["tensors"]["l1.mix.k.norm"]["dimensions"] == [16]
    assert report["tensors"]["l2.mix.w1"]["dimensions"] == [4, 64]
    assert report["tensors"]["l2.mlp.shared.sg"]["dimensions"] == [1, 64]
    assert "l0.norm2" not in report["tensors"] and "loop.step" not in report["tensors"]


@pytest.mark.gpu
def test_generate_runs_the_fifth_architecture(tmp_path):
    folder = helpers.make_tarupel_dir(str(tmp_path / "m"), "T1")
    for flags in (["--float-weights-f32"], []):
        out = subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "1,2,3", "-p", "9", "-n", "5",
                              "--temperature", "0", "-c", "64", *flags], capture_output=True, text=True)
        assert out.returncode == 0, out.stderr
        finished = [json.loads(l) for l in out.stdout.strip().splitlines() if l.startswith("{")]
        assert len(finished) == 2 and all(f["reason"] == "length" and f["tokens"] == 5 for f in finished)
        assert "Tarupel" in out.stderr
    sampled = [subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "4,5", "-n", "6", "--seed", "11"],
                              capture_output=True, text=True).stdout for _ in range(2)]
    assert sampled[0] == sampled[1] and sampled[0].count("\t") == 6


def test_inspect_and_random_take_the_sixth_architecture(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(helpers.TOLURAX["X3"]["config"]))
    out = subprocess.run([sys.executable, CLI, "random", "--config", str(config), "--out", str(tmp_path / "m"),
                          "--seed", "3", "--std", "0.1", "--norm-mean", "1", "--norm-std", "0.1"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    out = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "m"), "--tensors"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["config"]["architecture"] == "Tolurax" and len(report["config"]["layers"]) == 3
    assert report["tensors"]["l0.mix.left.pb"]["dimensions"] == [2] and report["tensors"]["l0.canon1"]["dimensions"] == [64, 1]
    assert report["tensors"]["l0.mix.right.w1"]["dimensions"] == [2, 64]
    assert report["tensors"]["l1.mix.q.conv"]["dimensions"] == [8, 1]
    assert "l1.norm2" not in report["tensors"] and "loop.in" not in report["tensors"]


@pytest.mark.gpu
def test_generate_runs_the_sixth_architecture(tmp_path):
    folder = helpers.make_tolurax_dir(str(tmp_path / "m"), "X1")
    for flags in (["--float-weights-f32"], []):
        out = subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "1,2,3", "-p", "9", "-n", "5",
                              "--temperature", "0", "-c", "64", *flags], capture_output=True, text=True)
        assert out.returncode == 0, out.stderr
        finished = [json.loads(l) for l in out.stdout.strip().splitlines() if l.startswith("{")]
        assert len(finished) == 2 and all(f["reason"] == "length" and f["tokens"] == 5 for f in finished)
        assert "Tolurax" in out.stderr
    sampled = [subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "4,5", "-n", "6", "--seed", "11"],
                              capture_output=True, text=True).stdout for _ in range(2)]
    assert sampled[0] == sampled[1] and sampled[0].count("\t") == 6


def test_inspect_and_random_take_the_seventh_architecture(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(helpers.MUNUPEL["M1"]["config"]))
    out = subprocess.run([sys.executable, CLI, "random", "--config", str(config), "--out", str(tmp_path / "m"),
                          "--seed", "3", "--std", "0.1", "--norm-mean", "1", "--norm-std", "0.1"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    out = subprocess.run([sys.executable, CLI, "inspect", str(tmp_path / "m"), "--tensors"],
                         capture_output=True, text=True, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert out.returncode == 0, out.stderr
    report = json.loads(out.stdout)
    assert report["config"]["architecture"] == "Munupel" and len(report["config"]["layers"]) == 5
    assert report["tensors"]["l0.mix.g"]["dimensions"] == [80, 72] and report["tensors"]["l1.mix.sink"]["dimensions"] == [3]
    assert report["tensors"]["l0.mix.o.b"]["dimensions"] == [72] and report["tensors"]["final.norm.b"]["dimensions"] == [72]
    assert not any(name.startswith("l3.") or ".norm2" in name for name in report["tensors"])


@pytest.mark.gpu
def test_generate_runs_the_seventh_architecture(tmp_path):
    folder = helpers.make_munupel_dir(str(tmp_path / "m"), "M1")
    for flags in (["--float-weights-f32"], []):
        out = subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "1,2,3", "-p", "9", "-n", "5",
                              "--temperature", "0", "-c", "64", *flags], capture_output=True, text=True)
        assert out.returncode == 0, out.stderr
        finished = [json.loads(l) for l in out.stdout.strip().splitlines() if l.startswith("{")]
        assert len(finished) == 2 and all(f["reason"] == "length" and f["tokens"] == 5 for f in finished)
        assert "Munupel" in out.stderr
    sampled = [subprocess.run([sys.executable, CLI, "generate", "-m", folder, "-p", "4,5", "-n", "6", "--seed", "11"],
                              capture_output=True, text=True).stdout for _ in range(2)]
    assert sampled[0] == sampled[1] and sampled[0].count("\t") == 6
