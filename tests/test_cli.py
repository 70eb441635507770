"""The command line as a user starts it: ``bin/flow-inference`` in a process of its own.
``doctor``, ``inspect``, ``init`` and ``replay`` need no GPU; ``generate`` does and is compared
with the plain implementation (reference: flow_engine/cli.py:48-120)."""
import json
import subprocess
import sys

import pytest

from helpers import CONFIGS, ROOT, make_folder
import plain_qwen2

CLI = [sys.executable, str(ROOT / "bin" / "flow-inference")]


def run_cli(*words, **kw):
    return subprocess.run(CLI + [str(w) for w in words], capture_output=True, text=True, timeout=900, **kw)


def test_doctor_reports_the_runtime():
    proc = run_cli("doctor")
    assert proc.returncode == 0, proc.stderr
    report = json.loads(proc.stdout)
    assert {"python", "platform", "torch", "cuda", "nvcc", "architectures"} <= set(report)
    assert "Qwen2ForCausalLM" in report["architectures"]


@pytest.mark.parametrize("name", ["A", "B"])
def test_inspect_explains_the_cache(name, tmp_path):
    folder = make_folder(tmp_path, name)
    c = CONFIGS[name]
    proc = run_cli("inspect", folder, "--kv-blocks", 10, "--block-size", 8)
    assert proc.returncode == 0, proc.stderr
    out = json.loads(proc.stdout)
    per_token = 2 * c["num_hidden_layers"] * c["num_key_value_heads"] * c["head_dim"]       # K and V, every layer
    assert out["kv_bf16_bytes"] == per_token * 2 * 10 * 8 and out["kv_fp32_bytes"] == per_token * 4 * 10 * 8
    assert out["architecture"]["hidden_size"] == c["hidden_size"] and out["layers_in_schedule"] == c["num_hidden_layers"]
    assert out["state_bytes_per_request"] == 0
    params = sum(t.numel() for t in plain_qwen2.read_folder(folder)[1].values())
    assert 2 * params <= out["weight_bf16_bytes"] <= 2 * params + 2 * 64 * 1024      # matrices in 16 bits, vectors stay in 32
    assert run_cli("inspect", folder, "--kv-blocks", 0).returncode != 0


def test_inspect_refuses_what_the_gate_refuses(tmp_path):
    folder = tmp_path / "m"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps({**CONFIGS["A"], "use_sliding_window": True}))
    proc = run_cli("inspect", folder)
    assert proc.returncode != 0 and "sliding_window" in proc.stderr


def test_init_writes_a_folder_and_replay_filters_events(tmp_path):
    config = tmp_path / "config.json"
    config.write_text(json.dumps(CONFIGS["B"]))
    proc = run_cli("init", tmp_path / "model", "--config", config, "--seed", 3)
    assert proc.returncode == 0, proc.stderr
    assert (tmp_path / "model" / "config.json").exists() and (tmp_path / "model" / "model.safetensors").exists()
    log = tmp_path / "log.jsonl"
    rows = [{"event": "launch", "argv": []}, {"event": "step", "tokens": 3}, {"event": "submit"},
            {"event": "finish", "finish_reason": "length"}]
    log.write_text("".join(json.dumps(r) + "\n" for r in rows))
    proc = run_cli("replay", log)
    assert proc.returncode == 0
    assert [json.loads(l)["event"] for l in proc.stdout.splitlines()] == ["step", "finish"]


def test_the_prompt_never_reaches_the_audit_log():
    from tessweave_engine_b200.engine.cli import argv_without_prompt
    assert argv_without_prompt(["x", "generate", "m", "--prompt", "secret words", "--max-tokens", "3"]) == \
        ["x", "generate", "m", "--prompt", "[REDACTED]", "--max-tokens", "3"]
    assert argv_without_prompt(["x", "--prompt=secret", "--prompt-ids", "1,2"]) == ["x", "--prompt=[REDACTED]", "--prompt-ids", "1,2"]


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["A", "B"])
def test_generate_as_a_user_starts_it(name, tmp_path):
    """init -> generate --prompt-ids in float32 -> the ids on standard output are the plain implementation's
    greedy continuation; the audit log holds the run's events and ``replay`` prints them."""
    config = tmp_path / "config.json"
    config.write_text(json.dumps(CONFIGS[name]))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 11).returncode == 0
    prompt = [5, 17, 3, 200, 41, 7, 99, 100, 23]
    log = tmp_path / "runs" / "engine.jsonl"
    proc = run_cli("generate", folder, "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-tokens", 8,
                   "--ignore-eos", "--log", log, "--block-size", 8, "--kv-blocks", 32, "--prefill-chunk", 4, "--max-context", 256)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = [int(t) for t in proc.stdout.strip().split(",")]
    cfg, weights = plain_qwen2.read_folder(folder)
    assert got == plain_qwen2.generate(cfg, weights, prompt, 8)
    done = json.loads(proc.stderr.strip().splitlines()[-1])
    assert done["finish_reason"] == "length" and done["usage"] == {"prompt_tokens": 9, "completion_tokens": 8, "total_tokens": 17}
    events = [json.loads(l)["event"] for l in log.read_text().splitlines()]
    assert events[0] == "launch" and "loaded" in events and "admit" in events and events.count("finish") == 1
    assert "--prompt-ids" in json.loads(log.read_text().splitlines()[0])["argv"]
    replayed = run_cli("replay", log)
    assert replayed.returncode == 0 and {json.loads(l)["event"] for l in replayed.stdout.splitlines()} <= \
        {"step", "admit", "finish", "first_token", "fatal"}
    assert sum(json.loads(l)["event"] == "step" for l in replayed.stdout.splitlines()) >= 3 + 7     # 9 prompt tokens in portions of 4, then 7 single tokens


# ---------------------------------------------------------------------------
# the Linurax decoder through the same command line
# ---------------------------------------------------------------------------
def test_doctor_and_inspect_know_linurax(tmp_path):
    from tiny_linurax import LINURAX_A
    assert "Linurax" in json.loads(run_cli("doctor").stdout)["architectures"]
    config = tmp_path / "config.json"
    config.write_text(json.dumps(LINURAX_A))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 2, "--init-std", 0.1).returncode == 0
    proc = run_cli("inspect", folder, "--kv-blocks", 10, "--block-size", 8)
    assert proc.returncode == 0, proc.stderr
    out = json.loads(proc.stdout)
    attention = [l["mixer"] for l in LINURAX_A["layers"] if l["type"] == "attention"]
    per_token = sum(2 * m["kv_heads"] * m["dim"] for m in attention)          # the key and the raw key kept as the value
    assert out["kv_bf16_bytes"] == per_token * 2 * 10 * 8 and out["layers_in_schedule"] == len(LINURAX_A["layers"])
    assert out["state_bytes_per_request"] == 4 * sum(l["mixer"]["width"] for l in LINURAX_A["layers"] if l["type"] == "mingru")
    assert out["architecture"]["width"] == LINURAX_A["width"]
    bad = tmp_path / "bad"
    bad.mkdir()
    (bad / "config.json").write_text(json.dumps({**LINURAX_A, "layers": [{**LINURAX_A["layers"][0], "type": "conv"}]}))
    proc = run_cli("inspect", bad)
    assert proc.returncode != 0 and "not implemented" in proc.stderr


@pytest.mark.gpu
def test_generate_linurax_as_a_user_starts_it(tmp_path):
    """init -> generate --prompt-ids in float32 -> the plain implementation's greedy continuation."""
    import plain_linurax
    from tiny_linurax import LINURAX_B
    config = tmp_path / "config.json"
    config.write_text(json.dumps(LINURAX_B))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 11, "--init-std", 0.2).returncode == 0
    prompt = [5, 17, 3, 20, 41, 7, 96, 10, 23]
    proc = run_cli("generate", folder, "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-tokens", 8,
                   "--ignore-eos", "--log", tmp_path / "runs" / "engine.jsonl", "--block-size", 8, "--kv-blocks", 32,
                   "--prefill-chunk", 4, "--max-context", 256)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = [int(t) for t in proc.stdout.strip().split(",")]
    assert got == plain_linurax.greedy(folder, prompt, 8)


# ---------------------------------------------------------------------------
# the Sapatar decoder through the same command line
# ---------------------------------------------------------------------------
def test_doctor_and_inspect_know_sapatar(tmp_path):
    from tiny_sapatar import SAPATAR_A
    assert "Sapatar" in json.loads(run_cli("doctor").stdout)["architectures"]
    config = tmp_path / "config.json"
    config.write_text(json.dumps(SAPATAR_A))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 2, "--init-std", 0.1).returncode == 0
    proc = run_cli("inspect", folder, "--kv-blocks", 10, "--block-size", 8)
    assert proc.returncode == 0, proc.stderr
    out = json.loads(proc.stdout)
    lefts = [l["mixer"]["left"] for l in SAPATAR_A["layers"] if l["type"] == "parallel"]
    per_token = sum(m["kv_heads"] * (m["dim"] + m["vdim"]) for m in lefts)          # keys and values of different sizes
    assert out["kv_bf16_bytes"] == per_token * 2 * 10 * 8 and out["layers_in_schedule"] == len(SAPATAR_A["layers"])
    states = 0
    for layer in SAPATAR_A["layers"]:
        m = layer["mixer"]
        if layer["type"] == "wkv":
            states += m["heads"] * m["dim"] * m["dim"] + SAPATAR_A["width"]
        elif layer["type"] == "retention":
            states += m["heads"] * m["dim"] * m["vdim"]
        else:
            states += m["right"]["heads"] * (m["right"]["dim"] * (m["right"]["vdim"] + 1) + 1)
    assert out["state_bytes_per_request"] == 4 * states
    bad = tmp_path / "bad"
    bad.mkdir()
    (bad / "config.json").write_text(json.dumps({**SAPATAR_A, "layers": [{**SAPATAR_A["layers"][0], "type": "conv"}]}))
    proc = run_cli("inspect", bad)
    assert proc.returncode != 0 and "not implemented" in proc.stderr


@pytest.mark.gpu
def test_generate_sapatar_as_a_user_starts_it(tmp_path):
    """init -> generate --prompt-ids in float32 -> the plain implementation's greedy continuation."""
    import plain_sapatar
    from tiny_sapatar import SAPATAR_D
    config = tmp_path / "config.json"
    config.write_text(json.dumps(SAPATAR_D))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 11, "--init-std", 0.2).returncode == 0
    prompt = [5, 17, 3, 20, 41, 7, 50, 10, 23]
    proc = run_cli("generate", folder, "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-tokens", 8,
                   "--ignore-eos", "--log", tmp_path / "runs" / "engine.jsonl", "--block-size", 8, "--kv-blocks", 32,
                   "--prefill-chunk", 4, "--max-context", 256)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = [int(t) for t in proc.stdout.strip().split(",")]
    assert got == plain_sapatar.greedy(folder, prompt, 8)


# ---------------------------------------------------------------------------
# the Nufatar decoder through the same command line
# ---------------------------------------------------------------------------
def test_doctor_and_inspect_know_nufatar(tmp_path):
    import plain_nufatar
    from tiny_nufatar import NUFATAR_A
    assert "Nufatar" in json.loads(run_cli("doctor").stdout)["architectures"]
    config = tmp_path / "config.json"
    config.write_text(json.dumps(NUFATAR_A))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 2, "--init-std", 0.1).returncode == 0
    proc = run_cli("inspect", folder, "--kv-blocks", 10, "--block-size", 8)
    assert proc.returncode == 0, proc.stderr
    out = json.loads(proc.stdout)
    runs = plain_nufatar.layer_runs(NUFATAR_A)
    per_token = states = 0
    for i, _ in runs:                                     # every run of a repeated layer keeps pages and a state of its own
        m = NUFATAR_A["layers"][i]["mixer"]
        lft, rgt = m["left"], m["right"]
        per_token += lft["kv_heads"] * (lft["dim"] + (lft["vdim"] if "rot" in lft else 0))       # values that are the keys cost nothing
        channels = 2 * rgt["kv_heads"] * rgt["dim"] + rgt["heads"] * rgt["vdim"]
        states += rgt["heads"] * rgt["dim"] * rgt["vdim"] + channels * (rgt["conv"] - 1)
    assert out["layers_in_schedule"] == len(runs) == 8
    assert out["kv_bf16_bytes"] == per_token * 2 * 10 * 8
    assert out["state_bytes_per_request"] == 4 * states
    bad = tmp_path / "bad"
    bad.mkdir()
    (bad / "config.json").write_text(json.dumps({**NUFATAR_A, "layers": [{**NUFATAR_A["layers"][0], "type": "parallel_3"}]}))
    proc = run_cli("inspect", bad)
    assert proc.returncode != 0 and "not implemented" in proc.stderr


@pytest.mark.gpu
def test_generate_nufatar_as_a_user_starts_it(tmp_path):
    """init -> generate --prompt-ids in float32 -> the plain implementation's greedy continuation."""
    import plain_nufatar
    from tiny_nufatar import NUFATAR_D
    config = tmp_path / "config.json"
    config.write_text(json.dumps(NUFATAR_D))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 11, "--init-std", 0.25).returncode == 0
    prompt = [5, 17, 3, 20, 41, 7, 50, 10, 23]
    proc = run_cli("generate", folder, "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-tokens", 8,
                   "--ignore-eos", "--log", tmp_path / "runs" / "engine.jsonl", "--block-size", 8, "--kv-blocks", 32,
                   "--prefill-chunk", 4, "--max-context", 256)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = [int(t) for t in proc.stdout.strip().split(",")]
    assert got == plain_nufatar.greedy(folder, prompt, 8)


# ---------------------------------------------------------------------------
# the Dugudra decoder through the same command line
# ---------------------------------------------------------------------------
def test_doctor_and_inspect_know_dugudra(tmp_path):
    from tiny_dugudra import DUGUDRA_A
    assert "Dugudra" in json.loads(run_cli("doctor").stdout)["architectures"]
    config = tmp_path / "config.json"
    config.write_text(json.dumps(DUGUDRA_A))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 2, "--init-std", 0.1).returncode == 0
    proc = run_cli("inspect", folder, "--kv-blocks", 10, "--block-size", 8)
    assert proc.returncode == 0, proc.stderr
    out = json.loads(proc.stdout)
    per_token = states = 0
    for layer in DUGUDRA_A["layers"]:
        m = layer["mixer"]
        if layer["type"] == "attention":
            per_token += m["kv_heads"] * (m["dim"] + m["vdim"])
        elif layer["type"] == "latent_attention":
            per_token += m["kv_rank"] + m["rot_dim"]            # one row per token serves as key and value
        else:
            states += m["heads"] * m["dim"] * m["vdim"]
    assert out["layers_in_schedule"] == len(DUGUDRA_A["layers"])
    assert out["kv_bf16_bytes"] == per_token * 2 * 10 * 8
    assert out["state_bytes_per_request"] == 4 * states
    bad = tmp_path / "bad"
    bad.mkdir()
    (bad / "config.json").write_text(json.dumps({**DUGUDRA_A, "layers": [{**DUGUDRA_A["layers"][0], "type": "conv"}]}))
    proc = run_cli("inspect", bad)
    assert proc.returncode != 0 and "not implemented" in proc.stderr


@pytest.mark.gpu
def test_generate_dugudra_as_a_user_starts_it(tmp_path):
    """init -> generate --prompt-ids in float32 -> the plain implementation's greedy continuation."""
    import plain_dugudra
    from tiny_dugudra import DUGUDRA_D
    config = tmp_path / "config.json"
    config.write_text(json.dumps(DUGUDRA_D))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 11, "--init-std", 0.25).returncode == 0
    prompt = [5, 17, 3, 20, 41, 7, 50, 10, 23]
    proc = run_cli("generate", folder, "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-tokens", 8,
                   "--ignore-eos", "--log", tmp_path / "runs" / "engine.jsonl", "--block-size", 8, "--kv-blocks", 32,
                   "--prefill-chunk", 4, "--max-context", 256)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = [int(t) for t in proc.stdout.strip().split(",")]
    assert got == plain_dugudra.greedy(folder, prompt, 8)


# ---------------------------------------------------------------------------
# the Varivik decoder through the same command line
# ---------------------------------------------------------------------------
def test_doctor_and_inspect_know_varivik(tmp_path):
    from tiny_varivik import VARIVIK_A
    assert "Varivik" in json.loads(run_cli("doctor").stdout)["architectures"]
    config = tmp_path / "config.json"
    config.write_text(json.dumps(VARIVIK_A))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 2, "--init-std", 0.1).returncode == 0
    proc = run_cli("inspect", folder, "--kv-blocks", 10, "--block-size", 8)
    assert proc.returncode == 0, proc.stderr
    out = json.loads(proc.stdout)
    per_token = sum(m["kv_heads"] * (m["dim"] + m["vdim"]) for m in (layer["mixer"] for layer in VARIVIK_A["layers"]))
    assert out["layers_in_schedule"] == len(VARIVIK_A["layers"])
    assert out["kv_bf16_bytes"] == per_token * 2 * 10 * 8
    assert out["state_bytes_per_request"] == 0
    bad = tmp_path / "bad"
    bad.mkdir()
    (bad / "config.json").write_text(json.dumps({**VARIVIK_A, "layers": [{**VARIVIK_A["layers"][0], "type": "conv"}]}))
    proc = run_cli("inspect", bad)
    assert proc.returncode != 0 and "not implemented" in proc.stderr


@pytest.mark.gpu
def test_generate_varivik_as_a_user_starts_it(tmp_path):
    """init -> generate --prompt-ids in float32 -> the plain implementation's greedy continuation."""
    import plain_varivik
    from tiny_varivik import VARIVIK_D
    config = tmp_path / "config.json"
    config.write_text(json.dumps(VARIVIK_D))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 11, "--init-std", 0.25).returncode == 0
    prompt = [5, 17, 3, 20, 41, 7, 50, 10, 23]
    proc = run_cli("generate", folder, "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-tokens", 8,
                   "--ignore-eos", "--log", tmp_path / "runs" / "engine.jsonl", "--block-size", 8, "--kv-blocks", 32,
                   "--prefill-chunk", 4, "--max-context", 256)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = [int(t) for t in proc.stdout.strip().split(",")]
    assert got == plain_varivik.greedy(folder, prompt, 8)


# ---------------------------------------------------------------------------
# the Bavetar decoder through the same command line
# ---------------------------------------------------------------------------
def test_doctor_and_inspect_know_bavetar(tmp_path):
    from tiny_bavetar import BAVETAR_A
    assert "Bavetar" in json.loads(run_cli("doctor").stdout)["architectures"]
    config = tmp_path / "config.json"
    config.write_text(json.dumps(BAVETAR_A))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 2, "--init-std", 0.1).returncode == 0
    proc = run_cli("inspect", folder, "--kv-blocks", 10, "--block-size", 8)
    assert proc.returncode == 0, proc.stderr
    out = json.loads(proc.stdout)
    mixers = [layer["mixer"] for layer in BAVETAR_A["layers"]]
    assert out["layers_in_schedule"] == len(mixers)
    assert out["kv_bf16_bytes"] == sum(m["kv_rank"] + m["rot_dim"] for m in mixers if "kv_rank" in m) * 2 * 10 * 8
    assert out["state_bytes_per_request"] == 4 * sum(
        m["heads"] * m["state"] * m["vdim"] + (m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]) * (m["conv"] - 1)
        for m in mixers if "state" in m)
    bad = tmp_path / "bad"
    bad.mkdir()
    (bad / "config.json").write_text(json.dumps({**BAVETAR_A, "layers": [{**BAVETAR_A["layers"][0], "type": "conv"}]}))
    proc = run_cli("inspect", bad)
    assert proc.returncode != 0 and "not implemented" in proc.stderr


@pytest.mark.gpu
def test_generate_bavetar_as_a_user_starts_it(tmp_path):
    """init -> generate --prompt-ids in float32 -> the plain implementation's greedy continuation."""
    import plain_bavetar
    from tiny_bavetar import BAVETAR_D
    config = tmp_path / "config.json"
    config.write_text(json.dumps(BAVETAR_D))
    folder = tmp_path / "model"
    assert run_cli("init", folder, "--config", config, "--seed", 11, "--init-std", 0.25).returncode == 0
    prompt = [5, 17, 3, 20, 41, 7, 50, 10, 23]
    proc = run_cli("generate", folder, "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32", "--max-tokens", 8,
                   "--ignore-eos", "--log", tmp_path / "runs" / "engine.jsonl", "--block-size", 8, "--kv-blocks", 32,
                   "--prefill-chunk", 4, "--max-context", 256)
    assert proc.returncode == 0, proc.stderr[-3000:]
    got = [int(t) for t in proc.stdout.strip().split(",")]
    assert got == plain_bavetar.greedy(folder, prompt, 8)
