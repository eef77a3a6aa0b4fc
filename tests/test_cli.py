"""The command line: the subcommands that need no device (random, inspect) here; generate and bench on the GPU."""

import json

import pytest

import tiny
from akas_b200.cli import main


def _config_text():
    data = dict(tiny.TINY_B)
    data.setdefault("architectures", ["Lfm2ForCausalLM"])
    return json.dumps(data)


def test_random_writes_a_folder_that_inspect_reads(tmp_path, capsys):
    main(["random", "--out", str(tmp_path / "inline"), "--config", _config_text(), "--seed", "4", "--dtype", "float32"])
    (tmp_path / "c.json").write_text(_config_text())
    main(["random", "--out", str(tmp_path / "file"), "--config", str(tmp_path / "c.json"), "--seed", "4", "--dtype", "float32"])
    capsys.readouterr()
    main(["inspect", "--model", str(tmp_path / "inline")])
    report = json.loads(capsys.readouterr().out)
    assert report["architecture"] == "Lfm2ForCausalLM"
    assert report["config"]["vocab_size"] == tiny.TINY_B["vocab_size"]
    assert "model.embed_tokens.weight" in report["inventory"]
    # the same seed gives the same tensors, whichever way the configuration came in
    assert (tmp_path / "inline" / "model.safetensors").read_bytes() == (tmp_path / "file" / "model.safetensors").read_bytes()


def test_prompt_must_be_token_ids(tmp_path):
    with pytest.raises(SystemExit):
        main(["generate", "--model", str(tmp_path), "--prompt", "hello world"])


@pytest.mark.gpu
def test_generate_and_bench_run(tmp_path, capsys):
    main(["random", "--out", str(tmp_path / "m"), "--config", _config_text(), "--seed", "5"])
    capsys.readouterr()
    main(["generate", "--model", str(tmp_path / "m"), "--prompt", "5,17 3", "--max-tokens", "6", "--out", str(tmp_path / "o.json")])
    printed = capsys.readouterr().out.split()
    saved = json.loads((tmp_path / "o.json").read_text())
    assert saved["prompt_tokens"] == [5, 17, 3] and [int(t) for t in printed] == saved["generated_tokens"]
    assert len(saved["generated_tokens"]) <= 6 and saved["finish_reason"] in ("length", "stop")
    main(["generate", "--model", str(tmp_path / "m"), "--prompt", "5 17 3", "--max-tokens", "6", "--temperature", "0.7",
          "--top-k", "20", "--seed", "2", "--dtype", "float32", "--ignore-eos"])
    assert len(capsys.readouterr().out.split()) == 6
    main(["bench", "--model", str(tmp_path / "m"), "--batches", "1", "2", "--prompts", "32", "--generated", "4", "--repeats", "2"])
    report = json.loads(capsys.readouterr().out)
    assert all(row["decode_tokens_per_s"] > 0 and row["prefill_tokens_per_s"] > 0 for row in report["rows"])
    # with tokens cached before the prompt, staggered lengths, and a comparison with an earlier report
    earlier = tmp_path / "earlier.json"
    main(["bench", "--model", str(tmp_path / "m"), "--batches", "3", "--prompts", "20", "--depths", "0", "24", "--mixed",
          "--generated", "3", "--repeats", "1", "--out", str(earlier)])
    report = json.loads(capsys.readouterr().out)
    assert [(row["depth"], row["mixed"]) for row in report["rows"]] == [(0, True), (24, True)]
    main(["bench", "--model", str(tmp_path / "m"), "--batches", "3", "--prompts", "20", "--depths", "0", "24", "--mixed",
          "--generated", "3", "--repeats", "1", "--baseline", str(earlier), "--max-regression", "0.99"])
    changes = json.loads(capsys.readouterr().out)["changes"]
    assert len(changes) == 2 and not any(change["regressed"] for change in changes)


def test_random_and_inspect_take_a_girelix_configuration(tmp_path, capsys):
    import tiny_girelix

    main(["random", "--out", str(tmp_path / "g"), "--config", json.dumps(tiny_girelix.CONFIGS["odd"]), "--seed", "2"])
    capsys.readouterr()
    main(["inspect", "--model", str(tmp_path / "g")])
    report = json.loads(capsys.readouterr().out)
    assert report["architecture"] == "Girelix" and report["config"] == json.loads(json.dumps(tiny_girelix.CONFIGS["odd"]))
    assert {"l0.mix.left.sink", "l1.mlp.e2.down", "l0.ls2", "head"} <= set(report["inventory"])


@pytest.mark.gpu
def test_generate_runs_a_girelix_folder(tmp_path, capsys):
    import tiny_girelix

    main(["random", "--out", str(tmp_path / "g"), "--config", json.dumps(tiny_girelix.CONFIGS["mix"]), "--seed", "2"])
    capsys.readouterr()
    for extra in ([], ["--temperature", "0.7", "--top-k", "20", "--seed", "2", "--dtype", "float32"]):
        main(["generate", "--model", str(tmp_path / "g"), "--prompt", "5 17 3 9", "--max-tokens", "7", "--ignore-eos", *extra])
        assert len(capsys.readouterr().out.split()) == 7


def test_random_and_inspect_take_a_penopel_configuration(tmp_path, capsys):
    import tiny_penopel

    config = tiny_penopel.CONFIGS["mix"]
    main(["random", "--out", str(tmp_path / "p"), "--config", json.dumps(config), "--seed", "4"])
    capsys.readouterr()
    main(["inspect", "--model", str(tmp_path / "p")])
    report = json.loads(capsys.readouterr().out)
    assert report["architecture"] == "Penopel" and report["config"] == json.loads(json.dumps(config))
    assert {"l0.norm1.alpha", "l0.mix.dkv.norm", "l0.mix.sink", "l1.mix.k.b", "l1.mlp.down.b", "l3.mix.q.b", "final.norm.b",
            "head"} <= set(report["inventory"])
    assert "l3.mix.k" not in report["inventory"]  # the layer reads another layer's keys and values


@pytest.mark.gpu
def test_generate_runs_a_penopel_folder(tmp_path, capsys):
    import tiny_penopel

    main(["random", "--out", str(tmp_path / "p"), "--config", json.dumps(tiny_penopel.CONFIGS["mix"]), "--seed", "4"])
    capsys.readouterr()
    for extra in ([], ["--temperature", "0.7", "--top-k", "20", "--seed", "2", "--dtype", "float32"]):
        main(["generate", "--model", str(tmp_path / "p"), "--prompt", "5 17 3 9", "--max-tokens", "7", "--ignore-eos", *extra])
        assert len(capsys.readouterr().out.split()) == 7


def test_random_and_inspect_take_a_kidarax_configuration(tmp_path, capsys):
    import tiny_kidarax

    config = tiny_kidarax.CONFIGS["mix"]
    main(["random", "--out", str(tmp_path / "k"), "--config", json.dumps(config), "--seed", "4"])
    capsys.readouterr()
    main(["inspect", "--model", str(tmp_path / "k")])
    report = json.loads(capsys.readouterr().out)
    assert report["architecture"] == "Kidarax" and report["config"] == json.loads(json.dumps(config))
    assert {"l0.norm1b.alpha", "l0.norm2b.b", "l0.mlp.router", "l0.mlp.e5.down", "l0.mlp.shared.sg", "l1.mix.dkv.norm", "l1.mix.sink",
            "l1.mlp.up", "l2.mix.k.b", "l2.mix.g", "final.norm.b"} <= set(report["inventory"])
    # no weight for the retention's norm, no head of its own, no shared expert where the layer names none, no feed-forward norms without a feed-forward
    assert not {"l0.mix.norm", "head", "l2.mlp.shared.gate", "l3.mlp.up"} & set(report["inventory"])


@pytest.mark.gpu
def test_generate_runs_a_kidarax_folder(tmp_path, capsys):
    import tiny_kidarax

    main(["random", "--out", str(tmp_path / "k"), "--config", json.dumps(tiny_kidarax.CONFIGS["mix"]), "--seed", "4"])
    capsys.readouterr()
    for extra in ([], ["--temperature", "0.7", "--top-k", "20", "--seed", "2", "--dtype", "float32"]):
        main(["generate", "--model", str(tmp_path / "k"), "--prompt", "5 17 3 9", "--max-tokens", "7", "--ignore-eos", *extra])
        assert len(capsys.readouterr().out.split()) == 7


def test_random_and_inspect_take_a_pekodra_configuration(tmp_path, capsys):
    import tiny_pekodra

    config = tiny_pekodra.CONFIGS["mix"]
    main(["random", "--out", str(tmp_path / "k"), "--config", json.dumps(config), "--seed", "4"])
    capsys.readouterr()
    main(["inspect", "--model", str(tmp_path / "k")])
    report = json.loads(capsys.readouterr().out)
    assert report["architecture"] == "Pekodra" and report["config"] == json.loads(json.dumps(config))
    assert {"loop.in", "head", "l0.norm1", "l0.norm2", "l0.mlp.router", "l0.mlp.e5.down", "l0.mlp.shared.up", "l1.mlp.gate.b",
            "l1.mlp.down.b", "l3.mix.v", "final.norm"} <= set(report["inventory"])
    # no gate matrices of experts, no shared gate, no biases in the mixer, no norm for a feed-forward that is not there
    assert not {"l0.mlp.e0.gate", "l0.mlp.shared.sg", "l0.mix.q.b", "l3.mlp.up"} & set(report["inventory"])


@pytest.mark.gpu
def test_generate_runs_a_pekodra_folder(tmp_path, capsys):
    import tiny_pekodra

    main(["random", "--out", str(tmp_path / "k"), "--config", json.dumps(tiny_pekodra.CONFIGS["mix"]), "--seed", "4"])
    capsys.readouterr()
    for extra in ([], ["--temperature", "0.7", "--top-k", "20", "--seed", "2", "--dtype", "float32"]):
        main(["generate", "--model", str(tmp_path / "k"), "--prompt", "5 17 3 9", "--max-tokens", "7", "--ignore-eos", *extra])
        assert len(capsys.readouterr().out.split()) == 7


def test_random_and_inspect_take_a_nuzulorn_configuration(tmp_path, capsys):
    import tiny_nuzulorn

    config = tiny_nuzulorn.CONFIGS["mix"]
    main(["random", "--out", str(tmp_path / "k"), "--config", json.dumps(config), "--seed", "4"])
    capsys.readouterr()
    main(["inspect", "--model", str(tmp_path / "k")])
    report = json.loads(capsys.readouterr().out)
    assert report["architecture"] == "Nuzulorn" and report["config"] == json.loads(json.dumps(config))
    assert {"embed", "bigram", "l0.norm1", "l0.norm2", "l0.mix.o.b", "l0.mix.g", "l0.mlp.correction", "l0.mlp.e5.gate", "l0.dwa", "l1.mix.lower",
            "l1.mix.f.b", "l1.mix.norm", "l2.mix.sink", "l4.dwa", "final.norm"} <= set(report["inventory"])
    # no head of its own, no output bias or gate of a capped layer, no bias of the matrix state's other projections
    assert not {"head", "l2.mix.o.b", "l2.mix.g", "l1.mix.q.b", "l2.mlp.router"} & set(report["inventory"])


@pytest.mark.gpu
def test_generate_runs_a_nuzulorn_folder(tmp_path, capsys):
    import tiny_nuzulorn

    main(["random", "--out", str(tmp_path / "k"), "--config", json.dumps(tiny_nuzulorn.CONFIGS["mix"]), "--seed", "4"])
    capsys.readouterr()
    for extra in ([], ["--temperature", "0.7", "--top-k", "20", "--seed", "2", "--dtype", "float32"]):
        main(["generate", "--model", str(tmp_path / "k"), "--prompt", "5 17 3 9", "--max-tokens", "7", "--ignore-eos", *extra])
        assert len(capsys.readouterr().out.split()) == 7
