"""The Nuzulorn decoder in the engine against the plain float64 statement of it (``plain_nuzulorn``).

Small configurations of the tests' own, random weights shaped so that faults show (norm weights, biases and sinks that are
not small, gates that forget slowly and fast, routers whose scores spread), and every way of cutting and batching. The
same tests run on a CPU with the plain PyTorch statements of the kernels (host logic: pages behind a window, blocks in
front of it, the previous token in a request's slot) and, marked ``gpu``, with the compiled kernels in float32 and
bfloat16. The kernels' new options are also compared one by one with their plain statements.
"""

import json
import math
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import plain_nuzulorn as plain
import traces

from tiny_nuzulorn import (ATT, ATT_LONG_BLOCK, ATT_MID, ATT_ODD, ATT_ONES, ATT_SELF, ATT_SHORT, ATT_WIDE, CAP, CAP_NEG, CAP_NEVER, CAP_STEP,
                           CONFIGS, HG, HG_WIDE, LENGTHS, PAGE, TOL, attn, capped, hgrn, layer, make_folder, model, moe, plant, prompts)

ROOT = Path(__file__).resolve().parent.parent
# A routing margin (the gap between two choice scores, or between the sums of two groups) below this may fall the other
# way: in bfloat16 through the rounding of the router's input and of the layers before it, in float32 through the order of sums.
CLOSE_CALL = {"float32": 2e-4, "bfloat16": 0.04}


def runner_for(folder, dtype, device, page, max_tokens, ops=None, max_requests=4, context=None, **kw):
    from akas_b200.config import EngineConfig
    from akas_b200.engine.runner import ModelRunner

    cfg = EngineConfig(dtype=dtype, device=device, page_size=page, max_tokens=max_tokens, max_requests=max_requests,
                       context=context or max_tokens, cuda_graphs=False, **kw)
    return ModelRunner(folder, cfg, ops=ops)


def oracle(config, w, tokens):
    """(logits [T, vocab], margin [T]): the least routing margin of a position over all routed layers; where it is a close
    call, the engine may decide the other way (and every later position may feel it through the mixers)."""
    margins = []
    logits = plain.forward(tokens, w, config, margins=margins).numpy()
    least = np.full(len(tokens), np.inf)
    for per_layer in margins:
        least = np.minimum(least, np.asarray(per_layer))
    return logits, least


def compare(got, want, dtype, what):
    for rid, (logits, least) in want.items():
        rows = np.nonzero(least >= CLOSE_CALL[dtype])[0]
        if dtype != "float32":
            error = np.abs(got[rid] - logits).max(axis=-1) / np.abs(logits).max()
            if len(error) > 3:
                assert np.median(error) <= 0.4 * TOL[dtype], f"{what}: request {rid}: median error {np.median(error):.3g}"
            if len(rows) == 0:
                continue
        bad = traces.first_bad(got[rid][rows], logits[rows], TOL[dtype])
        assert bad is None, (f"{what}: request {rid} first differs at position {rows[bad]} "
                             f"{traces.worst(got[rid][rows], logits[rows])}")


def run_modes(key, dtype, device, ops, tmp_path, modes):
    config = CONFIGS[key]
    folder, w = make_folder(config, seed=31, folder=tmp_path / key)
    reqs = {f"r{i}": p for i, p in enumerate(prompts(config["vocab"], LENGTHS[key], seed=6))}
    want = {rid: oracle(config, w, toks) for rid, toks in reqs.items()}
    page = PAGE[key]
    longest = -(-max(len(t) for t in reqs.values()) // page) * page
    for mode in modes:
        if mode == "mixed":
            steps, peak = traces.mixed(reqs, {rid: max(1, len(t) - 9) for rid, t in reqs.items()}, seed=3, live=3, page=page)
            runner = runner_for(folder, dtype, device, page, peak, ops, max_requests=3, context=longest)
        else:
            steps = getattr(traces, mode)(reqs)
            runner = runner_for(folder, dtype, device, page, longest, ops, max_requests=2)
        got = traces.replay(runner, steps)
        assert not runner.cache.live() and runner.cache.min_free_pages() == runner.cache.num_pages
        compare(got, want, dtype, f"{key}/{dtype}/{mode}")


MODES = ["whole", "tail_decoded", "portions", "mixed"]


@pytest.mark.parametrize("key", list(CONFIGS))
def test_every_way_of_cutting_on_the_plain_operations(key, tmp_path):
    from akas_b200.ops import reference

    run_modes(key, "float32", "cpu", reference, tmp_path, MODES)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("key", list(CONFIGS))
def test_every_way_of_cutting_on_the_kernels(key, dtype, tmp_path):
    run_modes(key, dtype, "cuda:0", None, tmp_path, MODES)


def test_config_round_trip_registry_and_inventory(tmp_path):
    from akas_b200.config import ConfigError, NuzulornConfig, config_from_dict, load_config
    from akas_b200.engine.runner import kernel_kinds
    from akas_b200.ops import reference
    from akas_b200.weights.loader import WeightError

    config = config_from_dict(CONFIGS["mix"])
    assert isinstance(config, NuzulornConfig) and config_from_dict(config.to_dict()) == config
    assert config_from_dict(json.loads(json.dumps(config.to_dict()))) == config
    spec = config.model_spec()
    assert [e.layer for e in spec.run_order()] == [0, 1, 2, 3, 4] and [e.average for e in spec.schedule] == [f"l{i}.dwa" for i in range(5)]
    assert all(l.arrangement == "pre_norm" and l.residual_multiplier == 0.6 and not l.mixer_norm.zero_centered for l in spec.layers)
    pooled, gated, cap = (spec.layers[i].mixer for i in (0, 1, 2))
    assert (pooled.window, pooled.pool, pooled.sink, pooled.gate, pooled.bias, pooled.out_bias) == (21, 8, True, "head", True, True)
    assert pooled.position.rotary == 16 and pooled.value_dim == 16 and pooled.softcap is None and pooled.general
    assert gated.kind == "hgrn2" and (gated.num_heads, gated.key_dim, gated.value_dim, gated.norm_eps) == (3, 12, 10, 1e-5)
    assert (cap.softcap, cap.distance_bias, cap.sink, cap.q_temperature, cap.out_bias) == (4.0, "linear", "learned", (0.5, 11), False)
    assert cap.position is None and cap.window is None and cap.gate is None and cap.bias and spec.layers[2].ffn is None
    ffn = spec.layers[0].ffn
    assert (ffn.scoring, ffn.renormalize, ffn.correction, ffn.groups, ffn.keep_groups, ffn.group_best) == ("sigmoid", False, True, 3, 2, 2)
    assert ffn.weight_scale == 1.7 and ffn.gated and ffn.shared_size is None
    assert spec.head_name is None and (spec.bigram.buckets, spec.bigram.mul_prev, spec.bigram.mul_cur) == (97, 31, 7)
    assert set(kernel_kinds(spec)) == {"attention_general", "rope", "moe", "recurrent"}
    folder, _ = make_folder(CONFIGS["odd"], seed=1, folder=tmp_path / "m")
    assert load_config(folder) == config_from_dict(CONFIGS["odd"])
    # a router without groups chooses among all experts, one without a scale weighs by the scores
    bare = json.loads(json.dumps(CONFIGS["odd"]))
    del bare["layers"][0]["mlp"]["router"]["groups"], bare["layers"][0]["mlp"]["router"]["scale"]
    ffn = config_from_dict(bare).model_spec().layers[0].ffn
    assert (ffn.groups, ffn.keep_groups, ffn.weight_scale) == (1, 1, 1.0)
    for change, message in ((lambda c: c["layers"][2]["mixer"].update(kv_heads=2), "kv_heads"),
                            (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "size"),
                            (lambda c: c["layers"][2]["mixer"]["mask"].pop("pool"), "pool"),
                            (lambda c: c["layers"][2]["mixer"].pop("mask"), "mask"),
                            (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=5), "rot.dims"),
                            (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=22), "rot.dims"),
                            (lambda c: c["layers"][0]["mixer"].update(softcap=0), "softcap"),
                            (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "every"),
                            (lambda c: c["layers"][0]["mixer"].pop("q_temp"), "q_temp"),
                            (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
                            (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
                            (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3), "keep"),
                            (lambda c: c["layers"][4]["mlp"]["router"].update(top=7), "top"),
                            (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
                            (lambda c: c["embedding"].pop("bigram"), "bigram"),
                            (lambda c: c.pop("residual_mult"), "residual_mult"),
                            (lambda c: c["layers"][0].update(type="retention"), "type")):
        broken = json.loads(json.dumps(CONFIGS["odd"]))
        change(broken)
        with pytest.raises(ConfigError, match=message):
            config_from_dict(broken)
    # a checkpoint without one of the averages, or with a tensor the design does not have, is refused
    from safetensors.torch import load_file, save_file

    tensors = load_file(str(folder / "model.safetensors"))
    assert tensors["bigram"].shape == (14, 52) and tensors["l3.dwa"].shape == (5,) and tensors["l2.mix.o.b"].shape == (52,)
    assert tensors["l2.mix.g"].shape == (3, 52) and "l0.mix.o.b" not in tensors and tensors["l1.mix.lower"].shape == (40,)
    assert "l1.norm2" not in tensors and "head" not in tensors
    del tensors["l3.dwa"]
    tensors["l0.mix.o.b"] = torch.ones(52, dtype=torch.bfloat16)
    tensors["l1.norm2"] = torch.ones(52, dtype=torch.bfloat16)  # the norm that a feed-forward would have: may lie about
    save_file(tensors, str(folder / "model.safetensors"))
    with pytest.raises(WeightError, match="l3.dwa") as caught:
        runner_for(folder, "float32", "cpu", 8, 64, reference)
    assert "l0.mix.o.b" in str(caught.value) and "l1.norm2" not in str(caught.value)


# --------------------------------------------------------------------------- each mechanism alone


def one_mechanism(config, tmp_path, seed=5, length=60, page=8):
    """The engine on the plain operations against the oracle for a small model that isolates a mechanism."""
    from akas_b200.ops import reference

    folder, w = make_folder(config, seed=seed, folder=tmp_path / "one")
    toks = prompts(config["vocab"], [length], seed=seed)[0]
    runner = runner_for(folder, "float32", "cpu", page, -(-length // page) * page, reference)
    got = traces.replay(runner, traces.portions({"a": toks}, sizes=(9, 1, 2, 17)))["a"]
    want = plain.forward(toks, w, config).numpy()
    assert traces.first_bad(got, want, TOL["float32"]) is None, traces.worst(got, want)
    return w, toks, want


def felt(changed, want, least=3e-4):
    assert np.abs(changed - want).max() > least * np.abs(want).max(), "the mechanism does not show in the logits"


@pytest.mark.parametrize("mixer", [ATT, ATT_LONG_BLOCK, ATT_ODD, ATT_SHORT, ATT_SELF, ATT_ONES, ATT_WIDE])
def test_windows_with_blocks_alone(mixer, tmp_path, monkeypatch):
    config = model(48, 60, [layer(mixer, None)])
    w, toks, want = one_mechanism(config, tmp_path)
    if mixer is not ATT_WIDE:  # an edge one token or one block off, in the oracle, shows
        for name, wrong in (("sees_token", lambda i, j, window: 0 <= i - j <= window),
                            ("sees_block", lambda i, b, window, pool: (b + 1) * pool - 1 < i - window),
                            ("sees_block", lambda i, b, window, pool: (b + 1) * pool - 1 <= i - window + 1),
                            ("sees_block", lambda i, b, window, pool: b * pool <= i - window),
                            ("sees_block", lambda *_: False)):
            with monkeypatch.context() as patch:
                patch.setattr(plain, name, wrong)
                if name == "sees_block" and mixer is ATT_ONES and wrong(0, 0, 1, 1) == plain.sees_block(0, 0, 1, 1) and wrong(5, 2, 3, 1):
                    continue  # (blocks of one token: where a block begins is where it ends)
                felt(plain.forward(toks, w, config).numpy(), want)
    sinkless = plain.attend
    monkeypatch.setattr(plain, "attend", lambda q, k, v, s, level: torch.softmax(s, dim=-1) @ v)
    felt(plain.forward(toks, w, config).numpy(), want)
    monkeypatch.setattr(plain, "attend", sinkless)
    for name in ("mix.q.b", "mix.k.b", "mix.v.b", "mix.o.b", "mix.g"):
        felt(plain.forward(toks, dict(w, **{"l0." + name: torch.zeros_like(w["l0." + name])}), config).numpy(), want)


def test_blocks_of_one_token_are_plain_attention():
    """With blocks of one token, a window and the blocks in front of it hold every token up to the query's own."""
    for i in range(40):
        seen = [j for j in range(40) if plain.sees_token(i, j, 9)] + [b for b in range(40) if plain.sees_block(i, b, 9, 1)]
        assert sorted(seen) == list(range(i + 1))
    # with longer ones, tokens that the window has passed wait until the last of their block has left it too
    assert plain.sees_block(30, 1, 15, 8) and not plain.sees_token(30, 15, 15)
    assert not plain.sees_block(29, 1, 15, 8) and plain.sees_token(29, 15, 15) and not plain.sees_token(29, 14, 15)


@pytest.mark.parametrize("mixer", [CAP, CAP_STEP, CAP_NEVER, CAP_NEG])
def test_capped_attention_alone(mixer, tmp_path, monkeypatch):
    config = model(48, 60, [layer(mixer, None)])
    w, toks, want = one_mechanism(config, tmp_path)
    m = config["layers"][0]["mixer"]
    if mixer is not CAP_NEVER:
        felt(plain.forward(toks, w, dict(config, layers=[layer(dict(m, q_temp=dict(coef=0.0, every=1)), None)])).numpy(), want)
        step = plain.temperature  # the step at p + 1 = every, not at p = every
        monkeypatch.setattr(plain, "temperature", lambda T, t: torch.cat([torch.ones(1, dtype=plain.F), step(T, t)[:-1]]))
        felt(plain.forward(toks, w, config).numpy(), want)
        monkeypatch.setattr(plain, "temperature", step)
        felt(plain.forward(toks, w, dict(config, layers=[layer(dict(m, softcap=1e6), None)])).numpy(), want)
    assert plain.temperature(3, dict(coef=0.5, every=2)).tolist() == [1.0, 1.0 + 0.5 * math.log(2.0), 1.0 + 0.5 * math.log(2.0)]
    for wrong in (lambda a, heads: 0.0, lambda a, heads: 2.0 ** (-8.0 * a / heads)):
        with monkeypatch.context() as patch:
            patch.setattr(plain, "slope", wrong)
            felt(plain.forward(toks, w, config).numpy(), want)
    felt(plain.forward(toks, dict(w, **{"l0.mix.sink": torch.full_like(w["l0.mix.sink"], -1e9)}), config).numpy(), want)


@pytest.mark.parametrize("mixer", [HG, HG_WIDE, hgrn(1, 5, 33)])
def test_forget_gates_that_write_alone(mixer, tmp_path):
    config = model(48, 60, [layer(mixer, None)])
    w, toks, want = one_mechanism(config, tmp_path)
    for name in ("mix.lower", "mix.f.b"):
        felt(plain.forward(toks, dict(w, **{"l0." + name: torch.zeros_like(w["l0." + name])}), config).numpy(), want)


def test_forget_gates_written_out():
    """The operation against the recurrence in closed form: what a token wrote is weighed by the products of the gates
    behind it."""
    from akas_b200.ops import reference

    g = torch.Generator().manual_seed(2)
    n, heads, dim, vdim = 11, 2, 6, 5
    q, f, v = (torch.randn(n, heads * width, generator=g) for width in (dim, dim, vdim))
    bias, lower = torch.randn(heads * dim, generator=g), torch.rand(heads * dim, generator=g)
    state = torch.zeros(3, heads, vdim, dim)
    cu, slots = torch.tensor([0, 4, n], dtype=torch.int32), torch.tensor([2, -1], dtype=torch.int32)
    got = reference.hgrn2_scan(q, f, v, bias, lower, state, cu, slots, heads, dim, vdim)
    assert (got[4:] == 0).all() and (state[:2] == 0).all()
    gate = (lower + (1 - lower) * torch.sigmoid(f + bias)).double().reshape(n, heads, dim)
    qa = plain.silu(q.double()).reshape(n, heads, dim)
    for t in range(4):
        want = torch.zeros(heads, vdim, dtype=torch.float64)
        for s in range(t + 1):
            share = (1 - gate[s]) * torch.prod(gate[s + 1 : t + 1], dim=0)
            want += (qa[t] * share).sum(-1, keepdim=True) * v[s].double().reshape(heads, vdim)
        assert (got[t].double().reshape(heads, vdim) - want).abs().max() < 1e-5


@pytest.mark.parametrize("mlp", [moe(24, 6, 2, groups=3, keep=1, scale=1.7), moe(16, 8, 3, groups=2, keep=1), moe(12, 6, 2, groups=6, keep=4),
                                 moe(8, 3, 3, scale=0.4), moe(20, 8, 4, groups=4, keep=4, scale=2.5), moe(12, 1, 1)])
def test_experts_alone(mlp, tmp_path):
    config = model(48, 60, [layer(ATT_WIDE, mlp)])
    w, toks, want = one_mechanism(config, tmp_path)
    if mlp["router"]["experts"] > mlp["router"]["top"]:
        felt(plain.forward(toks, dict(w, **{"l0.mlp.correction": -w["l0.mlp.correction"]}), config).numpy(), want)
    if mlp["router"]["scale"] != 1.0:
        felt(plain.forward(toks, w, dict(config, layers=[layer(ATT_WIDE, dict(mlp, router=dict(mlp["router"], scale=1.0)))])).numpy(), want)


def test_groups_are_judged_by_their_two_best_scores():
    """One group holds the largest choice score, another the two largest sums: the second stays. Negative choice scores
    compare as they are, and an expert of a group that is out is never chosen, whatever the others hold."""
    from akas_b200.ops import reference

    def logit(p):
        return math.log(p / (1.0 - p))

    scores = torch.tensor([0.95, 0.1, 0.2, 0.7, 0.65, 0.05, 0.6, 0.3, 0.1], dtype=torch.float64)
    w = torch.diag(torch.tensor([logit(float(s)) for s in scores]))
    h = torch.eye(9).sum(0, keepdim=True)
    for correction in (torch.zeros(9), torch.full((9,), -2.0)):
        chosen, weights = reference.moe_route(h, w.float(), correction, 3, 1, 2, scoring="sigmoid", renormalize=False, group_best=2, weight_scale=3.0)
        assert chosen.tolist() == [[3, 4]] and np.allclose(weights.numpy(), [[2.1, 1.95]], atol=1e-5)
        single, _ = reference.moe_route(h, w.float(), correction, 3, 1, 2, scoring="sigmoid", renormalize=False)
        assert single.tolist() == [[0, 2]]
        two, _ = reference.moe_route(h, w.float(), correction, 3, 2, 4, scoring="sigmoid", renormalize=False, group_best=2)
        assert two.tolist() == [[0, 3, 4, 2]]
        want, _ = plain.route(h.double(), {"router": w.double(), "correction": correction.double()}, "",
                              dict(experts=9, top=2, groups=dict(count=3, keep=1), scale=3.0))
        assert want.tolist() == [[3, 4]]
    # without a correction the groups still go by sums of scores, not of logits
    far = torch.diag(torch.tensor([9.0, 0.1, 0.0, 1.2, 1.1, 0.0]))
    chosen, _ = reference.moe_route(torch.ones(1, 6), far, None, 2, 1, 2, scoring="sigmoid", renormalize=False, group_best=2)
    assert chosen.tolist() == [[0, 1]] or torch.sigmoid(torch.tensor([9.0, 0.1])).sum() < torch.sigmoid(torch.tensor([1.2, 1.1])).sum()


def test_the_token_in_front_is_part_of_a_requests_state(tmp_path):
    """Rows of the second table against the oracle's hash for requests cut at every place, one token at a time included,
    several requests in a step, a request that sits a step out and a slot that is used again."""
    from akas_b200.ops import reference

    big = dict(buckets=13, mul_prev=1000003, mul_cur=99991)
    g = torch.Generator().manual_seed(4)
    table, pairs = torch.randn(40, 6, generator=g), torch.randn(14, 6, generator=g)
    state = torch.zeros(3, 1, dtype=torch.int32)
    a, b, c = prompts(40, [9, 5, 4], seed=1)
    at = {"a": 0, "b": 0, "c": 0}
    toks, slot = {"a": a, "b": b, "c": c}, {"a": 2, "b": 0, "c": 2}
    for step in ([("a", 3)], [("b", 1), ("a", 1)], [("b", 2)], [("a", 5), ("b", 2)], [("c", 1)], [("c", 3)]):
        if step[0][0] == "c" and at["c"] == 0:
            state[2] = 0  # the slot goes to another request: admission leaves it empty
        ids, seq, cu = [], [], [0]
        for i, (rid, count) in enumerate(step):
            ids += toks[rid][at[rid] : at[rid] + count]
            seq += [i] * count
            cu.append(len(ids))
        ids += [7]  # a token of no request
        seq += [-1]
        tensors = [torch.tensor(x, dtype=torch.int32) for x in (ids, cu, seq, [slot[rid] for rid, _ in step])]
        got = reference.bigram_embedding(tensors[0], table, pairs, big["mul_prev"], big["mul_cur"], state, *tensors[1:])
        row = 0
        for rid, count in step:
            rows = plain.bigram_rows(toks[rid], big)
            for k in range(count):
                p = at[rid] + k
                assert torch.allclose(got[row], table[toks[rid][p]] + pairs[rows[p]]), (rid, p)
                row += 1
            at[rid] += count
        assert torch.equal(got[row], table[7])
    assert plain.bigram_rows([3, 5], big) == [13, (3 * 1000003 + 5 * 99991) % 13]


def test_second_table_and_averages_show(tmp_path):
    config = model(48, 60, [layer(HG, moe(16, 4, 2)), layer(CAP, None), layer(ATT, moe(8, 3, 1))])
    w, toks, want = one_mechanism(config, tmp_path)
    felt(plain.forward(toks, dict(w, bigram=torch.zeros_like(w["bigram"])), config).numpy(), want)
    moved = w["bigram"].clone()
    moved[-1] = moved[0]
    felt(plain.forward(toks, dict(w, bigram=moved), config).numpy(), want)
    for i in range(3):
        for j in range(i + 2):
            changed = w[f"l{i}.dwa"].clone()
            changed[j] += 0.2
            felt(plain.forward(toks, dict(w, **{f"l{i}.dwa": changed}), config).numpy(), want)
    # the averages take the layers' results, not what earlier averages made of them
    x = plain.embed(toks, w, config)
    for i, entry in enumerate(config["layers"]):
        y = x + 0.6 * plain.mixer(plain.norm(x, w[f"l{i}.norm1"], 1e-5), w, f"l{i}.mix.", entry, 1e-5)
        if entry["mlp"]:
            y = y + 0.6 * plain.mixture(plain.norm(y, w[f"l{i}.norm2"], 1e-5), w, f"l{i}.mlp.", entry["mlp"])
        kept = [plain.embed(toks, w, config)] if i == 0 else kept
        x = plain.depth_average(kept + [y], w[f"l{i}.dwa"])
        kept.append(x)
    felt((plain.norm(x, w["final.norm"], 1e-5) @ w["embed"].T).numpy(), want)


def test_averages_behind_some_layers_only():
    """A run order in which only some entries are followed by an average, a layer runs twice, and the mixer does not add in
    place: the decoder against the sums written out."""
    from akas_b200.config import LayerSpec, ModelSpec, RMSNormSpec, ScheduleEntry
    from akas_b200.engine.batch import StepContext
    from akas_b200.models.decoder import Decoder
    from akas_b200.ops import reference
    from akas_b200.parts.base import Mixer, Runtime, register_mixer

    class Triple(Mixer):
        def forward(self, x, ctx, cache=None, residual=None, write=True):
            out = 3.0 * x.to(torch.float32)
            return out if residual is None else residual + out

    register_mixer("test_triple", Triple)

    class Spec:
        kind = "test_triple"

    norm = RMSNormSpec(12, 1e-5)
    layers = tuple(LayerSpec(Spec(), None, norm, None, f"m{i}.", "f.", f"n{i}", None, residual_multiplier=mult) for i, mult in enumerate((1.0, 0.5)))
    order = (ScheduleEntry(0), ScheduleEntry(1, average="a1"), ScheduleEntry(0, average="a2"), ScheduleEntry(1))
    for last in (None, "a3"):
        schedule = order[:3] + (ScheduleEntry(1, average=last),)
        decoder = Decoder(ModelSpec("T", 12, 20, layers, norm, "embed", "final", None, schedule=schedule, embedding_multiplier=2.0),
                          Runtime(torch.float32, torch.device("cpu"), reference))
        g = torch.Generator().manual_seed(5)
        w = {k: torch.randn(p.shape, generator=g) for k, p in decoder.params().items()}
        assert w["a1"].shape == (3,) and w["a2"].shape == (4,)
        decoder.load(lambda name: w[name])
        ids = torch.tensor([3, 9, 11, 0], dtype=torch.int32)
        rows = torch.tensor([2, 0], dtype=torch.int32)
        zero = torch.zeros(4, dtype=torch.int32)
        ctx = StepContext(4, 1, ids, zero, zero, zero[:2], zero[:1], rows, 2, [], 4, 4, False)
        got = decoder.forward(ctx, [None] * 4)
        d = {k: v.double() for k, v in w.items()}
        x = d["embed"][ids.long()] * 2.0
        results = [x]
        for layer_, mult, average in ((0, 1.0, None), (1, 0.5, "a1"), (0, 1.0, "a2"), (1, 0.5, last)):
            x = x + mult * 3.0 * plain.norm(x, d[f"n{layer_}"], 1e-5)
            results.append(x)
            if average:
                x = plain.depth_average(results, d[average])
        want = plain.norm(x, d["final"], 1e-5)[rows.long()] @ d["embed"].T
        assert (got.double() - want).abs().max() < 1e-5 * want.abs().max()


# --------------------------------------------------------------------------- what a position sees


WINDOW, BLOCK = 130, 3
SEEN = attn(4, 2, 24, 16, WINDOW, BLOCK, 0.25, 300.0, 16)


def seen_config():
    # a hash that ignores the token in front: a changed token then changes its own position's input only
    # (a wide one: a key that points along the query stands out of random ones by the root of the width)
    return model(192, 120, [layer(SEEN, None)], buckets=11, mul_prev=22, mul_cur=3, mult=1.0)


def seen_case(device, dtype, ops, tmp_path, decode, page):
    """One layer: the logits at position i change with the token at position j iff j is in i's window or in a block that
    lies wholly in front of it: at both sides of both edges, at page borders, the query itself; the tokens between the
    last whole block and the window never, nor later ones; with the query in a prompt's portion or decoded alone."""
    from akas_b200.engine.batch import StepEntry

    config = seen_config()
    folder, _ = make_folder(config, seed=44, folder=tmp_path / "edge")
    w = plant(folder, config, key_token=119, query_token=118, strength=0.7)  # token 119 at position j is felt by token 118 at position i
    for i in (290, 297):
        first = i - WINDOW + 1               # the window's first token
        whole = first // BLOCK * BLOCK        # tokens in front of this one are in whole blocks
        base = prompts(118, [300], seed=9)[0]
        base[i] = 118
        cases = sorted({0, 1, BLOCK - 1, BLOCK, 63, 64, whole - BLOCK - 1, whole - BLOCK, whole - 1, whole, first - 1, first, first + 1, 191, 192, 255, 256,
                        i - 1, i, i + 1, 299})

        def logits_at_i(tokens):
            runner = runner_for(folder, dtype, device, page, 320, ops)
            if decode:
                runner.step([StepEntry("a", tokens[:i], ())])
                out = runner.step([StepEntry("a", tokens[i:i + 1], (0,))])
            else:
                runner.step([StepEntry("a", tokens[:277], ())])
                out = runner.step([StepEntry("a", tokens[277:], (i - 277,))])
            return out.float().cpu().numpy()[0]

        ref = logits_at_i(base)
        for j in cases:
            seen = j < whole or first <= j <= i
            assert seen == (plain.sees_token(i, j, WINDOW) or plain.sees_block(i, j // BLOCK, WINDOW, BLOCK))
            changed = list(base)
            changed[j] = 119 if j != i else 7
            got = logits_at_i(changed)
            diff = np.abs(got - ref).max()
            if seen:
                assert diff > (2e-2 if j >= first else 5e-4) * np.abs(ref).max(), f"position {i} does not see {j} ({diff})"
            else:
                assert diff == 0.0, f"position {i} sees {j} (difference {diff})"
            if dtype == "float32" and j in (whole - 1, first):
                want = plain.forward(changed[: i + 1], w, config)[i].numpy()
                assert np.abs(got - want).max() <= TOL[dtype] * np.abs(want).max()


@pytest.mark.parametrize("page", [8, 12])
@pytest.mark.parametrize("decode", [False, True])
def test_what_a_position_sees_on_the_plain_operations(decode, page, tmp_path):
    from akas_b200.ops import reference

    seen_case("cpu", "float32", reference, tmp_path, decode, page)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page", [12, 64])
@pytest.mark.parametrize("decode", [False, True])
def test_what_a_position_sees_on_the_kernels(decode, page, dtype, tmp_path):
    seen_case("cuda:0", dtype, None, tmp_path, decode, page)


FAR = {"capped": capped(4, 2, 24, 16, 1.0, 30.0, 0.3, 64), "window": attn(4, 2, 24, 16, 497, 4, 1.0, 300.0, 16)}


def far_key_case(device, dtype, ops, tmp_path, kind, page):
    """One key far back among hundreds is made to stand out: at the start of a causal layer's context; as the oldest key
    that a window still holds, where one position further back it is a part of no whole block yet. The last position's
    attention must find it through scattered pages, in a portion and decoded alone."""
    from akas_b200.engine.batch import StepEntry

    config = dict(seen_config(), layers=[layer(FAR[kind], None)])
    folder, _ = make_folder(config, seed=47, folder=tmp_path / "far")
    w = plant(folder, config, key_token=119, query_token=118, strength=0.5)
    toks = prompts(118, [500], seed=2)[0]
    toks[3], toks[-1] = 119, 118  # position 499 sees positions 3..499 in the window; block 0 holds position 3 as well
    want = plain.forward(toks, w, config)[-1].numpy()
    moved = list(toks)
    moved[3], moved[2] = toks[2], 119
    past = plain.forward(moved, w, config)[-1].numpy()
    without = list(toks)
    without[3] = 5
    assert np.abs(plain.forward(without, w, config)[-1].numpy() - want).max() > 0.05 * np.abs(want).max(), "the far key does not stand out"
    if kind == "window":
        assert np.abs(past - want).max() > 0.05 * np.abs(want).max()
    for tokens, expected in ((toks, want), (moved, past)):
        for cuts in ([500], [499, 1], [130, 70, 2, 290, 8]):
            runner = runner_for(folder, dtype, device, page, 640, ops, context=512)
            runner.admit("other")  # the request's pages are not the pool's first
            runner.cache.reserve("other", 40)
            at = 0
            for c in cuts:
                out = runner.step([StepEntry("a", tokens[at:at + c], (c - 1,) if at + c == 500 else ())])
                at += c
            got = out.float().cpu().numpy()[0]
            assert np.abs(got - expected).max() <= TOL[dtype] * np.abs(expected).max(), cuts


@pytest.mark.parametrize("kind", list(FAR))
def test_a_far_key_is_found_on_the_plain_operations(kind, tmp_path):
    from akas_b200.ops import reference

    far_key_case("cpu", "float32", reference, tmp_path, kind, 16)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", list(FAR))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_is_found_on_the_kernels(dtype, kind, tmp_path):
    far_key_case("cuda:0", dtype, None, tmp_path, kind, 64)


def far_block_case(device, dtype, ops, tmp_path):
    """A whole block of one token far in front of the window is one key that stands out, once all of it is in front: one
    position earlier the same block, of which the window has passed all but the last token, is not seen at all."""
    from akas_b200.engine.batch import StepEntry

    config = dict(seen_config(), layers=[layer(attn(4, 2, 24, 16, 100, 12, 1.0, 300.0, 16), None)])
    folder, _ = make_folder(config, seed=48, folder=tmp_path / "block")
    w = plant(folder, config, key_token=119, query_token=118, strength=0.5)
    toks = prompts(118, [400], seed=2)[0]
    toks[24:36] = [119] * 12  # block 2
    for i in (134, 135, 136, 260, 399):
        cut = list(toks[: i + 1])
        cut[i] = 118
        want = plain.forward(cut, w, config)[i].numpy()
        other = list(cut)
        other[24:36] = prompts(118, [12], seed=3)[0]
        felt_here = np.abs(plain.forward(other, w, config)[i].numpy() - want).max() / np.abs(want).max()
        assert felt_here > 0.1, (i, felt_here)  # (at 134 the window still holds the block's last token)
        for cuts in ([i + 1], [i, 1], [30, 2, i - 40, 9]):
            runner = runner_for(folder, dtype, device, 16, 448, ops)
            at = 0
            for c in cuts:
                out = runner.step([StepEntry("a", cut[at:at + c], (c - 1,) if at + c == i + 1 else ())])
                at += c
            got = out.float().cpu().numpy()[0]
            assert np.abs(got - want).max() <= TOL[dtype] * np.abs(want).max(), (i, cuts)


def test_a_far_block_is_found_on_the_plain_operations(tmp_path):
    from akas_b200.ops import reference

    far_block_case("cpu", "float32", reference, tmp_path)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_block_is_found_on_the_kernels(dtype, tmp_path):
    far_block_case("cuda:0", dtype, None, tmp_path)


def reuse_case(device, dtype, ops, tmp_path):
    """Two requests one after the other in a pool of one slot and just enough pages: the second gets the first one's pages,
    blocks, matrix state and slot, and must compute as if it were alone (its first token has no token in front)."""
    from akas_b200.engine.batch import StepEntry

    config = CONFIGS["odd"]
    folder, w = make_folder(config, seed=12, folder=tmp_path / "m")
    a, b = prompts(config["vocab"], [90, 86], seed=5)
    runner = runner_for(folder, dtype, device, 16, 96, ops, max_requests=1)
    runner.step([StepEntry("a", a, ())])
    runner.release("a")
    runner.step([StepEntry("b", b[:41], ())])
    got = runner.step([StepEntry("b", b[41:], tuple(range(45)))]).float().cpu().numpy()
    logits, least = oracle(config, w, b)
    compare({"b": got}, {"b": (logits[41:], least[41:])}, dtype, "a slot used again")


def test_freed_pages_and_slots_are_used_again_and_not_read(tmp_path):
    from akas_b200.ops import reference

    reuse_case("cpu", "float32", reference, tmp_path)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_freed_pages_and_slots_on_the_kernels(dtype, tmp_path):
    reuse_case("cuda:0", dtype, None, tmp_path)


def test_pages_of_an_unfinished_block_stay(tmp_path):
    """A window of 5 tokens has long passed the first tokens of a block of 40 when its last one comes: their pages stay
    until then and go back behind it; and a page that one request left behind serves another one."""
    from akas_b200.engine.batch import StepEntry
    from akas_b200.ops import reference

    config = model(48, 60, [layer(attn(4, 2, 8, 12, 5, 40, 0.6, 300.0, 8), None), layer(attn(2, 1, 12, 8, 9, 6, 0.6, 300.0, 4), moe(16, 3, 1))])
    folder, w = make_folder(config, seed=12, folder=tmp_path / "m")
    a, b = prompts(60, [120, 50], seed=5)
    runner = runner_for(folder, "float32", "cpu", 8, 176, reference, max_requests=2, context=120)
    groups = runner.cache.groups
    assert sorted((g.window or 0, g.pool) for g in groups) == [(0, 0), (5, 40), (9, 6)]  # both layers' blocks share one
    long_block = next(i for i, g in enumerate(groups) if g.pool == 40)
    want = {"a": plain.forward(a, w, config).numpy(), "b": plain.forward(b, w, config).numpy()}
    at = {"a": 0, "b": 0}
    for step in range(60):
        entries = [StepEntry("a", a[at["a"]:at["a"] + 2], (0, 1))]
        if step >= 10 and at["b"] < len(b):
            entries.append(StepEntry("b", b[at["b"]:at["b"] + 1], (0,)))
        got = runner.step(entries).numpy()
        row = 0
        for e in entries:
            for k in range(len(e.tokens)):
                err = np.abs(got[row] - want[e.request][at[e.request] + k]).max() / np.abs(want[e.request]).max()
                assert err <= TOL["float32"], (step, e.request, k, err)
                row += 1
            at[e.request] += len(e.tokens)
        runner.cache.check()
        held = [p >= 0 for p in runner.cache.blocks("a", long_block)]
        needed = min(at["a"] - 4, at["a"] // 40 * 40)  # the next token's window, and the block it belongs to
        assert held == [8 * (p + 1) > needed for p in range(len(held))], (at["a"], held)


def test_a_batch_of_unequal_requests_equals_each_alone(tmp_path):
    """A request's logits beside three others of other lengths, and alone."""
    from akas_b200.engine.batch import StepEntry
    from akas_b200.ops import reference

    config = CONFIGS["mix"]
    folder, _ = make_folder(config, seed=14, folder=tmp_path / "m")
    ps = prompts(config["vocab"], [1, 37, 2, 80], seed=5)
    runner = runner_for(folder, "float32", "cpu", 8, 256, reference)
    together = runner.step([StepEntry(i, p, (len(p) - 1,)) for i, p in enumerate(ps)]).numpy()
    for i, p in enumerate(ps):
        alone = runner_for(folder, "float32", "cpu", 8, 256, reference).step([StepEntry("x", p, (len(p) - 1,))]).numpy()
        assert np.abs(alone[0] - together[i]).max() <= 1e-5 * np.abs(alone).max()


# --------------------------------------------------------------------------- generation


def _greedy(config, w, prompt, count):
    toks = list(prompt)
    for _ in range(count):
        toks.append(int(plain.forward(toks, w, config)[-1].argmax()))
    return toks[len(prompt):]


def generation_case(device, dtype, ops, tmp_path, graphs, pool=1024):
    from akas_b200 import Engine, EngineConfig

    config = CONFIGS["mix"]
    folder, w = make_folder(config, seed=61, folder=tmp_path / "gen")
    ps = prompts(config["vocab"], [1, 9, 40, 23, 3], seed=8)
    cfg = EngineConfig(dtype=dtype, device=device, page_size=8, max_requests=3, context=64, max_tokens=pool, prefill_chunk=13,
                       prefill_requests=2, cuda_graphs=graphs)
    with Engine(str(folder), config=cfg, ops=ops) as engine:
        results = engine.generate(ps, max_tokens=12)
        stats = dict(engine.stats)
    for prompt, result in zip(ps, results):
        assert result["generated_tokens"] == _greedy(config, w, prompt, 12)
    return stats


def test_greedy_generation_through_the_scheduler_on_the_plain_operations(tmp_path):
    from akas_b200.ops import reference

    generation_case("cpu", "float32", reference, tmp_path, False)


def test_greedy_generation_with_a_pool_too_small_for_all(tmp_path):
    """Requests that are put back and started again from their first token: the token in front of it is gone then."""
    from akas_b200.ops import reference

    stats = generation_case("cpu", "float32", reference, tmp_path, False, pool=72)
    assert any("preempt" in k and v for k, v in stats.items()), stats


@pytest.mark.gpu
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler_on_the_kernels(graphs, tmp_path):
    generation_case("cuda:0", "float32", None, tmp_path, graphs)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(dtype, tmp_path):
    """200 decoded tokens for three requests of different lengths through captured graphs, against one whole pass of
    the plain model."""
    from akas_b200 import Engine, EngineConfig, StepEntry

    config = CONFIGS["mix"]
    folder, w = make_folder(config, seed=71, folder=tmp_path / "long")
    ps = prompts(config["vocab"], [5, 70, 33], seed=3)
    feed = prompts(config["vocab"], [200, 200, 200], seed=4)
    cfg = EngineConfig(dtype=dtype, device="cuda:0", page_size=8, max_requests=4, context=512, max_tokens=2048)
    with Engine(str(folder), config=cfg) as engine:
        runner = engine.runner
        runner.step([StepEntry(i, p, ()) for i, p in enumerate(ps)])
        rows = [[] for _ in ps]
        for t in range(200):
            logits = runner.step([StepEntry(i, (feed[i][t],), (0,)) for i in range(3)]).float().cpu().numpy()
            for i in range(3):
                rows[i].append(logits[i])
        assert 4 in runner._graphs
    want = {}
    for i, p in enumerate(ps):
        logits, least = oracle(config, w, p + feed[i])
        want[i] = (logits[len(p):], least[len(p):])
    compare({i: np.stack(r) for i, r in enumerate(rows)}, want, dtype, f"long decoding/{dtype}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(dtype, tmp_path):
    """bin/trace_run as a user calls it, on a Nuzulorn folder: steps on standard input, logits as files."""
    config = CONFIGS["alone"]
    folder, w = make_folder(config, seed=27, folder=tmp_path / "m")
    reqs = {f"q{i}": p for i, p in enumerate(prompts(config["vocab"], [50, 3, 71, 20, 130], seed=7))}
    steps, peak = traces.mixed(reqs, {rid: max(1, len(t) - 5) for rid, t in reqs.items()}, seed=1, live=4, page=64)
    out = tmp_path / "out"
    proc = subprocess.run(
        [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
         "--max-tokens", str(peak)],
        input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    want = {rid: oracle(config, w, t) for rid, t in reqs.items()}
    at = {rid: 0 for rid in reqs}
    for s in steps:
        wanted = sum(len(e["want"]) for e in s["entries"])
        if not wanted:
            continue
        data = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(wanted, config["vocab"])
        row = 0
        for e in s["entries"]:
            for k in e["want"]:
                logits, least = want[e["id"]]
                p = at[e["id"]] + k
                if least[p] >= CLOSE_CALL[dtype]:
                    assert np.abs(data[row] - logits[p]).max() <= TOL[dtype] * np.abs(logits).max(), (s["step"], e["id"], k)
                row += 1
            at[e["id"]] += len(e["tokens"])


# --------------------------------------------------------------------------- the kernels' new options one by one


def _close(got, want, tol, what):
    got, want = got.double().cpu(), want.double().cpu()
    err = float((got - want).abs().max() / max(1e-30, float(want.abs().max())))
    assert err <= tol, f"{what}: {err:.3g}"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("c", [20, 77, 128, 2048])
def test_embedding_of_pairs_kernel(c, dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["elementwise"])
    g = torch.Generator().manual_seed(c)
    table, pairs = torch.randn(300, c, generator=g).to(dtype), torch.randn(38, c, generator=g).to(dtype)
    lens, slots = [1, 60, 2, 1], [3, 0, 5, 1]
    n = sum(lens)
    ids = torch.randint(0, 300, (n + 3,), generator=g).to(torch.int32)
    cu = torch.tensor([0] + list(np.cumsum(lens)) + [n], dtype=torch.int32)
    seq = torch.tensor(sum(([i] * k for i, k in enumerate(lens)), []) + [-1] * 3, dtype=torch.int32)
    slot = torch.tensor(slots + [-1], dtype=torch.int32)
    state = torch.tensor([[17], [0], [0], [250], [9], [0]], dtype=torch.int32)
    results = []
    for ops, device in ((reference, "cpu"), (cuda, "cuda")):
        st = state.clone().to(device)
        args = [t.to(device) for t in (ids, table, pairs)]
        rest = [t.to(device) for t in (cu, seq, slot)]
        out = torch.zeros(4, n + 3, c, device=device)
        both = ops.bigram_embedding(*args, 3000000019, 2000000011, st, *rest, out=out[1:3])
        again = ops.bigram_embedding(*args, 3000000019, 2000000011, state.clone().to(device), *rest)
        assert torch.equal(out[1], out[2]) and torch.equal(both, out[2]) and torch.equal(again, both) and (out[0] == 0).all() and (out[3] == 0).all()
        results.append((both.cpu(), st.cpu()))
    assert torch.equal(results[0][0], results[1][0]) and torch.equal(results[0][1], results[1][1])
    assert results[1][1].flatten().tolist() == [int(ids[60]) + 1, int(ids[63]) + 1, 0, int(ids[0]) + 1, 9, int(ids[62]) + 1]


@pytest.mark.gpu
@pytest.mark.parametrize("n,c,count", [(1, 20, 2), (9, 50, 5), (300, 128, 3), (33, 1024, 17), (17, 2048, 9), (5, 4096, 4), (3, 8192, 6), (20, 8200, 3), (40, 77, 40)])
def test_average_over_results_kernel(n, c, count):
    from akas_b200.ops import cuda, reference

    cuda.require(["elementwise"])
    g = torch.Generator().manual_seed(n * 1000 + c)
    history = (torch.randn(count + 2, n, c, generator=g) * 2).cuda()
    if n % 2:  # entries further apart than their rows are long
        history = torch.stack([history, history], dim=1)[:, 0]
    w, nw = torch.randn(count, generator=g).cuda(), torch.randn(c, generator=g).cuda()
    rows = torch.randint(0, n, (max(1, n // 3),), generator=g).to(torch.int32).cuda()
    for picked in (None, rows):
        for norm in (None, (nw, 1e-3, False, torch.float32), (nw, 1e-3, True, torch.bfloat16)):
            held = history.clone(memory_format=torch.preserve_format) if n % 2 == 0 else torch.stack([history, history], dim=1)[:, 0]
            out = held[count] if picked is None else None
            want, wanted_norm = reference.depth_average(history, count, w, None, rows=picked, norm=norm)
            got, normed = cuda.depth_average(held, count, w, out, rows=picked, norm=norm)
            _close(got, want, 3e-6, "average")
            assert torch.equal(held[:count], history[:count]) and torch.equal(held[count + 1:], history[count + 1:])
            if picked is None:
                assert got.data_ptr() == held[count].data_ptr()
            if normed is not None:
                _close(normed, wanted_norm, 5e-6 if norm[3] == torch.float32 else 8e-3, "norm of the average")
            elif norm is not None:  # sizes the fused kernel leaves alone, or few rows whose product norms them on its way in
                assert c % 4 or c > 8192 or (norm[3] == torch.bfloat16 and want.shape[0] <= 16 and c % 64 == 0)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims,page", [(6, 2, 24, 16, 16, 8), (3, 1, 10, 6, 0, 4), (8, 2, 64, 48, 32, 64), (2, 1, 128, 64, 0, 64)])
def test_query_temperature_kernel(heads, kv_heads, dim, vdim, dims, page, dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["attention_general"])
    g = torch.Generator().manual_seed(dim)
    n, start = 40, 500
    pages = -(-(start + n) // page)
    q, k, v = (torch.randn(n, width, generator=g) for width in (heads * dim, kv_heads * dim, kv_heads * vdim))
    table = torch.randperm(pages, generator=g).to(torch.int32)[None]
    seq, pos = torch.zeros(n, dtype=torch.int32), torch.arange(start, start + n, dtype=torch.int32)
    bias = [torch.randn(width, generator=g) for width in (heads * dim, kv_heads * dim, kv_heads * vdim)]
    tables = {}
    results = []
    for ops, device in ((reference, "cpu"), (cuda, "cuda")):
        if dims:
            freq = torch.tensor([300.0 ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
            tables = dict(zip(("cos", "sin"), (t.to(device) for t in reference.rope_tables(pos, freq))))
        for temperature in (None, (0.5, 1), (0.5, 13), (-0.3, 520)):
            pools = [torch.zeros(pages, kv_heads, page, width, dtype=dtype, device=device) for width in (dim, vdim)]
            out = ops.qk_norm_store(q.to(device), k.to(device), v.to(device), heads, kv_heads, dim, vdim, None, None, 0.0, *pools, table.to(device),
                                    seq.to(device), pos.to(device), page, temperature=temperature,
                                    **dict(zip(("q_bias", "k_bias", "v_bias"), (b.to(device) for b in bias))), **tables)
            results.append((out, *pools))
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    for want, got in zip(results[:4], results[4:]):
        for a, b, what in zip(got, want, ("queries", "keys", "values")):
            _close(a, b, tol, what)
    assert torch.equal(results[4][1], results[6][1])  # the keys have no temperature
    factor = torch.tensor([1.0 + 0.5 * math.log((p + 1) // 13 + 1) for p in pos.tolist()])
    _close(results[6][0].float().cpu(), results[4][0].float().cpu() * factor[:, None], 1e-6 if dtype == torch.float32 else 1.2e-2, "the temperature")


def _paged_case(lens, starts, heads, kv_heads, dim, vdim, page, block, dtype, seed):
    """Pages of several requests in one pool (tables scattered, one request of no tokens between), queries of their next
    tokens, and the blocks' pages."""
    g = torch.Generator().manual_seed(seed)
    width = max(-(-(s + l) // page) for s, l in zip(starts, lens)) + 1
    pages = len(lens) * width
    tables = torch.randperm(pages, generator=g).to(torch.int32).reshape(len(lens), width)
    other = torch.randperm(pages, generator=g).to(torch.int32).reshape(len(lens), width)
    entries = -(-page // block)
    pools = [torch.randn(pages, kv_heads, page, size, generator=g).to(dtype) for size in (dim, vdim)]
    blocks = [torch.zeros(pages, kv_heads, entries, size, dtype=dtype) for size in (dim, vdim)]
    n = sum(lens)
    seq = torch.tensor(sum(([i] * l for i, l in enumerate(lens)), []), dtype=torch.int32)
    pos = torch.tensor(sum((list(range(s, s + l)) for s, l in zip(starts, lens)), []), dtype=torch.int32)
    cu = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    q = torch.randn(n, heads * dim, generator=g).to(dtype)
    every = torch.tensor(sum(([i] * (s + l) for i, (s, l) in enumerate(zip(starts, lens))), []), dtype=torch.int32)
    whole = torch.tensor(sum((list(range(s + l)) for s, l in zip(starts, lens)), []), dtype=torch.int32)
    return q, pools, blocks, tables, other, seq, pos, cu, every, whole


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kv_heads,dim,vdim,page,block", [(2, 24, 16, 8, 8), (1, 20, 28, 16, 7), (4, 16, 24, 8, 20), (2, 8, 8, 16, 1), (2, 64, 48, 64, 16), (1, 10, 6, 4, 3)])
def test_block_means_kernel(kv_heads, dim, vdim, page, block, dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["attention_general"])
    lens, starts = [50, 1, 3, 1], [0, block - 1, 40, 5 * block - 1]
    q, pools, blocks, tables, other, seq, pos, cu, every, whole = _paged_case(lens, starts, kv_heads, kv_heads, dim, vdim, page, block, dtype, dim + block)
    seq = torch.cat([seq, torch.tensor([-1], dtype=torch.int32)])
    pos = torch.cat([pos, torch.tensor([block - 1], dtype=torch.int32)])
    results = []
    for ops, device in ((reference, "cpu"), (cuda, "cuda")):
        made = [b.clone().to(device) for b in blocks]
        ops.pool_blocks(*(p.to(device) for p in pools), *made, *(t.to(device) for t in (tables, other, seq, pos)), page, page, block)
        results.append(made)
    for a, b in zip(results[1], results[0]):
        _close(a, b, 2e-6 if dtype == torch.float32 else 8e-3, "means")
        assert torch.equal((a.cpu() == 0), (b == 0))  # the same entries are written
    # the last request's fifth block by hand
    first, last = 4 * block, 5 * block - 1
    mean = torch.stack([pools[0][tables[3, t // page].long(), :, t % page] for t in range(first, last + 1)]).double().mean(0)
    got = results[1][0][other[3, last // page].long(), :, 4 - last // page * page // block]
    _close(got, mean, 2e-6 if dtype == torch.float32 else 8e-3, "one block")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,page,block,window", [(6, 2, 24, 16, 8, 8, 21), (3, 1, 20, 28, 16, 7, 33), (4, 4, 16, 24, 8, 20, 30),
                                                                     (4, 2, 8, 8, 16, 1, 9), (8, 2, 64, 48, 64, 16, 90), (5, 5, 12, 10, 4, 12, 5),
                                                                     (4, 1, 48, 96, 64, 4, 136), (2, 2, 104, 128, 64, 3, 1), (40, 2, 16, 16, 8, 2, 64)])
def test_attention_over_a_window_and_blocks_kernel(heads, kv_heads, dim, vdim, page, block, window, dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["attention_general"] + (["attention_general_tc"] if dtype == torch.bfloat16 else []))
    lens, starts = [1, 1, 70, 3, 1, 130], [700, window, 200, 0, window + block - 2, 330]
    q, pools, blocks, tables, other, seq, pos, cu, every, whole = _paged_case(lens, starts, heads, kv_heads, dim, vdim, page, block, dtype, dim + block)
    reference.pool_blocks(*pools, *blocks, tables, other, every, whole, page, page, block)
    # one block far in front of the first request's window, and one of its neighbours that is not seen, stand out for every head
    g = torch.Generator().manual_seed(1)
    gate = torch.randn(q.shape[0], heads, generator=g)
    far = 5
    at = far * block + block - 1
    place = other[0, at // page].long(), far - at // page * page // block
    for a in range(kv_heads):
        blocks[0][place[0], a, place[1]] = (q[0].reshape(heads, dim)[a * (heads // kv_heads)] * 3.0).to(dtype)
    results = []
    for ops, device in ((reference, "cpu"), (cuda, "cuda")):
        class Ctx:
            cu_seqlens = cu.to(device)
            query_lens = tuple(lens)
            max_context = 800
            decode_only = False

        for sink, gated in ((False, None), (True, gate.to(device))):
            kb, vb = (b.to(device) for b in blocks)
            results.append(ops.attention_general(q.to(device), *(p.to(device) for p in pools), tables.to(device), seq.to(device), pos.to(device),
                                                 dim ** -0.5, window, 0, None, None, None, sink, gated, page, Ctx, out_scale=0.7,
                                                 blocks=(kb, vb, other.to(device), page, block)))
    for want, got in zip(results[:2], results[2:]):
        _close(got, want, 5e-6 if dtype == torch.float32 else 1.5e-2, "window and blocks")
    # token by token in float64, for the query just behind the edges
    t, r = int(cu[4]), 4
    p = int(pos[t])
    keys = [pools[0][tables[r, j // page].long(), :, j % page].double() for j in range(p + 1) if plain.sees_token(p, j, window)]
    vals = [pools[1][tables[r, j // page].long(), :, j % page].double() for j in range(p + 1) if plain.sees_token(p, j, window)]
    for b in range((p + 1) // block):
        if plain.sees_block(p, b, window, block):
            last = b * block + block - 1
            e = other[r, last // page].long(), b - last // page * page // block
            keys.append(blocks[0][e[0], :, e[1]].double())
            vals.append(blocks[1][e[0], :, e[1]].double())
    k, v = torch.stack(keys), torch.stack(vals)
    qt = q[t].double().reshape(kv_heads, heads // kv_heads, dim)
    s = torch.einsum("kgd,skd->kgs", qt, k) * dim ** -0.5
    direct = torch.einsum("kgs,skv->kgv", torch.softmax(s, -1), v).reshape(-1) * 0.7
    _close(results[2][t], direct, 1e-5 if dtype == torch.float32 else 1.5e-2, "against the equations")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,page,window", [(6, 2, 24, 16, 8, None), (3, 1, 20, 28, 16, 50), (8, 2, 96, 96, 64, None), (5, 5, 10, 6, 4, None),
                                                               (8, 1, 64, 80, 64, 300)])
def test_linear_distance_penalty_kernel(heads, kv_heads, dim, vdim, page, window, dtype):
    """score <- cap tanh(score / cap) - slope * distance with a learned logit in the denominator, in a prompt and decoded."""
    from akas_b200.ops import cuda, reference

    cuda.require(["attention_general"] + (["attention_general_tc"] if dtype == torch.bfloat16 else []))
    lens, starts = [1, 1, 70, 3, 130], [700, 0, 200, 0, 330]
    q, pools, _, tables, _, seq, pos, cu, _, _ = _paged_case(lens, starts, heads, kv_heads, dim, vdim, page, 1, dtype, dim)
    slopes = torch.tensor([plain.slope(a, heads) for a in range(heads)])
    sinks = torch.randn(heads, generator=torch.Generator().manual_seed(3))
    results = []
    for ops, device in ((reference, "cpu"), (cuda, "cuda")):
        class Ctx:
            cu_seqlens = cu.to(device)
            query_lens = tuple(lens)
            max_context = 800
            decode_only = False

        for cap in (None, 3.0):
            results.append(ops.attention_general(q.to(device), *(p.to(device) for p in pools), tables.to(device), seq.to(device), pos.to(device),
                                                 2.0 * dim ** -0.5, window, 0, cap, slopes.to(device), None, False, None, page, Ctx,
                                                 sinks=sinks.to(device)))
    for want, got in zip(results[:2], results[2:]):
        _close(got, want, 5e-6 if dtype == torch.float32 else 1.5e-2, "linear penalty")


@pytest.mark.gpu
@pytest.mark.parametrize("heads,dim,vdim", [(3, 12, 10), (1, 5, 33), (2, 20, 36), (4, 64, 128), (2, 128, 128), (2, 128, 40), (1, 8, 300), (2, 200, 24), (1, 600, 8), (1, 1024, 3)])
def test_forget_gates_that_write_kernel(heads, dim, vdim):
    """Token by token and in chunks against the plain statement: requests of unequal length, gates that are nearly shut,
    nearly open and in between, states carried in and out, a slot that stays untouched."""
    from akas_b200.ops import cuda, reference

    cuda.require(["recurrent"])
    g = torch.Generator().manual_seed(dim)
    lens, slots = [1, 300, 64, 2, 129], [4, 0, 3, 1, 5]
    n = sum(lens)
    wide = torch.randn(n, 2 * heads * dim + heads * vdim + 3, generator=g)
    q, f, v = wide[:, : heads * dim], wide[:, heads * dim : 2 * heads * dim], wide[:, 2 * heads * dim : 2 * heads * dim + heads * vdim]
    f *= 4.0
    bias = torch.randn(heads * dim, generator=g) * 3.0
    bias[:: 5], bias[1 :: 5] = 9.0, -30.0
    lower = torch.rand(heads * dim, generator=g)
    lower[1 :: 3] = 0.0
    lower[2 :: 7] = 0.999
    cu = torch.tensor([0] + list(np.cumsum(lens)) + [n], dtype=torch.int32)
    slot = torch.tensor(slots + [-1], dtype=torch.int32)
    state = torch.randn(6, heads, vdim, dim, generator=g)
    start = state.clone()
    want = reference.hgrn2_scan(q, f, v, bias, lower, state, cu, slot, heads, dim, vdim)
    w = wide.cuda()
    cols = (w[:, : heads * dim], w[:, heads * dim : 2 * heads * dim], w[:, 2 * heads * dim : 2 * heads * dim + heads * vdim])
    for longest in (None, 300):
        st = start.clone().cuda()
        args = (*cols, bias.cuda(), lower.cuda(), st, cu.cuda(), slot.cuda(), heads, dim, vdim)
        peek = cuda.hgrn2_scan(*args, write=False, longest=longest)
        assert torch.equal(st.cpu(), start)
        got = cuda.hgrn2_scan(*args, longest=longest)
        assert torch.equal(peek, got)
        _close(got, want, 1e-5, f"outputs, longest {longest}")
        _close(st, state, 1e-5, f"states, longest {longest}")
        assert torch.equal(st[2].cpu(), start[2])
    # a request in portions of any size ends where it ends in one step
    for cuts in ([300], [130, 1, 2, 167], [64, 64, 172], [200, 100]):
        st, rows, at = start.clone().cuda(), [], 1
        for c in cuts:
            rows.append(cuda.hgrn2_scan(*(x[at : at + c] for x in cols), bias.cuda(), lower.cuda(), st, torch.tensor([0, c], dtype=torch.int32).cuda(),
                                        slot[1:2].cuda(), heads, dim, vdim, longest=c))
            at += c
        _close(torch.cat(rows), want[1:301], 1e-5, f"portions {cuts}")
        _close(st[0], state[0], 1e-5, f"the state behind portions {cuts}")


@pytest.mark.gpu
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,vdim", [(3, 10), (4, 32), (2, 128), (1, 2048), (5, 33), (2, 1100)])
def test_head_norm_without_a_gate_kernel(heads, vdim, out_dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["recurrent"])
    g = torch.Generator().manual_seed(vdim)
    o, w = (torch.randn(21, heads * vdim, generator=g) * 3).cuda(), torch.randn(vdim, generator=g).cuda()
    for scale in (1.0, -0.3):
        want = reference.gated_rmsnorm(o, w, 1e-3, None, heads, vdim, out_dtype, out_scale=scale)
        got = cuda.gated_rmsnorm(o, w, 1e-3, None, heads, vdim, out_dtype, out_scale=scale)
        _close(got, want, 3e-6 if out_dtype == torch.float32 else 8e-3, "norm per head")
    direct = plain.norm(o.double().cpu().reshape(21, heads, vdim), w.double().cpu(), 1e-3).reshape(21, -1) * -0.3
    _close(got, direct, 3e-6 if out_dtype == torch.float32 else 8e-3, "against the equations")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,groups,keep,top,c,f", [(6, 3, 1, 2, 80, 24), (16, 4, 2, 4, 160, 136), (8, 8, 3, 3, 52, 20), (5, 1, 1, 2, 48, 16), (64, 8, 3, 6, 1104, 24),
                                                        (12, 2, 2, 5, 264, 40)])
def test_groups_and_the_experts_into_the_stream_kernel(experts, groups, keep, top, c, f, dtype):
    from akas_b200.ops import cuda, reference

    cuda.require(["moe"] + (["moe_grouped"] if dtype == torch.bfloat16 else []))
    g = torch.Generator().manual_seed(experts * 100 + c)
    n = 75
    h = torch.randn(n, c, generator=g).to(dtype).cuda()
    w_router = (torch.randn(experts, c, generator=g) * (2.0 / c ** 0.5)).cuda()
    for correction in (None, torch.randn(experts, generator=g).cuda() * 0.3, torch.full((experts,), -3.0, device="cuda")):
        for scoring in ("sigmoid", "softmax"):
            for best in (1, 2, 3):
                for renorm in (False, True):
                    options = dict(scoring=scoring, renormalize=renorm, group_best=best, weight_scale=1.6)
                    want = reference.moe_route(h, w_router, correction, groups, keep, top, **options)
                    got = cuda.moe_route(h, w_router, correction, groups, keep, top, **options)
                    same = (got[0] == want[0]).all(dim=1)  # a choice may differ where two scores are within rounding of each other
                    assert same.float().mean() > 0.9, (scoring, best, renorm)
                    _close(got[1][same], want[1][same], 1e-4, "weights")
    r = dict(experts=experts, top=top, groups=dict(count=groups, keep=keep), scale=1.6)
    correction = torch.randn(experts, generator=g) * 0.3
    chosen, weights = plain.route(h.double().cpu(), {"router": w_router.double().cpu(), "correction": correction.double()}, "", r)
    got = cuda.moe_route(h, w_router, correction.cuda(), groups, keep, top, scoring="sigmoid", renormalize=False, group_best=2, weight_scale=1.6)
    same = (got[0].cpu().long() == chosen).all(dim=1)
    assert same.float().mean() > 0.9
    _close(got[1].cpu()[same], weights[same], 1e-4, "the rule itself")
    w_gate_up = (torch.randn(experts, 2 * f, c, generator=g) * c ** -0.5).to(dtype).cuda()
    w_down = (torch.randn(experts, c, f, generator=g) * f ** -0.5).to(dtype).cuda()
    stream = torch.randn(n, c, generator=g).cuda()
    for rows in (n, 5):  # 75 tokens: the grouped product in bfloat16 where it takes the sizes; 5: token by token
        x = stream[:rows].clone()
        out = cuda.moe_experts(h[:rows], w_gate_up, w_down, got[0][:rows].contiguous(), got[1][:rows].contiguous(), update=(x, None, None, None, -0.4))
        assert out is x
        ref = reference.moe_experts(h[:rows], w_gate_up, w_down, got[0][:rows], got[1][:rows])
        _close(out, stream[:rows] - 0.4 * ref, 2e-5 if dtype == torch.float32 else 1.5e-2, "into the stream")
    if dtype == torch.bfloat16:
        assert cuda.moe_grouped_status() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layer_widths_of_a_real_model(dtype, tmp_path):
    """Widths at which every product, the attention and the grouped experts run on their tensor-core kernels (a width of
    1,024, heads of 64 and 128, sixteen experts of 512), a prompt of 700 tokens in one step, in portions beside another
    request, and its last tokens decoded: against the plain model."""
    from akas_b200.engine.batch import StepEntry

    # (only the last layer routes: a choice that falls the other way then moves its own position and no later one)
    config = model(1024, 2048, [layer(attn(16, 4, 64, 64, 200, 16, 0.125, 500000.0, 64), None), layer(hgrn(8, 64, 128), None),
                                layer(capped(8, 2, 128, 128, 0.09, 20.0, 0.3, 128), None), layer(hgrn(8, 128, 128), moe(512, 16, 3, groups=4, keep=2, scale=1.3))],
                   buckets=4099, mul_prev=131, mul_cur=7, mult=0.7, eps=1e-6)
    folder, w = make_folder(config, seed=5, folder=tmp_path / "m", std=0.012)
    toks, other = prompts(config["vocab"], [700, 150], seed=3)
    logits, least = oracle(config, w, toks)
    held = least >= {"float32": 2e-4, "bfloat16": 0.01}[dtype]
    rows = list(range(0, 700, 37)) + list(range(690, 700))
    tol = TOL[dtype]

    def check(got, at, what):
        keep = [i for i, p in enumerate(at) if held[p]]
        assert len(keep) > len(at) // 4
        err = np.abs(got[keep] - logits[np.asarray(at)[keep]]).max() / np.abs(logits).max()
        assert err <= tol, f"{what}: {err:.3g}"

    runner = runner_for(folder, dtype, "cuda:0", 64, 1024, None, max_requests=2, context=768)
    check(runner.step([StepEntry("a", toks, tuple(rows))]).float().cpu().numpy(), rows, "one step")
    runner.release("a")
    at, got, places = 0, [], []
    for k, (count, beside) in enumerate(((300, 100), (2, 0), (130, 50), (258, 0))):
        entries = [StepEntry("a", toks[at:at + count], tuple(range(count)))]
        if beside:
            entries.append(StepEntry("b", other[:beside] if k == 0 else other[100:150], ()))
        got.append(runner.step(entries).float().cpu().numpy())
        places += list(range(at, at + count))
        at += count
    for p in range(at, 700):
        got.append(runner.step([StepEntry("b", (5,), ()), StepEntry("a", toks[p:p + 1], (0,))]).float().cpu().numpy())
        places.append(p)
    check(np.concatenate(got), places, "portions beside another request, then single tokens")
