"""The Sagisun model through the framework's own loader, states, engine and entry points against the plain
statement of its equations.  Each case runs on the CPU (fp32) and, marked ``gpu``, on the kernels in fp32
and bf16."""

import io
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from axlearn_b200.common import prng
from axlearn_b200.common.module import functional
from axlearn_b200.common.safetensors_io import read_safetensors, write_safetensors
from axlearn_b200.experiments.text.gpt import sagisun
from axlearn_b200.inference import trace
from axlearn_b200.inference.decode_engine import ModuleDecodeEngine
from axlearn_b200.inference.model_loader import load_model
from axlearn_b200.ops import gla_ops, window_ops
from tests import sagisun_checkpoints as ckpt
from tests import sagisun_oracle as oracle

PLACES = [
    pytest.param(("cpu", torch.float32), id="cpu"),
    pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
    pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu),
]


def _tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed))


def _error(got, want):
    """Root mean square of the difference over that of the reference's deviation, worst row."""
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt().max() / w.pow(2).mean().sqrt()).item()


def _limit(dtype):
    return 2e-5 if dtype == torch.float32 else 0.12


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(ckpt.CONFIGS.items()):
        tensors = ckpt.random_tensors(cfg, rank=[12, 5, 16, 20, 8][i], seed=i)
        out[name] = (cfg, tensors, ckpt.save(tmp_path_factory.mktemp(name), cfg, tensors))
    return out


def _engine(checkpoint, place, batch, max_len):
    loaded = load_model(checkpoint[2], dtype=place[1], device=place[0])
    return ModuleDecodeEngine(loaded.decoder, loaded.parameters["decoder"], batch=batch, max_len=max_len,
                              dtype=place[1], device=place[0])


def _at(rows, positions):
    return torch.tensor(rows), torch.tensor(positions)


# ------------------------------------------------------------------------------ mechanisms, alone
def test_oracle_mechanisms_by_hand():
    """The plain statements themselves on numbers small enough to check by eye."""
    assert oracle.query_temperature(0, 0.5, 4) == 1.0 and oracle.query_temperature(2, 0.5, 4) == 1.0
    assert math.isclose(oracle.query_temperature(3, 0.5, 4), 1 + 0.5 * math.log(2))
    assert [oracle.distance_slope(h, 2) for h in range(2)] == [2.0 ** -4, 2.0 ** -8]
    assert [oracle.visible(5, j, 3) for j in range(7)] == [False, False, False, True, True, True, False]
    one = torch.ones(2, 1, 1, dtype=torch.float64)
    out, state = oracle.gated_linear_attention(one * 2, one * 3, one * 5, one * 0.5)
    assert out.flatten().tolist() == [30.0, 45.0] and state.item() == 22.5
    assert oracle.layer_order({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [0, 1, 2, 1, 2, 3]


def test_distance_slopes_and_temperature_match_the_oracle():
    for heads in (1, 2, 3, 6, 8, 12):
        got = window_ops.distance_slopes(heads).tolist()
        assert all(math.isclose(a, oracle.distance_slope(h, heads), rel_tol=1e-6) for h, a in enumerate(got))
    pos = torch.arange(40)
    got = window_ops.query_temperature(pos, 0.3, 7)
    want = [oracle.query_temperature(p, 0.3, 7) for p in range(40)]
    assert torch.allclose(got, torch.tensor(want, dtype=torch.float32))


def test_ring_positions():
    got = window_ops.ring_positions(4, torch.tensor([0, 2, 4, 7]))
    assert got.tolist() == [[-1, -1, -1, -1], [0, 1, -2, -1], [0, 1, 2, 3], [4, 5, 6, 3]]


@pytest.mark.parametrize("portion", [1, 2, 5, 40])
def test_window_reference_portions(portion):
    spec = window_ops.WindowSpec(4, 2, 6, 5, 7, scale=0.4, q_temp=(0.5, 4), distance_bias=True)
    cols = window_ops.WindowColumns(q=0, k=24, v=40, g=56)
    proj, t = torch.randn(2, 40, 80, generator=torch.Generator().manual_seed(0)), 40
    cache = {"key": torch.zeros(2, 7, 2, 6), "value": torch.zeros(2, 7, 2, 5)}
    outs = []
    for lo in range(0, t, portion):
        o, cache = window_ops.window_attention(proj[:, lo:lo + portion], spec, cols,
                                               start=torch.full((2,), lo, dtype=torch.int32), cache=cache)
        outs.append(o)
    got = torch.cat(outs, dim=1)[..., :20]
    for r in range(2):
        row = proj[r].double()
        want = oracle.window_attention(row[:, :24].reshape(t, 4, 6), row[:, 24:36].reshape(t, 2, 6),
                                       row[:, 40:50].reshape(t, 2, 5), scale=0.4, window=7, temperature=(0.5, 4))
        want = want.reshape(t, 20) * oracle.sigmoid(row[:, 56:76])
        assert (got[r] - want).abs().max() < 1e-5


@pytest.mark.parametrize("tau,chunk", [(16.0, 16), (0.05, 16), (1.0, 3)])
def test_linear_attention_reference(tau, chunk):
    spec = gla_ops.GlaSpec(heads=2, dim=6, vdim=5, rank=3, tau=tau, q_scale=6 ** -0.5, eps=1e-5)
    cols = gla_ops.GlaColumns(q=0, k=16, v=32, g=48, a1=64)
    g = torch.Generator().manual_seed(1)
    proj, a2, bias = torch.randn(1, 50, 72, generator=g), torch.randn(12, 3, generator=g), torch.randn(12, generator=g)
    norm = torch.rand(5, generator=g) + 0.5
    live = torch.tensor([50])
    got, state = gla_ops.reference_gated_linear_attention(proj, a2, bias, norm, spec, cols, live=live, state=None,
                                                          chunk=chunk)
    row = proj[0].double()
    w = {"a1": torch.eye(3, dtype=torch.float64), "a2": a2.double(), "a2.b": bias.double()}
    alpha = oracle.channel_decay(row[:, 64:67], w, 2, 6, tau)
    o, s = oracle.gated_linear_attention(row[:, :12].reshape(50, 2, 6) * 6 ** -0.5, row[:, 16:28].reshape(50, 2, 6),
                                         row[:, 32:42].reshape(50, 2, 5), alpha)
    want = (oracle.rms(o, 1e-5) * norm.double()).reshape(50, 10) * oracle.silu(row[:, 48:58])
    assert (got[0, :, :10] - want).abs().max() < 1e-4 and (state[0] - s).abs().max() < 1e-4


# ------------------------------------------------------------------------------ whole model
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(ckpt.CONFIGS))
def test_prompt_logits_match_the_oracle(checkpoints, name, place):
    cfg, tensors, _ = checkpoints[name]
    n = 140
    ids = _tokens(n, cfg["vocab"])
    want, _ = oracle.forward(cfg, tensors, ids)
    engine = _engine(checkpoints[name], place, 1, n)
    got = engine.prefill(ids[None], logits_at=_at([0] * n, list(range(n))))
    assert _error(got, want) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_decoding_matches_the_prompt(checkpoints, name, place):
    """First tokens by decoding from one token, then on past every window and ring edge."""
    cfg, tensors, _ = checkpoints[name]
    n = 120
    ids = _tokens(n, cfg["vocab"], seed=2)
    want, _ = oracle.forward(cfg, tensors, ids)
    engine = _engine(checkpoints[name], place, 1, n)
    rows = [engine.prefill(ids[None, :1], logits_at=_at([0], [0]))[0].clone()]
    for i in range(1, n):
        rows.append(engine.step_logits(ids[i:i + 1].to(place[0]))[0].clone())
    assert _error(torch.stack(rows), want) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("portion", [2, 3, 17, 64])
def test_portions_of_a_prompt(checkpoints, portion, place):
    cfg, tensors, _ = checkpoints["mixed"]
    n = 110
    ids = _tokens(n, cfg["vocab"], seed=3)
    want, _ = oracle.forward(cfg, tensors, ids)
    engine = _engine(checkpoints["mixed"], place, 1, n)
    rows = [engine.prefill(ids[None, :portion], logits_at=_at([0] * portion, list(range(portion))))]
    for lo in range(portion, n, portion):
        rows.append(engine.extend(ids[None, lo:lo + portion])[0])
    assert _error(torch.cat(rows), want) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch(checkpoints, name, place):
    """Every row of a ragged batch equals the request alone, through prompt, decoding with rows leaving,
    ragged continuations, and a second batch on the same (dirty) engine."""
    cfg, tensors, _ = checkpoints[name]
    engine = _engine(checkpoints[name], place, 3, 160)
    for seed, lengths in ((5, [1, 70, 33]), (9, [90, 2, 3])):
        ids = [_tokens(160, cfg["vocab"], seed=seed + r) for r in range(3)]
        want = [oracle.forward(cfg, tensors, x)[0] for x in ids]
        seen = list(lengths)
        prompts = torch.zeros(3, max(lengths), dtype=torch.int64)
        for r, n in enumerate(lengths):
            prompts[r, :n] = ids[r][:n]
        last = engine.prefill(prompts, lengths=torch.tensor(lengths), logits_at=_at([0, 1, 2], [n - 1 for n in lengths]))
        for r in range(3):
            assert _error(last[r:r + 1], want[r][lengths[r] - 1:lengths[r]]) < 1.5 * _limit(place[1])
        for step in range(40):
            active = torch.tensor([1, int(step < 20 or step >= 30), int(step != 7)])
            feed = torch.tensor([int(ids[r][seen[r]]) for r in range(3)])
            engine.set_active(active)
            logits = engine.step_logits(feed.to(place[0]))
            for r in range(3):
                if active[r]:
                    seen[r] += 1
                    assert _error(logits[r:r + 1], want[r][seen[r] - 1:seen[r]]) < 1.5 * _limit(place[1]), (step, r)
        assert engine.lengths.tolist() == seen
        live = torch.tensor([3, 0, 7])
        block = torch.zeros(3, 7, dtype=torch.int64)
        for r in range(3):
            block[r, :live[r]] = ids[r][seen[r]:seen[r] + int(live[r])]
        logits = engine.extend(block, live)
        for r in (0, 2):
            n = int(live[r])
            assert _error(logits[r, :n], want[r][seen[r]:seen[r] + n]) < 1.5 * _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("window", [16, 64])
def test_far_key_and_window_edge_in_the_model(tmp_path, place, window):
    """One early token carries a key and a value that stand out: inside the window it moves the logits,
    one position later it does not (the linear branch is silenced by its norm weight)."""
    cfg = ckpt.config(48, 64, [ckpt.layer(ckpt.left(2, 1, 32, 32, window, coef=0.0, scale=1.0), ckpt.right(1, 16, 16),
                                          None)], streams=2, mult=1.0)
    tensors = ckpt.random_tensors(cfg, seed=11)
    tensors["l0.mix.right.out"].zero_()
    tensors["embed"].mul_(0.3)
    tensors["embed"][:, :2] = 0
    tensors["embed"][7, 0] = 4.0        # the marked token
    tensors["embed"][:, 1] = 1.0        # the query side sees a constant
    for k in ("q", "k"):
        tensors[f"l0.mix.left.{k}"].zero_()
    tensors["l0.mix.left.q"][0, 1] = tensors["l0.mix.left.q"][32, 1] = 4.0
    tensors["l0.mix.left.k"][0, 0] = 4.0
    checkpoint = (cfg, tensors, ckpt.save(tmp_path, cfg, tensors))
    n, at = 100, 9
    ids = _tokens(n, 48, seed=1)
    ids[ids == 7] = 8
    other = ids.clone()
    ids[at] = 7
    want = [oracle.forward(cfg, tensors, x)[0] for x in (ids, other)]
    gap = (want[0] - want[1]).pow(2).mean(-1).sqrt() / want[0].std()
    assert gap[at + 1:at + window].min() > 0.2 and gap[at + window:].max() < 1e-6
    engine = _engine(checkpoint, place, 1, n)
    whole = engine.prefill(ids[None], logits_at=_at([0] * n, list(range(n))))
    assert _error(whole, want[0]) < _limit(place[1])
    engine.prefill(ids[None, :at + window - 4])
    rows = [engine.step_logits(ids[i:i + 1].to(place[0]))[0].clone() for i in range(at + window - 4, at + window + 6)]
    assert _error(torch.stack(rows), want[0][at + window - 4:at + window + 6]) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
def test_long_decoding_keeps_the_state(checkpoints, place):
    cfg, tensors, _ = checkpoints["five"]
    n = 420
    ids = _tokens(n, cfg["vocab"], seed=8)
    want, _ = oracle.forward(cfg, tensors, ids)
    engine = _engine(checkpoints["five"], place, 1, n)
    engine.prefill(ids[None, :20])
    rows = [engine.step_logits(ids[i:i + 1].to(place[0]))[0].clone() for i in range(20, n)]
    assert _error(torch.stack(rows), want[20:]) < _limit(place[1])


# ------------------------------------------------------------------------------ entry points
def _greedy(cfg, tensors, prompt, steps):
    ids, margins = list(prompt), []
    for _ in range(steps):
        logits, _ = oracle.forward(cfg, tensors, torch.tensor(ids))
        top = logits[-1].topk(2).values
        margins.append((top[0] - top[1]).item() / logits[-1].std().item())
        ids.append(int(logits[-1].argmax()))
    return ids[len(prompt):], margins


@pytest.mark.parametrize("place", PLACES)
def test_greedy_generation_through_sample_decode(checkpoints, place):
    from axlearn_b200.common import logit_modifiers

    cfg, tensors, path = checkpoints["mixed"]
    loaded = load_model(path, dtype=place[1], device=place[0])
    prompts = [[5, 9, 31, 77, 14], [12, 3], [44, 45, 46, 47, 48, 49, 50, 51, 52]]
    steps, longest = 12, 9
    prefix = torch.zeros(3, longest, dtype=torch.int64)
    for r, p in enumerate(prompts):
        prefix[r, :len(p)] = torch.tensor(p)
    from axlearn_b200.common.decoding import StopOnSubsequence

    with torch.no_grad():
        out, _ = functional(
            loaded.model, prng.PRNGKey(0), loaded.parameters,
            dict(input_batch={"prefix": prefix.to(place[0])}, max_sequence_length=longest + steps + 1,
                 logits_modifier=logit_modifiers.top_k_logits(1), stop_decoding_condition=StopOnSubsequence([[cfg["vocab"] + 5]])),
            method="sample_decode", is_training=False)
    for r, p in enumerate(prompts):
        got = out.sequences[r, 0, len(p) - 1:len(p) - 1 + steps].tolist()
        want, margins = _greedy(cfg, tensors, p, steps)
        for i, (a, b) in enumerate(zip(got, want)):
            if a != b:          # only a near-tie may fall the other way, and ends the comparison
                assert place[1] == torch.bfloat16 and margins[i] < 0.05, (r, i, got, want, margins)
                break


def test_several_decodes_and_beams_carry_the_states(checkpoints):
    cfg, tensors, path = checkpoints["odd"]
    loaded = load_model(path, dtype=torch.float32, device="cpu")
    prefix = torch.tensor([[5, 9, 31], [12, 3, 0]])
    with torch.no_grad():
        beams, _ = functional(loaded.model, prng.PRNGKey(0), loaded.parameters,
                              dict(input_batch={"prefix": prefix}, num_decodes=2, max_sequence_length=8),
                              method="beam_search_decode", is_training=False)
        samples, _ = functional(loaded.model, prng.PRNGKey(0), loaded.parameters,
                                dict(input_batch={"prefix": prefix}, num_decodes=3, max_sequence_length=9),
                                method="sample_decode", is_training=False)
    assert beams.live_sequences.shape[:2] == (2, 2) and samples.sequences.shape[:2] == (2, 3)
    # The score of the best live beam is the sum of its tokens' log-probabilities.
    seq = beams.live_sequences[0, 0].tolist()
    logits, _ = oracle.forward(cfg, tensors, torch.tensor([5] + seq[:-1]))
    lp = torch.log_softmax(logits, -1)
    total = sum(lp[i, t].item() for i, t in enumerate(seq) if i >= 2)
    assert math.isclose(total, beams.live_scores[0, 0].item(), rel_tol=1e-4, abs_tol=1e-3)


def test_generate_command(checkpoints, capsys):
    from axlearn_b200.cli.main import main

    cfg, tensors, path = checkpoints["five"]
    assert main(["generate", "--model", path, "--prompt", "4 8 15", "--prompt", "16,23", "--max_new_tokens", "5",
                 "--dtype", "float32", "--device", "cpu"]) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.strip().splitlines()]
    assert [x["prompt"] for x in lines] == [[4, 8, 15], [16, 23]]
    for line in lines:
        want, _ = _greedy(cfg, tensors, line["prompt"], 5)
        stop = want.index(1) + 1 if 1 in want else 5
        assert line["tokens"][:stop] == want[:stop]


@pytest.mark.parametrize("place", PLACES)
def test_trace_replay(checkpoints, tmp_path, monkeypatch, capsys, place):
    cfg, tensors, path = checkpoints["odd"]
    a, b, c = (_tokens(30, cfg["vocab"], seed=s).tolist() for s in (1, 2, 3))
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:9], "want": [0, 8]}, {"id": "b", "tokens": b[:3], "want": []}]},
        {"step": 1, "entries": [{"id": "b", "tokens": b[3:4], "want": [0]}, {"id": "a", "tokens": a[9:10], "want": [0]}]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[10:11], "want": []}], "end": ["a"]},
        {"step": 3, "entries": [{"id": "b", "tokens": b[4:5], "want": [0]}], "end": ["b"]},
        {"step": 7, "entries": [{"id": "c", "tokens": c[:20], "want": [19, 4]}], "end": []},
        {"step": 8, "entries": [{"id": "c", "tokens": c[20:24], "want": [3]}], "end": ["c"]},
    ]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(map(json.dumps, steps)) + "\n"))
    assert trace.main(["--model", path, "--dtype", "float32" if place[1] == torch.float32 else "bfloat16", "--out",
                       str(tmp_path), "--max-tokens", "64", "--device", place[0]]) == 0
    assert [x for x in capsys.readouterr().out.split("\n") if x] == [f"done {s['step']}" for s in steps]
    full = {n: oracle.forward(cfg, tensors, torch.tensor(x))[0] for n, x in (("a", a), ("b", b), ("c", c))}
    want = {0: [("a", 0), ("a", 8)], 1: [("b", 3), ("a", 9)], 3: [("b", 4)], 7: [("c", 19), ("c", 4)], 8: [("c", 23)]}
    assert sorted(os.listdir(tmp_path)) == sorted(f"{s}.f32" for s in want)
    for step, places in want.items():
        data = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32)
        got = data.reshape(len(places), cfg["vocab"])
        assert _error(got, torch.stack([full[n][p] for n, p in places])) < 1.5 * _limit(place[1])


def test_trace_run_is_a_program():
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = subprocess.run([os.path.join(root, "bin", "trace_run"), "--help"], capture_output=True, text=True, check=True)
    assert "--max-tokens" in out.stdout


# ------------------------------------------------------------------------------ configuration, loading, training
def test_loader_refuses_what_it_does_not_know(tmp_path):
    cfg = ckpt.CONFIGS["five"]
    tensors = ckpt.random_tensors(cfg)
    extra = dict(tensors, **{"l0.mix.left.bias": torch.zeros(3)})
    short = {k: v for k, v in tensors.items() if k != "l1.norm2"}
    with pytest.raises(ValueError, match="no part of the model"):
        load_model(ckpt.save(tmp_path / "extra", cfg, extra))
    with pytest.raises(KeyError, match="l1.norm2"):
        load_model(ckpt.save(tmp_path / "short", cfg, short))
    with pytest.raises(ValueError, match="expected"):
        load_model(ckpt.save(tmp_path / "shape", cfg, dict(tensors, **{"final.norm": torch.zeros(3)})))
    with pytest.raises(ValueError, match="unknown architecture"):
        load_model(ckpt.save(tmp_path / "arch", dict(cfg, architecture="Other"), tensors))
    bad = dict(cfg, layers=[dict(cfg["layers"][0], type="serial")] * 2)
    with pytest.raises(ValueError, match="mixer type"):
        sagisun.model_config(bad)


def test_safetensors_round_trip(tmp_path):
    tensors = {"a": torch.arange(6, dtype=torch.int32).reshape(2, 3), "b": torch.randn(5).bfloat16(),
               "empty": torch.zeros(0, 4), "scalar": torch.tensor(2.5)}
    path = str(tmp_path / "t.safetensors")
    write_safetensors(path, tensors, metadata={"format": "pt"})
    back = read_safetensors(path)
    assert all(back[k].dtype == v.dtype and torch.equal(back[k], v) for k, v in tensors.items())


def test_trains_and_matches_finite_differences():
    """The registered test size takes gradient steps (loss falls), and one gradient agrees with a
    difference quotient."""
    cfg = sagisun.model_config(sagisun.size_config("test", vocab_size=64), gate_rank=4).set(name="m")
    model = cfg.instantiate(parent=None)
    params = model.initialize_parameters_recursively(prng.PRNGKey(0))
    leaves = []

    def walk(node):
        for k, v in node.items():
            if isinstance(v, dict):
                walk(v)
            else:
                node[k] = v.requires_grad_(True)
                leaves.append(node[k])

    walk(params)
    ids = _tokens(2 * 25, 64, seed=4).reshape(2, 25) % 62 + 2
    batch = {"input_ids": ids[:, :-1], "target_labels": ids[:, 1:]}

    def loss():
        (value, _), _ = functional(model, prng.PRNGKey(1), params, dict(input_batch=batch), is_training=True)
        return value

    first = loss()
    first.backward()
    mix = params["decoder"]["transformer"]["layer1"]["mixer_connection"]["mix"]
    grad = mix.grad[0, 1].item()
    with torch.no_grad():
        values = []
        for d in (1e-2, -1e-2):
            mix[0, 1] += d
            values.append(loss().item())
            mix[0, 1] -= d
    assert abs((values[0] - values[1]) / 2e-2 - grad) < 2e-3 + 0.02 * abs(grad)
    assert all(p.grad is not None for p in leaves)
    opt = torch.optim.Adam(leaves, lr=3e-3)
    for _ in range(12):
        opt.zero_grad()
        loss().backward()
        opt.step()
    assert loss().item() < first.item() - 0.3


def test_named_trainer_config():
    from axlearn_b200.experiments.text.gpt import c4_trainer

    cfg = c4_trainer.named_trainer_configs()["sagisun-test"]()
    assert cfg.model.decoder.transformer.num_streams == 2 and cfg.model.decoder.transformer.loop == (1, 2, 2)
