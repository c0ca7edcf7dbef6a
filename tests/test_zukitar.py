"""The Zukitar model through the framework's own loader, states, engine and entry points against the plain
statement of its equations.  Each case runs on the CPU (fp32) and, marked ``gpu``, on the kernels in fp32
and bf16."""

import io
import json
import math
import os
import sys

import pytest
import torch

from axlearn_b200.common import prng
from axlearn_b200.common.module import functional
from axlearn_b200.experiments.text.gpt import zukitar
from axlearn_b200.inference import trace
from axlearn_b200.inference.decode_engine import ModuleDecodeEngine
from axlearn_b200.inference.model_loader import load_model
from axlearn_b200.ops import expert_ops, hyper_ops, latent_ops, ssd_ops
from tests import zukitar_checkpoints as ckpt
from tests import zukitar_oracle as oracle

PLACES = [
    pytest.param(("cpu", torch.float32), id="cpu"),
    pytest.param(("cuda", torch.float32), id="cuda-f32", marks=pytest.mark.gpu),
    pytest.param(("cuda", torch.bfloat16), id="cuda-bf16", marks=pytest.mark.gpu),
]
F64 = torch.float64


def _tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed))


def _want(cfg, tensors, ids):
    return oracle.run(ids, {k: v.double() for k, v in tensors.items()}, cfg)[0]


def _error(got, want):
    """Root mean square of the difference over that of the reference's deviation, worst row."""
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt().max() / w.pow(2).mean().sqrt()).item()


def _limit(dtype):
    return 1e-5 if dtype == torch.float32 else 0.04


@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    out = {}
    for i, (name, cfg) in enumerate(ckpt.CONFIGS.items()):
        tensors = ckpt.random_tensors(cfg, seed=i)
        out[name] = (cfg, tensors, ckpt.save(tmp_path_factory.mktemp(name), cfg, tensors))
    return out


def _engine(checkpoint, place, batch, max_len):
    loaded = load_model(checkpoint[2], dtype=place[1], device=place[0])
    return ModuleDecodeEngine(loaded.decoder, loaded.parameters["decoder"], batch=batch, max_len=max_len,
                              dtype=place[1], device=place[0])


def _at(rows, positions):
    return torch.tensor(rows), torch.tensor(positions)


def _whole(engine, ids):
    return engine.prefill(ids[None], logits_at=_at([0] * len(ids), list(range(len(ids)))))


# ------------------------------------------------------------------------------ mechanisms, alone
def test_oracle_mechanisms_by_hand():
    """The plain statements themselves on numbers small enough to check by eye."""
    x = torch.tensor([1.0, 0.0, 0.0, 2.0, 7.0], dtype=F64)
    got = oracle.rotate_interleaved(x, 3, 4, 100.0)
    want = [math.cos(3), math.sin(3), -2 * math.sin(0.3), 2 * math.cos(0.3), 7.0]
    assert torch.allclose(got, torch.tensor(want, dtype=F64))
    one = torch.ones(2, 1, dtype=F64)
    w = torch.tensor([[2.0, 10.0]], dtype=F64)
    conv = oracle.causal_conv_silu(one, w, torch.zeros(1, dtype=F64)).flatten()
    assert torch.allclose(conv, oracle.silu(torch.tensor([10.0, 12.0], dtype=F64)))
    # Two tokens, dt = log 2 and 1, rate 1: the state halves ... exp(-1) ... and adds dt B x.
    y, s = oracle.ssd_recurrence(one[..., None] * 3, one[..., None] * 5, one[..., None] * 2,
                                 torch.tensor([[math.log(2)], [1.0]], dtype=F64), torch.zeros(1, dtype=F64),
                                 torch.full((1,), 0.5, dtype=F64))
    s1 = math.log(2) * 15
    s2 = math.exp(-1) * s1 + 15
    assert torch.allclose(y.flatten(), torch.tensor([2 * s1 + 1.5, 2 * s2 + 1.5], dtype=F64)) and abs(s.item() - s2) < 1e-12
    # The gate comes ahead of the norm, parts are normed apart.
    n = oracle.gated_group_norm(torch.tensor([[1.0, 3.0]], dtype=F64), torch.tensor([[1.0, 1.0]], dtype=F64),
                                torch.tensor([2.0, 3.0], dtype=F64), 2, 0.0)
    assert torch.allclose(n, torch.tensor([[2.0, 3.0]], dtype=F64))
    eye = torch.eye(1, dtype=F64)
    got = [oracle.clamped_expert(torch.full((1, 1), v, dtype=F64), eye, eye, eye, 2.0).item() for v in (9.0, -9.0)]
    assert math.isclose(got[0], 2 / (1 + math.exp(-3.404)) * 3) and math.isclose(got[1], 9 / (1 + math.exp(9 * 1.702)))
    ids, weight = oracle.route(torch.tensor([[1.0]], dtype=F64), torch.tensor([[0.0], [3.0], [1.0]], dtype=F64), 2)
    assert ids.tolist() == [[1, 2]] and torch.allclose(weight, torch.sigmoid(torch.tensor([[3.0, 1.0]], dtype=F64)))


def test_rotation_matches_the_oracle():
    x = torch.randn(6, 10, generator=torch.Generator().manual_seed(0))
    got = latent_ops.rotate_interleaved(x, torch.arange(6) * 1000, 8, 300.0)
    for p in range(6):
        want = oracle.rotate_interleaved(x[p].double(), 1000 * p, 8, 300.0)
        assert (got[p] - want).abs().max() < 1e-5


@pytest.mark.parametrize("portion", [1, 2, 5, 40])
def test_latent_reference_portions(portion):
    mixer = ckpt.latent(3, 6, 4, 5, 7, base=50.0, scale=0.4)["mixer"]
    spec = latent_ops.LatentSpec(3, 6, 4, 5, 7, 4, 50.0, 0.4, 1e-5)
    cols, t, g = latent_ops.LatentColumns(q=0, c=32, r=40), 40, torch.Generator().manual_seed(0)
    proj = torch.randn(2, t, 44, generator=g)
    norm, uk, uv = torch.rand(7, generator=g) + 0.5, torch.randn(18, 7, generator=g), torch.randn(15, 7, generator=g)
    cache, outs = {"latent": torch.zeros(2, t, spec.row_width)}, []
    uk_stored = torch.nn.functional.pad(uk.t(), (0, 6, 0, 1))
    uv_stored = torch.nn.functional.pad(uv, (0, 1, 0, 9))
    for lo in range(0, t, portion):
        o, cache = latent_ops.latent_attention(proj[:, lo:lo + portion], norm, uk_stored, uv_stored, spec, cols,
                                               start=torch.full((2,), lo, dtype=torch.int32), cache=cache)
        outs.append(o)
    got = torch.cat(outs, dim=1)
    assert got.shape[-1] == 16 and got[..., 15:].abs().max() == 0
    eye = torch.eye(44, dtype=F64)
    for r in range(2):
        w = {"q": eye[:30], "dkv": eye[torch.tensor(list(range(32, 39)) + list(range(40, 44)))], "dkv.norm": norm.double(),
             "uk": uk.double(), "uv": uv.double(), "o": torch.eye(15, dtype=F64)}
        want = oracle.latent_attention(proj[r].double(), w, mixer, 1e-5)
        assert (got[r, :, :15] - want).abs().max() < 1e-5


@pytest.mark.parametrize("portion", [1, 2, 3, 50])
@pytest.mark.parametrize("taps", [1, 2, 4])
def test_ssd_reference_portions(portion, taps):
    mixer = ckpt.mamba(6, 5, 7, 3, taps, 2)["mixer"]
    spec = ssd_ops.SsdSpec(6, 5, 7, 3, taps, 2, 1e-5)
    t, g = 50, torch.Generator().manual_seed(1)
    proj = torch.randn(1, t, 120, generator=g)
    cols = ssd_ops.SsdColumns(z=0, xbc=32, dt=104)
    conv, bias = torch.randn(72, taps, generator=g), torch.randn(72, generator=g)
    vec = {k: torch.randn(6, generator=g) for k in ("dt_bias", "A_log", "D")}
    norm = torch.rand(30, generator=g) + 0.5
    weights = ssd_ops.SsdWeights(conv.t(), bias, vec["dt_bias"], vec["A_log"], vec["D"], norm)
    state = {"ssm": torch.zeros(1, 6, 7, 5), "conv": torch.zeros(1, taps, 72)}
    outs = []
    for lo in range(0, t, portion):
        o, state = ssd_ops.ssd_mix(proj[:, lo:lo + portion], weights, spec, cols, state=state,
                                   start=torch.full((1,), lo, dtype=torch.int32))
        outs.append(o)
    eye = torch.eye(120, dtype=F64)
    rows = torch.cat([eye[:30], eye[32:104], eye[104:110]])
    w = {"in": rows, "conv": conv.double(), "conv.b": bias.double(), "norm": norm.double(), "o": torch.eye(30, dtype=F64)}
    w.update({k: v.double() for k, v in vec.items()})
    want = oracle.mamba2(proj[0].double(), w, mixer, 1e-5)
    assert (torch.cat(outs, dim=1)[0, :, :30] - want).abs().max() < 2e-4


@pytest.mark.parametrize("experts,top,limit", [(5, 1, 0.5), (6, 3, 1.5), (3, 3, 8.0), (1, 1, 1.0)])
def test_expert_reference(experts, top, limit):
    g = torch.Generator().manual_seed(experts)
    h, f, d = torch.randn(9, 12, generator=g), 10, 12
    w = {f"e{e}.{n}": torch.randn(*s, generator=g) for e in range(experts)
         for n, s in (("gate", (f, d)), ("up", (f, d)), ("down", (d, f)))}
    w["router"] = torch.randn(experts, d, generator=g)
    gate_up, down = torch.zeros(experts, 128, 64), torch.zeros(experts, 64, 64)
    for e in range(experts):
        gate_up[e, :f, :d], gate_up[e, 64:64 + f, :d], down[e, :d, :f] = w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]
    got = expert_ops.expert_feed_forward(h, h @ w["router"].T, gate_up, down, top=top, width=d, hidden=f,
                                         gate=hyper_ops.Gate("clamped", limit=limit))
    want = oracle.mixture(h.double(), {k: v.double() for k, v in w.items()},
                          {"router": {"top": top}, "expert": {"limit": limit}})
    assert got.shape == (9, 16) and (got[:, :d] - want).abs().max() < 1e-4


def test_gates_match_the_oracle():
    x = torch.linspace(-6, 6, 97)
    u = torch.linspace(3, -3, 97)
    got = hyper_ops.gate_values(x, u, hyper_ops.Gate("gelu_tanh"))
    assert (got - oracle.gelu_tanh(x.double()) * u).abs().max() < 1e-5


# ------------------------------------------------------------------------------ whole model
@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", list(ckpt.CONFIGS))
def test_prompt_logits_match_the_oracle(checkpoints, name, place):
    cfg, tensors, _ = checkpoints[name]
    ids = _tokens(150, cfg["vocab"])
    engine = _engine(checkpoints[name], place, 1, 150)
    assert _error(_whole(engine, ids), _want(cfg, tensors, ids)) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("length", [1, 2, 3, 15, 16, 17, 63, 64, 65, 127, 128, 129])
def test_prompt_lengths_around_tiles_and_chunks(checkpoints, length, place):
    """Prompts that end just inside, on and just outside a chunk or tile, and the tokens decoded after them."""
    cfg, tensors, _ = checkpoints["wide" if length > 64 else "mixed"]
    ids = _tokens(length + 3, cfg["vocab"], seed=length)
    want = _want(cfg, tensors, ids)
    engine = _engine(checkpoints["wide" if length > 64 else "mixed"], place, 1, length + 3)
    rows = [_whole(engine, ids[:length])]
    rows += [engine.step_logits(ids[i:i + 1].to(place[0])).clone() for i in range(length, length + 3)]
    assert _error(torch.cat(rows), want) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["mixed", "odd", "ones", "wide"])
def test_decoding_matches_the_prompt(checkpoints, name, place):
    """Everything after the first token is decoded."""
    cfg, tensors, _ = checkpoints[name]
    n = 90
    ids = _tokens(n, cfg["vocab"], seed=2)
    engine = _engine(checkpoints[name], place, 1, n)
    rows = [engine.prefill(ids[None, :1], logits_at=_at([0], [0]))[0].clone()]
    for i in range(1, n):
        rows.append(engine.step_logits(ids[i:i + 1].to(place[0]))[0].clone())
    assert _error(torch.stack(rows), _want(cfg, tensors, ids)) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("portion", [2, 3, 17, 64])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_portions_of_a_prompt(checkpoints, portion, place, name):
    cfg, tensors, _ = checkpoints[name]
    n = 110
    ids = _tokens(n, cfg["vocab"], seed=3)
    engine = _engine(checkpoints[name], place, 1, n)
    rows = [_whole(engine, ids[:portion])]
    for lo in range(portion, n, portion):
        rows.append(engine.extend(ids[None, lo:lo + portion])[0])
    assert _error(torch.cat(rows), _want(cfg, tensors, ids)) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_unequal_requests_in_one_batch(checkpoints, name, place):
    """Every row of a ragged batch equals the request alone, through prompt, decoding with rows leaving,
    ragged continuations, and a second batch on the same (dirty) engine."""
    cfg, tensors, _ = checkpoints[name]
    engine = _engine(checkpoints[name], place, 3, 160)
    for seed, lengths in ((5, [1, 70, 33]), (9, [90, 2, 3])):
        ids = [_tokens(160, cfg["vocab"], seed=seed + r) for r in range(3)]
        want = [_want(cfg, tensors, x) for x in ids]
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
@pytest.mark.parametrize("at", [0, 1, 63, 64])
def test_a_far_key_is_seen(tmp_path, place, at):
    """One early token carries a key that stands out among hundreds: it moves every later logit, through
    whole prompts and through the cache of a decoding step."""
    cfg = ckpt.config(48, 64, [(ckpt.latent(2, 16, 8, 32, 32, scale=1.0), None)], logit_scale=1.0)
    tensors = ckpt.random_tensors(cfg, seed=11)
    tensors["embed"].mul_(0.3)
    tensors["embed"][:, :2] = 0
    tensors["embed"][7, 0] = 4.0        # the marked token
    tensors["embed"][:, 1] = 1.0        # the query side sees a constant
    for k in ("q", "uk"):
        tensors[f"l0.mix.{k}"].zero_()
    tensors["l0.mix.dkv"][0] = 0
    tensors["l0.mix.dkv"][0, 0] = 8.0   # latent column 0 holds the mark
    tensors["l0.mix.q"][0, 1] = tensors["l0.mix.q"][24, 1] = 3.0
    tensors["l0.mix.uk"][0, 0] = tensors["l0.mix.uk"][16, 0] = 2.0
    checkpoint = (cfg, tensors, ckpt.save(tmp_path, cfg, tensors))
    n = 400
    ids = _tokens(n, 48, seed=1)
    ids[ids == 7] = 8
    other = ids.clone()
    ids[at] = 7
    want = [_want(cfg, tensors, x) for x in (ids, other)]
    gap = (want[0] - want[1]).pow(2).mean(-1).sqrt() / want[0].std()
    assert gap[at + 1:].min() > 0.2
    engine = _engine(checkpoint, place, 1, n)
    assert _error(_whole(engine, ids), want[0]) < _limit(place[1])
    engine.prefill(ids[None, :n - 70])
    rows = [engine.step_logits(ids[i:i + 1].to(place[0]))[0].clone() for i in range(n - 70, n)]
    assert _error(torch.stack(rows), want[0][n - 70:]) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
@pytest.mark.parametrize("at", [0, 62, 63, 64, 65, 300])
def test_a_far_input_stays_in_the_state(tmp_path, place, at):
    """One token writes much into a slow state (its step size stands out): it moves every later logit across
    chunks, and across the seam between prompt and decoding."""
    cfg = ckpt.config(48, 64, [(ckpt.mamba(4, 16, 16, 2, 4, 1), None)], logit_scale=1.0)
    tensors = ckpt.random_tensors(cfg, seed=13)
    tensors["embed"].mul_(0.3)
    tensors["embed"][:, 0] = 0
    tensors["embed"][7, 0] = 4.0
    inner, gn = 64, 32
    rows = slice(2 * inner + 2 * gn, None)
    tensors["l0.mix.in"][rows] = 0
    tensors["l0.mix.in"][rows, 0] = 2.0
    tensors["l0.mix.dt_bias"].fill_(-6.0)
    tensors["l0.mix.A_log"].fill_(-5.0)
    tensors["l0.mix.conv.b"][inner + gn:] = 2.0     # C hardly changes: what was written is read all along
    tensors["l0.mix.D"].mul_(0.1)
    checkpoint = (cfg, tensors, ckpt.save(tmp_path, cfg, tensors))
    n = 400
    ids = _tokens(n, 48, seed=1)
    ids[ids == 7] = 8
    other = ids.clone()
    ids[at] = 7
    want = [_want(cfg, tensors, x) for x in (ids, other)]
    gap = (want[0] - want[1]).pow(2).mean(-1).sqrt() / want[0].std()
    assert gap[at + 4:].median() > 0.3 and gap[at + 4:].min() > 0.03
    engine = _engine(checkpoint, place, 1, n)
    assert _error(_whole(engine, ids), want[0]) < _limit(place[1])
    engine.prefill(ids[None, :n - 70])
    rows = [engine.step_logits(ids[i:i + 1].to(place[0]))[0].clone() for i in range(n - 70, n)]
    assert _error(torch.stack(rows), want[0][n - 70:]) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
def test_strong_and_weak_decays(tmp_path, place):
    """Decays from exp(-60) a token to none at all in one layer: nothing overflows, nothing is lost."""
    cfg = ckpt.config(48, 64, [(ckpt.mamba(6, 16, 32, 2, 3, 2), None)], logit_scale=1.0)
    tensors = ckpt.random_tensors(cfg, seed=14)
    tensors["l0.mix.A_log"].copy_(torch.tensor([4.0, 2.0, 0.0, -3.0, -9.0, 3.0]))
    tensors["l0.mix.dt_bias"].copy_(torch.tensor([0.5, 1.0, -2.0, 0.0, 0.0, -5.0]))
    checkpoint = (cfg, tensors, ckpt.save(tmp_path, cfg, tensors))
    ids = _tokens(200, 48, seed=3)
    engine = _engine(checkpoint, place, 1, 200)
    assert _error(_whole(engine, ids), _want(cfg, tensors, ids)) < _limit(place[1])


@pytest.mark.parametrize("place", PLACES)
def test_long_decoding_keeps_the_state(checkpoints, place):
    cfg, tensors, _ = checkpoints["small"]
    n = 420
    ids = _tokens(n, cfg["vocab"], seed=8)
    want = _want(cfg, tensors, ids)
    engine = _engine(checkpoints["small"], place, 1, n)
    engine.prefill(ids[None, :20])
    rows = [engine.step_logits(ids[i:i + 1].to(place[0]))[0].clone() for i in range(20, n)]
    assert _error(torch.stack(rows), want[20:]) < _limit(place[1])


# ------------------------------------------------------------------------------ entry points
def _greedy(cfg, tensors, prompt, steps):
    ids, margins = list(prompt), []
    for _ in range(steps):
        logits = _want(cfg, tensors, torch.tensor(ids))
        top = logits[-1].topk(2).values
        margins.append((top[0] - top[1]).item() / logits[-1].std().item())
        ids.append(int(logits[-1].argmax()))
    return ids[len(prompt):], margins


@pytest.mark.parametrize("place", PLACES)
def test_greedy_generation_through_sample_decode(checkpoints, place):
    from axlearn_b200.common import logit_modifiers
    from axlearn_b200.common.decoding import StopOnSubsequence

    cfg, tensors, path = checkpoints["mixed"]
    loaded = load_model(path, dtype=place[1], device=place[0])
    prompts = [[5, 9, 31, 77, 14], [12, 3], [44, 45, 46, 47, 48, 49, 50, 51, 52]]
    steps, longest = 12, 9
    prefix = torch.zeros(3, longest, dtype=torch.int64)
    for r, p in enumerate(prompts):
        prefix[r, :len(p)] = torch.tensor(p)
    with torch.no_grad():
        out, _ = functional(
            loaded.model, prng.PRNGKey(0), loaded.parameters,
            dict(input_batch={"prefix": prefix.to(place[0])}, max_sequence_length=longest + steps + 1,
                 logits_modifier=logit_modifiers.top_k_logits(1),
                 stop_decoding_condition=StopOnSubsequence([[cfg["vocab"] + 5]])),
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
    seq = beams.live_sequences[0, 0].tolist()
    lp = torch.log_softmax(_want(cfg, tensors, torch.tensor([5] + seq[:-1])), -1)
    total = sum(lp[i, t].item() for i, t in enumerate(seq) if i >= 2)
    assert math.isclose(total, beams.live_scores[0, 0].item(), rel_tol=1e-4, abs_tol=1e-3)


def test_generate_command(checkpoints, capsys):
    from axlearn_b200.cli.main import main

    cfg, tensors, path = checkpoints["small"]
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
    full = {n: _want(cfg, tensors, torch.tensor(x)) for n, x in (("a", a), ("b", b), ("c", c))}
    want = {0: [("a", 0), ("a", 8)], 1: [("b", 3), ("a", 9)], 3: [("b", 4)], 7: [("c", 19), ("c", 4)], 8: [("c", 23)]}
    assert sorted(os.listdir(tmp_path)) == sorted(f"{s}.f32" for s in want)
    for step, places in want.items():
        data = torch.frombuffer(bytearray((tmp_path / f"{step}.f32").read_bytes()), dtype=torch.float32)
        got = data.reshape(len(places), cfg["vocab"])
        assert _error(got, torch.stack([full[n][p] for n, p in places])) < 1.5 * _limit(place[1])


# ------------------------------------------------------------------------------ configuration, loading, training
def test_loader_refuses_what_it_does_not_know(tmp_path):
    cfg = ckpt.CONFIGS["small"]
    tensors = ckpt.random_tensors(cfg)
    with pytest.raises(ValueError, match="no part of the model"):
        load_model(ckpt.save(tmp_path / "extra", cfg, dict(tensors, **{"l0.mix.q": torch.zeros(3)})))
    with pytest.raises(KeyError, match="l1.norm2"):
        load_model(ckpt.save(tmp_path / "short", cfg, {k: v for k, v in tensors.items() if k != "l1.norm2"}))
    with pytest.raises(ValueError, match="expected"):
        load_model(ckpt.save(tmp_path / "shape", cfg, dict(tensors, **{"l1.mix.dkv": torch.zeros(40, 32)})))
    with pytest.raises(ValueError, match="mixer type"):
        zukitar.model_config(dict(cfg, layers=[dict(cfg["layers"][0], type="other")] * 2))
    with pytest.raises(ValueError, match="feed-forward kind"):
        zukitar.model_config(dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "other"})] * 2))


def test_declared_kernels_are_enough():
    """Every entry point that the model's operations bind is in the sources it declares for a first build."""
    import inspect
    import re

    from axlearn_b200.csrc import build
    from axlearn_b200.ops import cuda_ops, moe_ops, skinny_ops

    used = set()
    for where in (latent_ops, ssd_ops, expert_ops, skinny_ops, hyper_ops, moe_ops._grouped_argtypes, moe_ops._gmm_kernel,
                  cuda_ops.gemm):
        used |= {x for x in re.findall(r"axb_[a-z0-9_]+", inspect.getsource(where)) if not x.startswith("axb_grouped")}
    defined = set()
    for path in build.sources(only=zukitar.KERNEL_SOURCES):
        with open(path, encoding="utf-8") as f:
            defined |= set(re.findall(r'extern "C" [a-z ]+ (axb_\w+)\(', f.read()))
    assert used and not used - defined, used - defined
    # ... and binding the grouped product needs no other library part.
    assert "cuda_ops.lib()" in inspect.getsource(moe_ops._grouped_argtypes)


def test_residual_connection_is_the_plain_residual():
    g = torch.Generator().manual_seed(0)
    x, y, w = torch.randn(2, 3, 20, generator=g), torch.randn(2, 3, 24, generator=g), torch.rand(20, generator=g)
    streams, h = hyper_ops.hyper_step(x, y, write=hyper_ops.PLAIN_WRITE, read=None, norm_scale=w, eps=1e-5,
                                      norm_offset=0.0, num_streams=1, dtype=torch.float32, h_multiplier=3.0)
    want = x + y[..., :20]
    assert torch.allclose(streams[:, :, 0], want)
    assert torch.allclose(h[..., :20], 3 * oracle.rms_norm(want, w, 1e-5), atol=1e-5) and h[..., 20:].abs().max() == 0


def test_trains():
    """The registered test size takes gradient steps: every parameter has a gradient, the loss falls."""
    model = zukitar.model_config(zukitar.size_config("test", vocab_size=64)).set(name="m").instantiate(parent=None)
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
    assert all(p.grad is not None for p in leaves)
    opt = torch.optim.Adam(leaves, lr=3e-3)
    for _ in range(12):
        opt.zero_grad()
        loss().backward()
        opt.step()
    assert loss().item() < first.item() - 0.3


def test_named_trainer_config():
    from axlearn_b200.experiments.text.gpt import c4_trainer

    cfg = c4_trainer.named_trainer_configs()["zukitar-test"]()
    assert cfg.model.decoder.transformer.num_streams == 1 and len(cfg.model.decoder.transformer.layer) == 3
