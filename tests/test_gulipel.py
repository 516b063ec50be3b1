"""The Gulipel decoder through the engine against the plain implementation (tests/plain/gulipel.py).

Without a GPU the engine runs on the stand-in kernels (tests/emulated_ops.py), which checks the
configuration, the model description, the caches and states (the embedding's own among them), and the step
function's cutting and batching; on a B200 the same traces run on the CUDA kernels in 32-bit and in bfloat16, together
with tests that aim at single mechanisms."""
import copy
import math
import os

import numpy as np
import pytest
import torch

from leone_b200.engine.engine import Engine
from leone_b200.registry import config_from_dict, config_from_folder, spec_from_config
from tests import replay
from tests.gulipel_tiny import (PAGE_TOKENS, TINY, as_bf16, left, mamba, model, parallel, right, tiny_config,
                                tiny_tensors)
from tests.plain import gulipel as plain

FP32 = dict(rtol=4e-5, atol_scale=4e-5)
# bfloat16: the gained weights make scores, decays and gates sharp, which also amplifies rounding; the
# 32-bit runs are the sharp tests, these catch a wrong path or operand
BF16 = dict(rtol=8e-2, atol_scale=8e-2)
LENGTHS = [40, 7, 75, 33, 1, 64, 50]


def _bf16_round(t):
    return t.to(torch.bfloat16).to(t.dtype)


def _plain(which, tensors, bf16=False, raw=None):
    """In bfloat16 the plain model has the same stored weights and rounds what the cache holds, what the norms give
    the sublayers, and a recurrence's projections."""
    r = _bf16_round if bf16 else None
    return plain.PlainGulipel(raw or TINY[which], as_bf16(tensors) if bf16 else tensors, cache_round=r, read_round=r, act_round=r)


def _engine(which, tensors, dtype, device, ops=None, max_tokens=512, page=None, raw=None, **kw):
    spec = spec_from_config(config_from_dict(raw) if raw is not None else tiny_config(which))
    return Engine(spec, dict(tensors), dtype=dtype, device=device, ops=ops, page_tokens=page or PAGE_TOKENS[which],
                  max_tokens=max_tokens, max_requests=kw.pop("max_requests", 4),
                  max_batch_tokens=kw.pop("max_batch_tokens", 128), **kw)


def _requests(vocab, lengths=LENGTHS, seed=100):
    return {f"r{i}": replay.random_tokens(vocab, n, seed + i) for i, n in enumerate(lengths)}


def _traces(reqs):
    return {"whole": replay.trace_whole(reqs), "tail": replay.trace_decode_tail(reqs, tail=20),
            "portions": replay.trace_portions(reqs), "mixed": replay.trace_mixed(reqs, seed=3)}


def _run(steps, eng, oracle, reqs, what, dtype="float32"):
    out = replay.run_trace_engine(eng, steps)
    if dtype == "float32":
        return replay.compare(steps, out, oracle, reqs, what=what, **FP32)
    # (a single position whose sums nearly cancel magnifies the rounding: a few rows may pass the bound, by no more
    # than three times)
    return replay.compare(steps, out, oracle, reqs, what=what, rows_over=0.02, **BF16)


# -- configuration and description (CPU) ---------------------------------------------------------
def test_config_round_trip_and_spec():
    for which, raw in TINY.items():
        cfg = config_from_dict(raw)
        assert cfg.to_json_dict() == raw
        spec = spec_from_config(cfg)
        assert all(ls.block == "sandwich_norm" for ls in spec.layers) and spec.lm_head_name == "head"
        assert [ls.prefix for ls in spec.layers] == [f"l{i}" for i in range(len(raw["layers"]))]
        assert [ls.feed_forward is None for ls in spec.layers] == [e["mlp"] is None for e in raw["layers"]]
        assert [ls.mixer.kind for ls in spec.layers] == \
            ["side_by_side" if e["type"].startswith("parallel") else "mamba2" for e in raw["layers"]]
    raw = copy.deepcopy(TINY["A"])
    for entry in raw["layers"]:
        entry["type"] = {"mamba2": "mamba2_11"}.get(entry["type"], entry["type"])
    assert spec_from_config(config_from_dict(raw)) == spec_from_config(tiny_config("A"))      # the number is a name only


def test_config_rejections():
    from leone_b200.config.base import ConfigError
    for patch in (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4),
                  lambda c: c["layers"][1]["mixer"]["right"].update(kv_heads=3),
                  lambda c: c["layers"][1]["mixer"]["left"]["q_temp"].update(every=0),
                  lambda c: c["layers"][1]["mixer"]["left"].pop("scale"),
                  lambda c: c["layers"][1]["mixer"].pop("right"),
                  lambda c: c["layers"][0]["mixer"].update(groups=3),
                  lambda c: c["layers"][0]["mixer"].update(norm_groups=3),
                  lambda c: c["layers"][0]["mixer"].update(conv=0),
                  lambda c: c["layers"][0]["mixer"].update(conv=17),
                  lambda c: c["layers"][0]["mixer"].pop("state"),
                  lambda c: c["layers"][0].update(type="mamba3"),
                  lambda c: c["layers"][0].update(type="mamba2_x"),
                  lambda c: c["layers"][0]["mlp"].update(kind="moe"),
                  lambda c: c["embedding"]["bigram"].update(buckets=0),
                  lambda c: c["embedding"]["bigram"].pop("mul_prev"),
                  lambda c: c["embedding"]["bigram"].update(mul_cur=-1),
                  lambda c: c["token_side"].update(dim=0),
                  lambda c: c.update(logit_softcap=-1.0),
                  lambda c: c.pop("width"), lambda c: c.update(layers=[])):
        raw = copy.deepcopy(TINY["A"])
        patch(raw)
        with pytest.raises(ConfigError):
            config_from_dict(raw)


def test_sizes_come_from_the_checkpoint(tmp_path):
    """The inner widths of decay and gate, and the number of positions where the file does not say it, are the
    tensors' shapes, layer by layer."""
    from leone_b200.weights.safetensors import write_safetensors
    from tests.emulated_ops import EmulatedOps
    raw = copy.deepcopy(TINY["B"])
    for entry in raw["layers"]:
        for key in ("decay_rank", "gate_rank"):
            entry["mixer"].get("right", {}).pop(key, None)
    folder = str(tmp_path)
    del raw["max_positions"]
    import json
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump(raw, fh)
    write_safetensors(os.path.join(folder, "model.safetensors"), tiny_tensors("B"))
    cfg = config_from_folder(folder)
    assert [(m.mixer.right.decay_rank, m.mixer.right.gate_rank) for m in cfg.layers if m.type.startswith("parallel")] == [(3, 2), (9, 1)]
    assert cfg.max_positions == 512
    eng = Engine.from_folder(folder, dtype="float32", device="cpu", ops=EmulatedOps(), page_tokens=8, max_tokens=64,
                             max_requests=1, max_batch_tokens=32)
    toks = replay.random_tokens(101, 9, 1)
    got = eng.step([("r", toks, [8])])[0]
    want = _plain("B", tiny_tensors("B")).logits(toks)[8]
    assert float((got.double() - want).abs().max()) <= 3e-5 * float(want.abs().max())


# -- the plain implementation's own mechanisms, against their definitions (CPU) -----------------------
def test_plain_pair_rows_and_positions():
    big = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert plain.bigram_rows([4, 5, 0], big) == [10, (12 + 35) % 10, 15 % 10]
    W = {"embed": torch.eye(6).double(), "bigram": torch.arange(11.0)[:, None].double().expand(11, 6) * 100,
         "pos": torch.arange(8.0)[:, None].double().expand(8, 6) * 1000}
    x = plain.embed([4, 5, 0], W, {"embedding": {"scale": 2.0, "bigram": big}})
    assert x[:, 1].tolist() == [1000.0, 1700.0, 2500.0] and [x[0, 4].item(), x[1, 5].item(), x[2, 0].item()] == [1002.0, 1702.0, 2502.0]
    assert plain.embed([4, 5], W, {})[1].tolist() == [1000.0] * 5 + [1001.0]


def test_plain_query_temperature():
    t = plain.query_temperature(8, {"coef": 0.5, "every": 3}, torch.float64)
    steps = [0, 0, 1, 1, 1, 2, 2, 2]
    assert torch.allclose(t, torch.tensor([1 + 0.5 * math.log(s + 1) for s in steps], dtype=torch.float64), atol=1e-15)


def test_plain_ssd_by_hand():
    """Two state rows, a decay of a half at the second token, a step of 3 at the third."""
    x = torch.tensor([[[4.0]], [[1.0]], [[10.0]]]).double()
    B = torch.tensor([[[1.0, 0.0]], [[0.0, 2.0]], [[1.0, 1.0]]]).double()
    C = torch.tensor([[[1.0, 1.0]], [[1.0, 0.0]], [[0.0, 1.0]]]).double()
    dt = torch.tensor([[1.0], [1.0], [3.0]]).double()
    y, S = plain.ssd_recurrence(x, B, C, dt, torch.tensor([math.log(2.0)]).double())
    assert torch.allclose(y[:, 0, 0], torch.tensor([4.0, 2.0, 2.0 / 8 + 30.0]).double())
    assert torch.allclose(S[0, :, 0], torch.tensor([2.0 / 8 + 30.0, 2.0 / 8 + 30.0]).double())


def test_plain_delta_rule_by_hand():
    """The channel that decays forgets before the correction is formed; a full beta replaces what a key held."""
    q = torch.tensor([[[1.0, 1.0]]] * 3).double()
    k = torch.tensor([[[1.0, 0.0]], [[0.0, 1.0]], [[1.0, 0.0]]]).double()
    v = torch.tensor([[[8.0]], [[3.0]], [[5.0]]]).double()
    g = torch.tensor([[[0.5, 1.0]]] * 3).double()
    o, S = plain.delta_recurrence(q, k, v, g, torch.tensor([[1.0], [1.0], [0.5]]).double())
    # third token: the first row holds 8 / 4 = 2, u = (5 - 2) / 2
    assert o[:, 0, 0].tolist() == [8.0, 4.0 + 3.0, 3.5 + 3.0] and S[0, :, 0].tolist() == [3.5, 3.0]
    W = {"a1": torch.zeros(2, 3).double(), "a2": torch.zeros(4, 2).double(), "A_log": torch.tensor([0.0, math.log(2.0)]).double(),
         "dt_bias": torch.tensor([0.0, 40.0, -60.0, 0.0]).double()}
    a = plain.channel_decay(torch.ones(1, 3).double(), W, 2, 2)[0]
    assert torch.allclose(a, torch.tensor([[0.5, math.exp(-40.0)], [1.0, 0.25]]).double())


def test_plain_conv_norms_and_gates():
    x = torch.tensor([[1.0], [2.0], [5.0]]).double()
    assert plain.short_conv(x, torch.tensor([[10.0, 1.0]]).double(), torch.tensor([0.5]).double())[:, 0].tolist() == [1.5, 12.5, 25.5]
    r = plain.grouped_rms(torch.tensor([[3.0, 4.0, 0.0, 2.0]]).double(), 2, 0.0)[0]
    assert torch.allclose(r, torch.tensor([3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 0.0, math.sqrt(2.0)]).double())
    z = torch.tensor([0.7], dtype=torch.float64)
    assert abs(float(plain.gelu_tanh(z)) - 0.35 * (1 + math.tanh(math.sqrt(2 / math.pi) * (0.7 + 0.044715 * 0.343)))) < 1e-15


# -- the step function on stand-in kernels (CPU) ------------------------------------------------
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
@pytest.mark.parametrize("mode", ["whole", "portions", "mixed"])
def test_replay_on_stand_in_kernels(which, mode):
    from tests.emulated_ops import EmulatedOps
    tensors = tiny_tensors(which)
    reqs = _requests(TINY[which]["vocab"], [23, 7, 30, 1, 12], seed=300)
    steps = _traces(reqs)[mode]
    eng = _engine(which, tensors, "float32", "cpu", EmulatedOps(), max_tokens=replay.max_live_tokens(steps))
    _run(steps, eng, _plain(which, tensors), reqs, f"{which} {mode} stand-in")
    assert all(f == eng.num_pages for f in eng.cache.free_pages())


def _streams(which, tensors, eng, toks):
    seen = []
    for block in eng.model.blocks:
        inner = block.forward

        def hooked(ctx, cache, hidden, inner=inner, **kw):
            r = inner(ctx, cache, hidden, **kw)
            seen.append(hidden.cpu().clone())
            return r
        block.forward = hooked
    eng.step([("r", toks, [])])
    want = _plain(which, tensors).residuals(toks)
    assert len(seen) == len(want)
    for i, got in enumerate(seen):
        assert float((got.double() - want[i]).abs().max()) <= 3e-5 * float(want[i].abs().max()), i


@pytest.mark.parametrize("which", ["A", "B"])
def test_residual_stream_after_every_layer_on_stand_in_kernels(which):
    """The stream after each layer, read from the engine's buffer by a hook on the blocks."""
    from tests.emulated_ops import EmulatedOps
    tensors = tiny_tensors(which)
    _streams(which, tensors, _engine(which, tensors, "float32", "cpu", EmulatedOps()), replay.random_tokens(97, 19, 4))


def test_caches_and_states():
    from tests.emulated_ops import EmulatedOps
    eng = _engine("A", tiny_tensors("A"), "float32", "cpu", EmulatedOps())
    assert [(g.spec.num_kv_heads, g.spec.head_dim, g.spec.value_head_dim) for g in eng.cache.groups] == [(2, 16, 24)]
    shapes = sorted(tuple(t.shape[1:]) for t in eng._run_state.values())
    # Mamba-2: state and convolution; the delta rule: both; the embedding: the last token
    assert shapes == sorted([(4, 12, 16), (3, 112), (4, 12, 20), (2, 128), (6, 20, 8), (1, 168), (4, 12, 16), (3, 112), (1,)])
    names = [s.name for s in eng.model.weight_specs()]
    assert len(names) == len(set(names)) and {"bigram", "pos", "side.embed", "head", "l1.mix.left.q.b", "l1.mix.right.q.conv",
                                              "l2.mix.conv.b", "l0.mlp.down.b", "l3.ls1", "l0.ls2"} <= set(names)
    assert "l3.ls2" not in names and "l3.norm2b" not in names


# -- on the GPU ----------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", ["whole", "tail", "portions", "mixed"])
def test_replay_on_the_gpu(which, dtype, mode):
    tensors = tiny_tensors(which)
    reqs = _requests(TINY[which]["vocab"])
    steps = _traces(reqs)[mode]
    eng = _engine(which, tensors, dtype, "cuda:0", max_tokens=replay.max_live_tokens(steps))
    _run(steps, eng, _plain(which, tensors, dtype == "bfloat16"), reqs, f"{which}/{dtype}/{mode}", dtype)
    if mode == "mixed":
        blocks = sum(-(-len(t) // eng.page_tokens) for t in reqs.values())
        assert blocks > eng.num_pages and len(reqs) > eng.max_requests, "pages and slots must be used again"
    assert all(f == eng.num_pages for f in eng.cache.free_pages())


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_residual_stream_after_every_layer_on_the_gpu(which):
    tensors = tiny_tensors(which)
    _streams(which, tensors, _engine(which, tensors, "float32", "cuda:0"), replay.random_tokens(TINY[which]["vocab"], 61, 4))


@pytest.mark.gpu
@pytest.mark.parametrize("switch", ["LEONE_NO_SSD_MMA", "LEONE_NO_DELTA_MMA", "LEONE_NO_TENSOR_CORES", "LEONE_NO_MASKED_MMA"])
@pytest.mark.parametrize("which", ["C", "D"])
def test_bfloat16_kernel_switches(which, switch, monkeypatch):
    """With a bfloat16 kernel's switch thrown its any-size form runs, and the same traces still agree
    with the plain implementation (prompt portions of 100 tokens and decode)."""
    monkeypatch.setenv(switch, "1")
    tensors = tiny_tensors(which)
    reqs = _requests(TINY[which]["vocab"], [130, 40, 75])
    steps = replay.trace_portions(reqs, sizes=(100, 2, 1, 1, 30))
    eng = _engine(which, tensors, "bfloat16", "cuda:0", max_tokens=replay.max_live_tokens(steps), max_batch_tokens=128)
    _run(steps, eng, _plain(which, tensors, True), reqs, f"{which} with {switch}", "bfloat16")


@pytest.mark.gpu
@pytest.mark.parametrize("which,index", [(w, i) for w in TINY for i in range(len(TINY[w]["layers"]))])
def test_each_layer_alone(which, index):
    """A model of one layer: its mixer and feed-forward with nothing else to hide behind, in portions down to
    one token."""
    raw = copy.deepcopy(TINY[which])
    raw["layers"] = [raw["layers"][index]]
    tensors = {k.replace(f"l{index}.", "l0."): v for k, v in tiny_tensors(which).items()
               if not k.startswith("l") or k.startswith(f"l{index}.")}
    if "token_side" in raw:
        dim = raw["token_side"]["dim"]
        tensors["side.embed"] = tensors["side.embed"][:, index * dim:(index + 1) * dim].contiguous()
    reqs = _requests(raw["vocab"], [45, 2, 19])
    steps = replay.trace_portions(reqs, sizes=(2, 7, 1, 2, 13))
    eng = _engine(which, tensors, "float32", "cuda:0", raw=raw, max_tokens=192, max_requests=2, max_batch_tokens=64)
    _run(steps, eng, plain.PlainGulipel(raw, tensors), reqs, f"{which} layer {index}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompt_and_long_decode(dtype):
    """A prompt of many pages and chunks, then 150 single-token steps; position 0 alone first."""
    tensors = tiny_tensors("C")
    reqs = {"one": replay.random_tokens(256, 1, 5), "long": replay.random_tokens(256, 460, 77)}
    steps = replay.trace_decode_tail(reqs, tail=150)
    eng = _engine("C", tensors, dtype, "cuda:0", max_tokens=512, max_batch_tokens=512)
    _run(steps, eng, _plain("C", tensors, dtype == "bfloat16"), reqs, f"long {dtype}", dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_beside_decoded_tokens(dtype):
    """Steps in which one request's portion is cut into chunks while others bring one token or a few, in both
    orders; the portions end inside a chunk and inside a group of 16 tokens."""
    tensors = tiny_tensors("C")
    reqs = _requests(256, [333, 40, 301, 12], seed=9)
    at, steps = {r: 0 for r in reqs}, []
    for sizes in ({"r1": 20}, {"r1": 1, "r0": 187}, {"r0": 1, "r1": 1, "r2": 150}, {"r2": 131, "r3": 3, "r1": 2}, {"r0": 130, "r3": 1},
                  {"r0": 15, "r1": 16, "r2": 20, "r3": 8}):
        entries = []
        for rid, n in sizes.items():
            toks = reqs[rid][at[rid]:at[rid] + n]
            entries.append({"id": rid, "tokens": toks, "want": list(range(len(toks)))})
            at[rid] += len(toks)
        steps.append({"step": len(steps), "entries": entries, "end": []})
    assert at == {r: len(t) for r, t in reqs.items()}
    eng = _engine("C", tensors, dtype, "cuda:0", max_tokens=832, max_batch_tokens=512)
    _run(steps, eng, _plain("C", tensors, dtype == "bfloat16"), reqs, f"long portions {dtype}", dtype)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,tol", [("float32", 2e-5), ("bfloat16", 6e-2)])
def test_unequal_requests_together_and_alone(dtype, tol):
    """Four requests of unequal lengths in one step give what each gives alone."""
    tensors = tiny_tensors("C")
    reqs = _requests(256, [90, 3, 41, 17], seed=50)
    eng = _engine("C", tensors, dtype, "cuda:0", max_tokens=512, max_batch_tokens=256)
    together = eng.step([(r, t, list(range(len(t)))) for r, t in reqs.items()]).cpu()
    at = 0
    for r, t in reqs.items():
        eng.close(r)
        alone = eng.step([(r + "alone", t, list(range(len(t))))]).cpu()
        eng.close(r + "alone")
        assert float((alone - together[at:at + len(t)]).abs().max()) <= tol * float(alone.abs().max()), r
        at += len(t)


@pytest.mark.gpu
def test_page_size_does_not_change_fp32_logits():
    """Pages of another size hold the same rows, so the logits are equal to the bit."""
    tensors = tiny_tensors("A")
    reqs = _requests(97, [50, 21, 64])
    steps = replay.trace_mixed(reqs, seed=5)
    outs = []
    for pt in (4, 16, 64):
        eng = _engine("A", tensors, "float32", "cuda:0", max_tokens=replay.max_live_tokens(steps), page=pt)
        outs.append(replay.run_trace_engine(eng, steps))
    for k in outs[0]:
        assert np.array_equal(outs[0][k], outs[1][k]) and np.array_equal(outs[0][k], outs[2][k])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_slot_used_again_starts_from_nothing(dtype):
    """One state slot: the second request gets the slot (recurrent and convolution states, the last token) and the pages
    the first one left, and must read none of it."""
    tensors = tiny_tensors("C")
    reqs = _requests(256, [37, 29, 61], seed=35)
    steps = replay.trace_portions(reqs, sizes=(1, 1, 2, 9, 40))
    eng = _engine("C", tensors, dtype, "cuda:0", max_tokens=64, max_requests=1)
    _run(steps, eng, _plain("C", tensors, dtype == "bfloat16"), reqs, "slot used again", dtype)


def _stand_out_model(kind):
    """A one-layer model in which token 7, and no other, writes something that token 9, and no other, reads.
    ``attention``: a key dimension that only token 7 fills and a query dimension that only token 9 fills, with scores far
    above all others; the delta rule beside it gives nothing.  ``delta``: the same through the recurrence's keys and
    queries, with a decay that forgets next to nothing in that channel; the attention gives nothing.  ``mamba2``:
    through a row of the state that only token 7 writes and only token 9 reads."""
    if kind == "mamba2":
        raw = model(64, 32, 1e-6, [mamba(2, 12, 8, 1, 2, 3)], positions=400)
    else:
        raw = model(64, 32, 1e-6, [parallel(left(2, 1, 8, 12, 0.7), right(2, 1, 8, 12, 3, 4, 4))], positions=400)
    t = tiny_tensors(None, seed=3, raw=raw)
    t["pos"][:] = 0.0
    t["embed"][:, :2] = 0.0
    for tok, coord in ((7, 0), (9, 1)):
        t["embed"][tok] = 0.0
        t["embed"][tok, coord] = 1.0
    t["l0.norm1"][:] = 1.0
    if kind == "attention":
        t["l0.mix.right.o"][:] = 0.0
        for name in ("q", "k"):
            t[f"l0.mix.left.{name}"][:, :2] = 0.0
            t[f"l0.mix.left.{name}"][4] = 0.0
            t[f"l0.mix.left.{name}.b"][4] = 0.0
        t["l0.mix.left.k"][4, 0] = t["l0.mix.left.q"][4, 1] = 3.0
    elif kind == "delta":
        t["l0.mix.left.o"][:] = 0.0
        for name in ("q", "k"):
            t[f"l0.mix.right.{name}"][:, :2] = 0.0
            t[f"l0.mix.right.{name}"][3] = 0.0
            t[f"l0.mix.right.{name}.conv"][3] = torch.tensor([0.0, 0.0, 1.0])
        t["l0.mix.right.k"][3, 0] = t["l0.mix.right.q"][3, 1] = 3.0
        t["l0.mix.right.a2"].view(2, 8, 4)[:, 3] = 0.0
        t["l0.mix.right.dt_bias"].view(2, 8)[:, 3] = -20.0
    else:
        # rows of the input product: z 24, x 24, B 8, C 8, dt 2; B and C are channels 24..40 of the convolution
        t["l0.mix.in"][48 + 3] = 0.0
        t["l0.mix.in"][48 + 3, 0] = 3.0
        t["l0.mix.in"][56:64] = 0.0
        t["l0.mix.in"][56 + 3, 1] = 3.0
        t["l0.mix.conv"][[27, 35]] = torch.tensor([0.0, 0.0, 1.0])
        t["l0.mix.conv.b"][27] = 0.0
        t["l0.mix.conv.b"][32:40] = 0.0
        t["l0.mix.A_log"][:] = -14.0
    return raw, t


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,bound", [("float32", 3e-5), ("bfloat16", 4e-2)])
@pytest.mark.parametrize("kind,q_pos,k_pos", [
    ("attention", 330, 0), ("attention", 200, 17), ("attention", 48, 47), ("attention", 64, 15), ("attention", 33, 16),
    ("attention", 65, 64), ("delta", 300, 2), ("delta", 40, 39), ("delta", 65, 0), ("delta", 17, 16), ("delta", 32, 31),
    ("mamba2", 300, 2), ("mamba2", 40, 39), ("mamba2", 65, 0), ("mamba2", 17, 16), ("mamba2", 64, 63), ("mamba2", 192, 127),
    ("mamba2", 192, 128), ("mamba2", 340, 63), ("mamba2", 340, 64)])
def test_a_far_write_is_read(kind, q_pos, k_pos, dtype, bound):
    """What one token wrote hundreds of tokens back (a key at a page's border; a write into a recurrent state at the
    border of a group of 16 tokens or of a chunk) is what another reads, in a prompt, in portions, and through
    decoding."""
    raw, tensors = _stand_out_model(kind)
    base = [t if t not in (7, 9) else 8 for t in replay.random_tokens(64, q_pos + 4, 9)]
    base[q_pos] = 9
    marked = list(base)
    marked[k_pos] = 7
    oracle = _plain(None, tensors, dtype == "bfloat16", raw=raw)
    delta = float((oracle.logits(marked)[q_pos] - oracle.logits(base)[q_pos]).abs().max())
    eng = _engine(None, tensors, dtype, "cuda:0", raw=raw, page=16, max_tokens=704, max_requests=2, max_batch_tokens=352)
    for name, toks in (("marked", marked), ("base", base)):
        want = oracle.logits(toks)[q_pos]
        limit = bound * float(want.abs().max())
        assert delta > 3 * limit, ("the test's own premise", delta, limit)
        whole = eng.step([(name, toks, [q_pos])])[0].cpu()
        eng.close(name)
        assert float((whole.double() - want).abs().max()) <= limit, (name, "prompt")
        for cut in {max(1, q_pos - 2), min(k_pos + 1, q_pos), max(1, q_pos - 20)}:
            eng.step([(name, toks[:cut], [])])
            last = None
            for p in range(cut, q_pos + 1):
                last = eng.step([(name, [toks[p]], [0])])[0].cpu()
            eng.close(name)
            if last is not None:
                assert float((last.double() - want).abs().max()) <= limit, (name, "decoded from", cut)


def test_stand_out_models_hold_their_premise():
    """The marked token changes the reader's logits by far more than any bound above (CPU)."""
    for kind in ("attention", "delta", "mamba2"):
        raw, tensors = _stand_out_model(kind)
        base = [t if t not in (7, 9) else 8 for t in replay.random_tokens(64, 330, 9)]
        base[325] = 9
        marked = list(base)
        marked[2] = 7
        oracle = _plain(None, tensors, raw=raw)
        a, b = oracle.logits(marked)[325], oracle.logits(base)[325]
        assert float((a - b).abs().max()) > 0.15 * float(a.abs().max()), kind


def _step_ctx(q_lens, ctx_lens, slots, dev="cuda:0"):
    """What the kernels read of a step: ``q_lens[s]`` new tokens of sequence ``s`` that end at ``ctx_lens[s]``."""
    from types import SimpleNamespace
    starts = [0]
    for x in q_lens:
        starts.append(starts[-1] + x)
    seqs = [s for s, x in enumerate(q_lens) for _ in range(x)]
    pos = [c - x + i for x, c in zip(q_lens, ctx_lens) for i in range(x)]
    return SimpleNamespace(n_seqs=len(q_lens), n_tokens=int(sum(q_lens)), q_lens=np.asarray(q_lens),
                           q_start=torch.tensor(starts, dtype=torch.int32, device=dev),
                           slot_ids=torch.tensor(slots, dtype=torch.int32, device=dev),
                           seq_of_token=torch.tensor(seqs, dtype=torch.int32, device=dev),
                           positions=torch.tensor(pos, dtype=torch.int32, device=dev), max_q_len=max(q_lens),
                           max_ctx_len=max(ctx_lens), decode_only=max(q_lens) == 1,
                           status=torch.zeros(4, dtype=torch.int32, device=dev)), starts


@pytest.mark.gpu
@pytest.mark.parametrize("heads,groups,n_state,vdim,strong", [
    (3, 1, 12, 20, 0.0), (1, 1, 5, 7, 0.0), (4, 4, 16, 16, 0.0), (4, 2, 64, 64, 0.0), (6, 3, 128, 64, 0.0), (2, 1, 128, 128, 0.0),
    (2, 2, 160, 24, 0.0), (1, 1, 300, 40, 0.0), (2, 1, 48, 48, 0.0), (2, 2, 32, 200, 0.0), (4, 1, 96, 80, 0.0), (2, 1, 256, 64, 0.0),
    # steps and decays so strong that a few tokens together leave nothing, or a single one
    (2, 1, 64, 64, 3.0), (2, 2, 128, 64, 6.0), (3, 1, 16, 24, 30.0)])
def test_ssd_kernels_against_the_plain_recurrence(heads, groups, n_state, vdim, strong, monkeypatch):
    """The recurrence's kernels alone in every form (the walk's register forms, tensor cores, chunks side by side): three
    sequences in steps of unequal sizes with the state carried in slots that are not in order."""
    from leone_b200.ops.cuda import CudaOps
    g = torch.Generator().manual_seed(n_state + vdim)
    lengths, slots = [277, 3, 85], [2, 0, 3]
    inner, bc = heads * vdim, groups * n_state
    acts = [torch.randn(n, inner + 2 * bc, generator=g).to(torch.bfloat16) for n in lengths]
    raws = [torch.randn(n, heads + 3, generator=g).to(torch.bfloat16) for n in lengths]
    a_log, dt_bias, skip = torch.randn(heads, generator=g) * 0.5 - 1, torch.randn(heads, generator=g) + strong, torch.randn(heads, generator=g)
    cuts = [[200, 1, 1, 2, 73], [1, 2], [2, 1, 82]]
    want, states = [], []
    for s, n in enumerate(lengths):
        a = acts[s].double()
        x = a[:, :inner].view(n, heads, vdim)
        B = a[:, inner:inner + bc].view(n, groups, n_state).repeat_interleave(heads // groups, dim=1)
        C = a[:, inner + bc:].view(n, groups, n_state).repeat_interleave(heads // groups, dim=1)
        y, S = plain.ssd_recurrence(x, B, C, plain.softplus(raws[s][:, 3:].double() + dt_bias.double()), torch.exp(a_log.double()))
        want.append((y + skip.double()[None, :, None] * x).reshape(n, inner))
        states.append(S)
    for dtype, switch, chunk, tol in ((torch.float32, "0", 0, 3e-5), (torch.bfloat16, "1", 0, 3e-5), (torch.bfloat16, "0", 0, 1e-4),
                                      (torch.bfloat16, "0", 64, 1e-4), (torch.bfloat16, "0", 128, 1e-4)):
        monkeypatch.setenv("LEONE_NO_SSD_MMA", switch)
        ops = CudaOps("cuda:0", dtype)
        state = torch.randn(4, heads, n_state, vdim, generator=g).cuda()       # what a slot held before must not matter
        state[slots] = 0.0
        done = [0, 0, 0]
        got = [torch.zeros(n, inner, dtype=torch.float64) for n in lengths]
        for step in range(5):
            live = [s for s in range(3) if step < len(cuts[s])]
            q_lens = [cuts[s][step] for s in live]
            ctx, starts = _step_ctx(q_lens, [done[s] + cuts[s][step] for s in live], [slots[s] for s in live])
            act = torch.cat([acts[s][done[s]:done[s] + cuts[s][step]] for s in live]).to(dtype).cuda()
            raw = torch.cat([raws[s][done[s]:done[s] + cuts[s][step]] for s in live]).to(dtype).cuda()
            out = torch.zeros(sum(q_lens), inner, device="cuda:0")
            ops.ssd(ctx, act, raw, out, state, a_log.cuda(), dt_bias.cuda(), skip.cuda(), heads, groups, n_state, vdim,
                    x_off=0, b_off=inner, c_off=inner + bc, dt_off=3, chunk=chunk if max(q_lens) > chunk else 0)
            assert int(ctx.status[0]) == 0
            for j, s in enumerate(live):
                got[s][done[s]:done[s] + cuts[s][step]] = out[starts[j]:starts[j + 1]].cpu().double()
                done[s] += cuts[s][step]
        for s in range(3):
            err = float((got[s] - want[s]).abs().max()) / float(want[s].abs().max())
            assert err <= tol, (dtype, switch, chunk, s, err)
            serr = float((state[slots[s]].cpu().double() - states[s]).abs().max()) / float(states[s].abs().max())
            assert serr <= tol, (dtype, switch, chunk, s, "state", serr)


@pytest.mark.gpu
@pytest.mark.parametrize("per_channel", [True, False])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,strong", [
    (4, 2, 12, 20, 0.0), (1, 1, 36, 12, 0.0), (6, 3, 10, 14, 0.0), (2, 1, 64, 64, 0.0), (2, 2, 128, 128, 0.0), (3, 1, 144, 24, 0.0),
    (1, 1, 300, 40, 0.0), (8, 2, 32, 33, 0.0), (1, 1, 512, 64, 0.0), (2, 1, 100, 72, 0.0), (1, 1, 65, 1, 0.0),
    # decays so strong that sixteen of them together leave nothing (and single ones that leave next to nothing), or none
    (2, 1, 64, 64, 4.0), (2, 2, 128, 40, 30.0), (3, 1, 48, 32, -12.0)])
def test_delta_rule_kernels_against_the_plain_recurrence(heads, kv_heads, dim, vdim, strong, per_channel, monkeypatch):
    """The recurrence's kernels alone in every form (the walk's register forms, tensor cores), with a decay per key channel
    and with one per head: three sequences in steps of unequal sizes with the state carried in slots that are not in
    order."""
    from leone_b200.ops.cuda import CudaOps
    g = torch.Generator().manual_seed(dim + vdim)
    lengths, slots = [277, 3, 85], [2, 0, 3]
    qk, hv = kv_heads * dim, heads * vdim
    acts = [torch.randn(n, 2 * qk + hv, generator=g) for n in lengths]
    for a in acts:
        # every key is like the one before it, so that the corrections matter
        for t in range(1, len(a)):
            a[t, qk:2 * qk] = 0.7 * a[t - 1, qk:2 * qk] + 0.5 * a[t, qk:2 * qk]
    raws = [(torch.randn(n, 2 * heads + 3, generator=g) * 2).to(torch.bfloat16) for n in lengths]
    zs = [torch.randn(n, heads * dim + 5, generator=g) * 2 - 1 + strong for n in lengths]
    a_log, dt_bias = torch.randn(heads, generator=g) * 0.5, torch.randn(heads, generator=g) - 2 + strong
    cuts = [[200, 1, 1, 2, 73], [1, 2], [2, 1, 82]]
    rep = heads // kv_heads
    want, states = [], []
    for s, n in enumerate(lengths):
        a, r = acts[s].double(), raws[s].double()
        q = (plain.unit(a[:, :qk].view(n, kv_heads, dim)) * dim ** -0.5).repeat_interleave(rep, dim=1)
        k = plain.unit(a[:, qk:2 * qk].view(n, kv_heads, dim)).repeat_interleave(rep, dim=1)
        z = zs[s][:, :heads * dim].double().view(n, heads, dim) if per_channel else (r[:, 3:3 + heads] + dt_bias.double())[:, :, None].expand(n, heads, dim)
        decay = torch.exp(-torch.exp(a_log.double())[None, :, None] * plain.softplus(z))
        o, S = plain.delta_recurrence(q, k, a[:, 2 * qk:].view(n, heads, vdim), decay, torch.sigmoid(r[:, 3 + heads:]))
        want.append(o.reshape(n, hv))
        states.append(S)
    for dtype, raw_dtype, switch, tol in ((torch.float32, torch.float32, "0", 3e-5), (torch.bfloat16, torch.bfloat16, "1", 3e-5),
                                          (torch.bfloat16, torch.bfloat16, "0", 1e-4), (torch.bfloat16, torch.float32, "0", 1e-4)):
        monkeypatch.setenv("LEONE_NO_DELTA_MMA", switch)
        ops = CudaOps("cuda:0", dtype)
        state = torch.randn(4, heads, dim, vdim, generator=g).cuda()        # what a slot held before must not matter
        state[slots] = 0.0
        done, got = [0, 0, 0], [torch.zeros(n, hv, dtype=torch.float64) for n in lengths]
        for step in range(5):
            live = [s for s in range(3) if step < len(cuts[s])]
            q_lens = [cuts[s][step] for s in live]
            ctx, starts = _step_ctx(q_lens, [done[s] + cuts[s][step] for s in live], [slots[s] for s in live])
            act, raw, z = (torch.cat([src[s][done[s]:done[s] + cuts[s][step]] for s in live]).cuda() for src in (acts, raws, zs))
            out = torch.zeros(sum(q_lens), hv, device="cuda:0")
            kw = {"channel_logits": z[:, :heads * dim]} if per_channel else {}
            ops.gated_delta(ctx, act, raw.to(raw_dtype), out, state, a_log.cuda(), None if per_channel else dt_bias.cuda(), heads,
                            kv_heads, dim, vdim, 0, qk, 2 * qk, 3, 3 + heads, dim ** -0.5, **kw)
            assert int(ctx.status[0]) == 0
            for j, s in enumerate(live):
                got[s][done[s]:done[s] + cuts[s][step]] = out[starts[j]:starts[j + 1]].cpu().double()
                done[s] += cuts[s][step]
        for s in range(3):
            err = float((got[s] - want[s]).abs().max()) / float(want[s].abs().max())
            assert err <= tol, (dtype, switch, s, err)
            serr = float((state[slots[s]].cpu().double() - states[s]).abs().max()) / float(states[s].abs().max())
            assert serr <= tol, (dtype, switch, s, "state", serr)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_embedding_kernel_against_its_definition(dtype):
    """Pair rows across steps (the previous token comes from the slot), at a sequence's first token, with large
    multipliers; position rows; a slot that held another sequence's token."""
    from leone_b200.ops.cuda import CudaOps
    ops = CudaOps("cuda:0", dtype)
    g = torch.Generator().manual_seed(2)
    for width, buckets, a, b in ((20, 7, 3, 5), (1030, 1, 4, 9), (256, 65521, 2_000_003, 1_000_000_007)):
        table, pairs, places = (torch.randn(rows, width, generator=g).to(dtype) for rows in (5000, buckets + 1, 40))
        toks = [[int(x) for x in torch.randint(0, 5000, (n,), generator=g)] for n in (25, 3, 9)]
        cuts, slots = [[12, 1, 1, 2, 9], [1, 2], [7, 1, 1]], [2, 0, 3]
        for use_pairs, use_places in ((True, True), (False, True), (True, False)):
            words = torch.full((4, 1), 1234567, dtype=torch.int32, device="cuda:0")
            done = [0, 0, 0]
            for step in range(5):
                live = [s for s in range(3) if step < len(cuts[s])]
                q_lens = [cuts[s][step] for s in live]
                ctx, starts = _step_ctx(q_lens, [done[s] + cuts[s][step] for s in live], [slots[s] for s in live])
                ctx.token_ids = torch.tensor(sum((toks[s][done[s]:done[s] + cuts[s][step]] for s in live), []), dtype=torch.int32, device="cuda:0")
                out = torch.zeros(sum(q_lens), width, device="cuda:0")
                ops.embedding_sum(ctx, table.cuda(), out, scale=1.7, pairs=pairs.cuda() if use_pairs else None, buckets=buckets,
                                  mul_prev=a, mul_cur=b, last_token=words, places=places.cuda() if use_places else None)
                assert int(ctx.status[0]) == 0
                for j, s in enumerate(live):
                    rows = plain.bigram_rows(toks[s], {"buckets": buckets, "mul_prev": a, "mul_cur": b})
                    for i in range(cuts[s][step]):
                        p = done[s] + i
                        want = table[toks[s][p]].double() * 1.7
                        want = want + (pairs[rows[p]].double() if use_pairs else 0) + (places[p].double() if use_places else 0)
                        assert float((out[starts[j] + i].cpu().double() - want).abs().max()) < 2e-6, (s, p)
                    done[s] += cuts[s][step]
    # a position that the table lacks is reported, not read
    ctx, _ = _step_ctx([2], [42], [0])
    ctx.token_ids = torch.tensor([1, 2], dtype=torch.int32, device="cuda:0")
    out = torch.zeros(2, 256, device="cuda:0")
    ops.embedding_sum(ctx, table.cuda(), out, places=places.cuda())
    assert int(ctx.status[0]) != 0


@pytest.mark.gpu
def test_small_kernels_against_their_definitions():
    """The gated norm in groups; the norm added to the stream with the norm that follows it; products with biases in every
    epilogue and orientation; the convolution's bias; the query temperature."""
    from leone_b200.ops.cuda import CudaOps
    g = torch.Generator().manual_seed(1)
    for dtype in (torch.float32, torch.bfloat16):
        ops = CudaOps("cuda:0", dtype)
        tight, loose = (1e-5, 1e-2)
        tol = tight if dtype == torch.float32 else loose
        for n, groups, group in ((37, 3, 14), (5, 2, 192), (9, 1, 4096), (3, 8, 512), (2, 1, 5000), (4, 6, 21)):
            width = groups * group
            y, z = torch.randn(n, width, generator=g) * 3, (torch.randn(n, width + 16, generator=g) * 2).to(dtype)
            w = 1 + 0.1 * torch.randn(width, generator=g)
            out = torch.zeros(n, width, dtype=dtype, device="cuda:0")
            ops.grouped_gate_norm(y.cuda(), z.cuda()[:, 16:], w.cuda(), out, 1e-5, groups)
            want = plain.grouped_rms(y.double() * plain.silu(z[:, 16:].double()), groups, 1e-5) * w.double()
            assert float((out.cpu().double() - want).abs().max()) <= tol * float(want.abs().max()), (n, groups, group)
        for width in (36, 70, 256, 2048, 4096, 9000):
            n = 11
            a, dst = torch.randn(n, width, generator=g), torch.randn(n, width, generator=g)
            wa, wn = 1 + 0.1 * torch.randn(width, generator=g), 1 + 0.1 * torch.randn(width, generator=g)
            d, nxt = dst.clone().cuda(), torch.zeros(n, width, dtype=dtype, device="cuda:0")
            ops.rms_norm_add(d, a.cuda(), wa.cuda(), 1e-5, following=(wn.cuda(), 1e-6, nxt))
            want = plain.rms(a.double(), 1e-5) * wa.double() + dst.double()
            assert float((d.cpu().double() - want).abs().max()) < 1e-5
            want = plain.rms(want, 1e-6) * wn.double()
            assert float((nxt.cpu().double() - want).abs().max()) <= tol * float(want.abs().max()), width
        for m, k, n in ((1, 64, 48), (8, 128, 80), (17, 96, 100), (70, 72, 40), (200, 128, 272), (300, 256, 512), (600, 64, 528), (5, 50, 13)):
            x = torch.randn(m, k, generator=g).to(dtype)
            w, bias = (torch.randn(n, k, generator=g) * 0.3).to(dtype), torch.randn(n, generator=g) * 2
            res = torch.randn(m, n, generator=g)
            want = x.double() @ w.double().t() + bias.double()
            pm = ops.prepare_matrix(w.cuda(), bias.cuda())
            for out_dtype in {dtype, torch.float32}:
                out = torch.zeros(m, n, dtype=out_dtype, device="cuda:0")
                ops.linear(x.cuda(), pm, out)
                t = 1e-5 if out_dtype == torch.float32 else 1e-2
                assert float((out.cpu().double() - want).abs().max()) <= t * float(want.abs().max()), (m, k, n, out_dtype)
            out = res.clone().cuda()
            ops.linear(x.cuda(), pm, out, residual=out)
            assert float((out.cpu().double() - want - res.double()).abs().max()) <= 1e-5 * float(want.abs().max()), (m, k, n)
            gate, up = ((torch.randn(n, k, generator=g) * 0.3).to(dtype) for _ in range(2))
            gb, ub = torch.randn(n, generator=g), torch.randn(n, generator=g)
            out = torch.zeros(m, n, dtype=dtype, device="cuda:0")
            ops.linear_swiglu(x.cuda(), ops.prepare_gate_up(gate.cuda(), up.cuda(), gb.cuda(), ub.cuda()), out)
            want = plain.silu(x.double() @ gate.double().t() + gb.double()) * (x.double() @ up.double().t() + ub.double())
            assert float((out.cpu().double() - want).abs().max()) <= (1e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max()), (m, k, n)
    # the convolution with a bias, over steps with state, in every tap count's form
    ops = CudaOps("cuda:0", torch.float32)
    for channels, taps in ((10, 3), (64, 4), (24, 1), (12, 7)):
        x, w, b = torch.randn(59, channels, generator=g), torch.randn(channels, taps, generator=g), torch.randn(channels, generator=g)
        state = torch.zeros(2, taps - 1, channels, device="cuda:0") if taps > 1 else None
        got = []
        for lo, hi in ((0, 37), (37, 38), (38, 40), (40, 59)):
            ctx, _ = _step_ctx([hi - lo], [hi], [1])
            out = torch.zeros(hi - lo, channels, device="cuda:0")
            part = x[lo:hi].cuda()
            ops.short_conv(ctx, part, w.cuda(), state, out, activation="silu", update_state=state is not None and hi - lo == 1, bias=b.cuda())
            if state is not None and hi - lo != 1:
                ops.short_conv_state(ctx, part, state)
            got.append(out.cpu())
        want = plain.silu(plain.short_conv(x.double(), w.double(), b.double()))
        assert float((torch.cat(got).double() - want).abs().max()) < 1e-5, (channels, taps)


@pytest.mark.gpu
@pytest.mark.parametrize("dim,every", [(16, 1), (64, 10), (128, 64)])
def test_query_temperature_steps(dim, every):
    """The factor on a query, position by position, in both forms of the preparation kernel (the steps are where
    ``position + 1`` reaches a multiple)."""
    from leone_b200.ops.cuda import CudaOps
    n, heads, kv = 150, 3, 1
    for dtype in (torch.float32, torch.bfloat16):
        ops = CudaOps("cuda:0", dtype)
        ctx, _ = _step_ctx([n], [n], [0])
        qkv = torch.ones(n, (heads + 2 * kv) * dim, dtype=dtype, device="cuda:0")
        ops.attention_prepare(ctx, qkv, heads, kv, dim, dim, None, None, None, 1e-6, None, "half_split", None, query_temp=(0.7, every))
        want = plain.query_temperature(n, {"coef": 0.7, "every": every}, torch.float64)
        got = qkv.cpu().double()
        assert float((got[:, :heads * dim] - want[:, None]).abs().max()) <= (1e-6 if dtype == torch.float32 else 1e-2) * float(want.max())
        assert torch.equal(got[:, heads * dim:], torch.ones_like(got[:, heads * dim:]))


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "C", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(dtype, which, tmp_path):
    """generate(): admission, prompt portions mixed with decode, captured decode steps (with the
    recurrent states and last tokens in their slots), finish."""
    from leone_b200 import generate
    from leone_b200.weights.safetensors import write_safetensors
    folder = str(tmp_path / "model")
    tiny_config(which).write(folder)
    tensors = tiny_tensors(which)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    oracle = _plain(which, tensors, dtype == "bfloat16")
    prompts = [replay.random_tokens(TINY[which]["vocab"], n, 60 + n) for n in (1, 9, 40, 23, 5)]
    for kw in (dict(), dict(prefill_chunk=7, max_batch_tokens=16, use_graphs=False, prefill_first=False)):
        got = generate(folder, prompts, 10, dtype=dtype, eos_token_id=-1, max_running=3, **kw)
        for p, toks in zip(prompts, got):
            assert len(toks) == 10
            seq = list(p)
            for t in toks:
                logits = oracle.logits(seq)[-1]
                gap = float(logits.max() - logits[t])
                assert gap <= (1e-4 if dtype == "float32" else 0.05) * float(logits.abs().max()), (kw, seq, t, gap)
                seq.append(t)


@pytest.mark.gpu
def test_trace_program_on_a_written_model(tmp_path):
    """bin/trace_run as a user runs it: a folder with config.json and model.safetensors (the inner widths in the
    tensors only), steps over stdin."""
    from leone_b200.weights.safetensors import write_safetensors
    folder, out = str(tmp_path / "model"), str(tmp_path / "out")
    raw = copy.deepcopy(TINY["A"])
    for entry in raw["layers"]:
        for key in ("decay_rank", "gate_rank"):
            entry["mixer"].get("right", {}).pop(key, None)
    config_from_dict(raw).write(folder)
    tensors = {k: v.to(torch.bfloat16) for k, v in tiny_tensors("A").items()}
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    reqs = _requests(97, [30, 5, 41, 17, 8])
    steps = replay.trace_mixed(reqs, seed=11)
    got = replay.run_trace_program(folder, "float32", steps, out, replay.max_live_tokens(steps), extra=("--page-tokens", "4"))
    oracle = plain.PlainGulipel(raw, {k: v.float() for k, v in tensors.items()})
    replay.compare(steps, got, oracle, reqs, what="trace program", **FP32)
