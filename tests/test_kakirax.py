"""The Kakirax decoder through the engine against the plain implementation (tests/plain/kakirax.py).

Without a GPU the engine runs on the stand-in kernels (tests/emulated_ops.py), which checks the
configuration, the model description, layers that run other layers' tensors, the caches and states, and the
step function's cutting and batching; on a B200 the same traces run on the CUDA kernels in 32-bit and in
bfloat16, together with tests that aim at single mechanisms."""
import copy
import math
import os

import numpy as np
import pytest
import torch

from leone_b200.engine.engine import Engine
from leone_b200.registry import config_from_dict, config_from_folder, spec_from_config
from tests import replay
from tests.kakirax_tiny import PAGE_TOKENS, TINY, as_bf16, attn, gla, model, tiny_config, tiny_tensors
from tests.plain import kakirax as plain

FP32 = dict(rtol=3e-5, atol_scale=3e-5)
# bfloat16: the gained weights make scores, decays and gates sharp, which also amplifies rounding; the
# 32-bit runs are the sharp tests, these catch a wrong path or operand
BF16 = dict(rtol=8e-2, atol_scale=8e-2)
LENGTHS = [40, 7, 75, 33, 1, 64, 50]


def _bf16_round(t):
    return t.to(torch.bfloat16).to(t.dtype)


def _plain(which, tensors, bf16=False, raw=None):
    """In bfloat16 the plain model has the same stored weights and rounds what the cache holds and what
    the norms give the sublayers."""
    return plain.PlainKakirax(raw or TINY[which], as_bf16(tensors) if bf16 else tensors,
                              cache_round=_bf16_round if bf16 else None, read_round=_bf16_round if bf16 else None)


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


def _random(raw, seed, gain=4.0):
    return tiny_tensors(None, seed=seed, gain=gain, raw=raw)


def _one_layer(entry, vocab=64, width=32, eps=1e-6, **kw):
    return model(vocab, width, eps, [entry], **kw)


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
        assert all(ls.block == "pre_norm" for ls in spec.layers) and spec.lm_head_name is None
        own = [i for i, e in enumerate(raw["layers"]) if "weights_of" not in e]
        assert [ls.prefix for ls in spec.layers] == [f"l{i}" for i in own]
        assert [ls.feed_forward is None for ls in spec.layers] == [raw["layers"][i]["mlp"] is None for i in own]
        assert len(spec.run_order) == len(raw["layers"])
    assert spec_from_config(tiny_config("A")).run_order == (0, 1, 0, 2, 1)
    assert spec_from_config(tiny_config("C")).run_order == (0, 1, 1, 2, 0, 3, 1)      # layer 6 runs 2, which runs 1


def test_config_rejections():
    from leone_b200.config.base import ConfigError
    for patch in (lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
                  lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3),
                  lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18),
                  lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(high=0.5),
                  lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("low"),
                  lambda c: c["layers"][0].update(type="conv"),
                  lambda c: c["layers"][1]["mixer"].update(tau=0.0),
                  lambda c: c["layers"][1]["mixer"].pop("vdim"),
                  lambda c: c["layers"][1]["mlp"].update(kind="moe"),
                  lambda c: c["layers"][2].update(weights_of=2),            # itself
                  lambda c: c["layers"][2].update(weights_of=4),            # a layer of another kind
                  lambda c: c["layers"][2].update(weights_of=9),
                  lambda c: c["layers"][2]["mixer"].update(scale=0.5),      # not described as its source is
                  lambda c: c["layers"][0].update(weights_of=2),            # a circle
                  lambda c: c.update(logit_softcap=-1.0),
                  lambda c: c.pop("width"), lambda c: c.update(layers=[])):
        raw = copy.deepcopy(TINY["A"])
        patch(raw)
        with pytest.raises(ConfigError):
            config_from_dict(raw)


def test_decay_width_comes_from_the_checkpoint(tmp_path):
    """A configuration that does not say how wide the decay's inner projection is takes it from the tensors,
    layer by layer; without a checkpoint it stays open."""
    from leone_b200.weights.safetensors import write_safetensors
    raw = copy.deepcopy(TINY["D"])
    for entry in raw["layers"]:
        entry["mixer"].pop("decay_rank", None)
    folder = str(tmp_path)
    config_from_dict(raw).write(folder)
    assert config_from_folder(folder).needs_tensor_shapes()
    write_safetensors(os.path.join(folder, "model.safetensors"), tiny_tensors("D"))
    cfg = config_from_folder(folder)
    assert [layer.mixer.decay_rank for layer in cfg.layers if layer.type == "gla"] == [16, 4, 12]
    from tests.emulated_ops import EmulatedOps
    eng = Engine.from_folder(folder, dtype="float32", device="cpu", ops=EmulatedOps(), page_tokens=8, max_tokens=64,
                             max_requests=1, max_batch_tokens=32)
    toks = replay.random_tokens(200, 9, 1)
    got = eng.step([("r", toks, [8])])[0]
    want = _plain("D", tiny_tensors("D")).logits(toks)[8]
    assert float((got.double() - want).abs().max()) <= 3e-5 * float(want.abs().max())


# -- the plain implementation's own mechanisms, against their definitions (CPU) -----------------------
def test_plain_frequencies_by_wavelength():
    rot = {"base": 100.0, "dims": 8, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}}
    plainf = plain.frequencies({"base": 100.0, "dims": 8})
    f = plain.frequencies(rot)
    waves = [2 * math.pi / x for x in plainf]          # 6.3, 19.9, 62.8, 198.7: kept below 16, divided above 64
    assert waves[0] < 16 < waves[1] < waves[2] < 64 < waves[3]
    assert f[0] == plainf[0] and f[3] == plainf[3] / 4
    for i in (1, 2):
        s = (64 / waves[i] - 1) / 3
        assert abs(f[i] - ((1 - s) * plainf[i] / 4 + s * plainf[i])) < 1e-15 and f[i] != plainf[i]
    from leone_b200.parts.rotary import scaled_frequencies
    got, mag = scaled_frequencies(8, 100.0, {"kind": "wavelength", **rot["scaling"]})
    assert mag == 1.0 and max(abs(a - b) for a, b in zip(got, f)) < 1e-15


def test_plain_recurrence_by_hand():
    """Two channels, one of which forgets half each token: o sums what each channel still holds."""
    q = torch.tensor([[[1.0, 1.0]]] * 3, dtype=torch.float64)
    k = torch.tensor([[[1.0, 0.0]], [[0.0, 1.0]], [[0.0, 0.0]]], dtype=torch.float64)
    v = torch.tensor([[[8.0]], [[3.0]], [[100.0]]], dtype=torch.float64)
    alpha = torch.tensor([[[0.5, 1.0]]] * 3, dtype=torch.float64)
    o, S = plain.gla_recurrence(q, k, v, alpha)
    assert o[:, 0, 0].tolist() == [8.0, 4.0 + 3.0, 2.0 + 3.0] and S[0, :, 0].tolist() == [2.0, 3.0]
    W = {"a1": torch.zeros(2, 3).double(), "a2": torch.zeros(4, 2).double(), "a2.b": torch.tensor([0.0, 1.0, -3.0, 40.0]).double()}
    a = plain.channel_decay(torch.ones(1, 3).double(), W, 2.0)[0]
    assert abs(float(a[0]) - math.sqrt(0.5)) < 1e-15 and abs(float(a[2]) - (1 + math.exp(3)) ** -0.5) < 1e-15


def test_plain_layer_norm_gelu_and_rotation():
    x = torch.tensor([[1.0, 2.0, 6.0]], dtype=torch.float64)
    y = plain.layer_norm(x, torch.tensor([1.0, 2.0, 1.0]).double(), torch.tensor([0.0, 0.0, 5.0]).double(), 0.0)[0]
    sd = math.sqrt((4 + 1 + 9) / 3)
    assert abs(float(y[0]) + 2 / sd) < 1e-15 and abs(float(y[1]) + 2 / sd) < 1e-15 and abs(float(y[2]) - 3 / sd - 5) < 1e-15
    z = torch.tensor([0.7], dtype=torch.float64)
    assert abs(float(plain.gelu_tanh(z)) - 0.35 * (1 + math.tanh(math.sqrt(2 / math.pi) * (0.7 + 0.044715 * 0.343)))) < 1e-15
    r = plain.rotate(torch.arange(1.0, 7.0, dtype=torch.float64).view(1, 1, 6), [2], {"base": 100.0, "dims": 4}, torch.float64)[0, 0]
    a = [2.0, 2.0 * 100.0 ** -0.5]
    assert abs(float(r[0]) - (1 * math.cos(a[0]) - 3 * math.sin(a[0]))) < 1e-12
    assert abs(float(r[3]) - (4 * math.cos(a[1]) + 2 * math.sin(a[1]))) < 1e-12 and r[4:].tolist() == [5.0, 6.0]


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


def test_residual_stream_after_every_layer_run_on_stand_in_kernels():
    """The stream after each layer run, read from the engine's buffer by a hook on the blocks."""
    from tests.emulated_ops import EmulatedOps
    tensors = tiny_tensors("A")
    toks = replay.random_tokens(97, 19, 4)
    eng = _engine("A", tensors, "float32", "cpu", EmulatedOps())
    seen = []
    for block in eng.model.blocks:
        inner = block.forward

        def hooked(ctx, cache, hidden, inner=inner, **kw):
            r = inner(ctx, cache, hidden, **kw)
            seen.append(hidden.clone())
            return r
        block.forward = hooked
    eng.step([("r", toks, [])])
    want = _plain("A", tensors).residuals(toks)
    assert len(seen) == 5
    for i, got in enumerate(seen):
        assert float((got.double() - want[i]).abs().max()) <= 3e-5 * float(want[i].abs().max()), i


def test_every_layer_run_has_a_cache_or_state_of_its_own():
    from tests.emulated_ops import EmulatedOps
    eng = _engine("C", tiny_tensors("C"), "float32", "cpu", EmulatedOps())
    groups = sorted((g.spec.kind, g.spec.num_kv_heads, g.spec.head_dim, g.spec.value_head_dim, len(g.spec.layers))
                    for g in eng.cache.groups)
    assert groups == [("full", 2, 64, 64, 2), ("full", 2, 128, 32, 1)]     # layers 0 and 4 share tensors, not rows
    assert sorted(tuple(t.shape[1:]) for t in eng._run_state.values()) == [(2, 64, 128)] * 3 + [(4, 128, 32)]
    assert len({t.data_ptr() for t in eng._run_state.values()}) == 4
    names = [s.name for s in eng.model.weight_specs()]
    assert len(names) == len(set(names)) and not any(n.startswith(("l2.", "l4.", "l6.")) for n in names)


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
@pytest.mark.parametrize("switch", ["LEONE_NO_GLA_MMA", "LEONE_NO_TENSOR_CORES", "LEONE_NO_MASKED_MMA", "LEONE_NO_TILED_ATTENTION"])
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
@pytest.mark.parametrize("which,index", [("A", 0), ("A", 1), ("A", 3), ("B", 0), ("B", 1), ("B", 2), ("B", 3), ("C", 0), ("C", 1),
                                         ("C", 3), ("C", 5), ("D", 0), ("D", 1), ("D", 2), ("D", 3)])
def test_each_layer_alone(which, index):
    """A model of one layer: its mixer and feed-forward with nothing else to hide behind, in portions down to
    one token."""
    raw = copy.deepcopy(TINY[which])
    raw["layers"] = [raw["layers"][index]]
    tensors = {k.replace(f"l{index}.", "l0."): v for k, v in tiny_tensors(which).items()
               if not k.startswith("l") or k.startswith(f"l{index}.")}
    reqs = _requests(raw["vocab"], [45, 2, 19])
    steps = replay.trace_portions(reqs, sizes=(2, 7, 1, 2, 13))
    eng = _engine(which, tensors, "float32", "cuda:0", raw=raw, max_tokens=192, max_requests=2, max_batch_tokens=64)
    _run(steps, eng, plain.PlainKakirax(raw, tensors), reqs, f"{which} layer {index}")


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
@pytest.mark.parametrize("dtype,tol", [("float32", 1e-5), ("bfloat16", 6e-2)])
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
    """One state slot: the second request gets the slot (recurrent states of every layer run) and the pages the
    first one left, and must read none of it."""
    tensors = tiny_tensors("C")
    reqs = _requests(256, [37, 29, 61], seed=35)
    steps = replay.trace_portions(reqs, sizes=(1, 1, 2, 9, 40))
    eng = _engine("C", tensors, dtype, "cuda:0", max_tokens=64, max_requests=1)
    _run(steps, eng, _plain("C", tensors, dtype == "bfloat16"), reqs, "slot used again", dtype)


def _stand_out_model(kind):
    """A one-layer model in which token 7, and no other, writes something that token 9, and no other, reads.
    ``attention``: a key dimension (not rotated) that only token 7 fills and a query dimension that only token 9
    fills, with scores far above all others.  ``gla``: the same through the recurrence's keys and queries, with
    a decay that forgets next to nothing in that channel."""
    if kind == "attention":
        raw = _one_layer(attn(2, 1, 8, 12, 3.0, rot_dims=4))
    else:
        raw = _one_layer(gla(2, 8, 12, 16.0, 4))
    t = _random(raw, 3)
    t["embed"][:, :2] = 0.0
    for tok, coord in ((7, 0), (9, 1)):
        t["embed"][tok] = 0.0
        t["embed"][tok, coord] = 1.0
    t["l0.norm1"][:] = 1.0
    t["l0.norm1.b"][:] = 0.0
    row = 4 if kind == "attention" else 3
    for name in ("q", "k"):
        t[f"l0.mix.{name}"][:, :2] = 0.0
        t[f"l0.mix.{name}"][row] = 0.0
    # (after the norm the coordinate is about 5.4 for its token and, the mean being taken off, a few tenths for others)
    t["l0.mix.k"][row, 0] = t["l0.mix.q"][row, 1] = 3.0
    if kind == "gla":
        t["l0.mix.a2"][row] = 0.0
        t["l0.mix.a2.b"][row] = 9.0
    return raw, t


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,bound", [("float32", 3e-5), ("bfloat16", 4e-2)])
@pytest.mark.parametrize("kind,q_pos,k_pos", [
    ("attention", 330, 0), ("attention", 200, 17), ("attention", 48, 47), ("attention", 64, 15), ("attention", 33, 16),
    ("attention", 65, 64), ("gla", 300, 2), ("gla", 40, 39), ("gla", 65, 0), ("gla", 17, 16), ("gla", 32, 31), ("gla", 192, 127),
    ("gla", 192, 128), ("gla", 340, 63), ("gla", 340, 64)])
def test_a_far_write_is_read(kind, q_pos, k_pos, dtype, bound):
    """What one token wrote hundreds of tokens back (a key at a page's border; a write into the recurrent state
    at the border of a group of 16 tokens or of a chunk) is what another reads, in a prompt, in portions, and
    through decoding."""
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


def _step_ctx(q_lens, ctx_lens, slots, dev="cuda:0"):
    """What the kernels read of a step: ``q_lens[s]`` new tokens of sequence ``s`` that end at ``ctx_lens[s]``."""
    from types import SimpleNamespace
    starts = [0]
    for x in q_lens:
        starts.append(starts[-1] + x)
    return SimpleNamespace(n_seqs=len(q_lens), n_tokens=int(sum(q_lens)), q_lens=np.asarray(q_lens),
                           q_start=torch.tensor(starts, dtype=torch.int32, device=dev),
                           slot_ids=torch.tensor(slots, dtype=torch.int32, device=dev), max_q_len=max(q_lens),
                           max_ctx_len=max(ctx_lens), decode_only=max(q_lens) == 1,
                           status=torch.zeros(4, dtype=torch.int32, device=dev)), starts


@pytest.mark.gpu
@pytest.mark.parametrize("heads,dim,vdim,rank,tau,strong", [
    (3, 12, 20, 5, 4.0, 0.0), (1, 5, 7, 3, 1.0, 0.0), (2, 64, 64, 16, 16.0, 0.0), (2, 128, 128, 16, 16.0, 0.0), (1, 144, 40, 24, 8.0, 0.0),
    (1, 300, 24, 4, 12.0, 0.0), (1, 512, 40, 8, 12.0, 0.0), (2, 32, 200, 12, 6.0, 0.0), (2, 96, 80, 32, 2.0, 0.0), (4, 40, 56, 9, 5.0, 0.0),
    (2, 128, 256, 16, 16.0, 0.0), (3, 20, 132, 7, 3.0, 0.0),
    # decays so strong that sixteen of them together leave nothing (and single ones that leave next to nothing)
    (2, 64, 64, 16, 1.0, 4.0), (2, 128, 128, 8, 1.0, 9.0), (1, 20, 24, 6, 1.0, 60.0)])
def test_gla_kernels_against_the_plain_recurrence(heads, dim, vdim, rank, tau, strong):
    """The recurrence's kernels alone in every form (the walk's register forms, tensor cores, chunks side by
    side): three sequences in steps of unequal sizes with the state carried in slots that are not in order."""
    from leone_b200.ops.cuda import CudaOps
    g = torch.Generator().manual_seed(dim + vdim)
    lengths, slots = [277, 3, 85], [2, 0, 3]
    hd, hv = heads * dim, heads * vdim
    cols = -(-(2 * hd + 2 * hv + rank) // 16) * 16
    offs = dict(q_off=0, k_off=hd, v_off=2 * hd, gate_off=2 * hd + hv, u_off=2 * hd + 2 * hv)
    rows = [torch.randn(n, cols, generator=g) for n in lengths]
    w2, bias = torch.randn(rank, hd, generator=g) * rank ** -0.5 * 2, torch.randn(hd, generator=g) - strong
    norm_w = 1 + 0.1 * torch.randn(vdim, generator=g)
    cuts = [[200, 1, 1, 2, 73], [1, 2], [2, 1, 82]]
    scale = dim ** -0.5
    want, states = [], []
    for s, n in enumerate(lengths):
        r = rows[s].double()
        z = r[:, offs["u_off"]:offs["u_off"] + rank] @ w2.double() + bias.double()
        alpha = (torch.sigmoid(z) ** (1.0 / tau)).view(n, heads, dim)
        o, S = plain.gla_recurrence(r[:, :hd].view(n, heads, dim) * scale, r[:, hd:2 * hd].view(n, heads, dim),
                                    r[:, 2 * hd:2 * hd + hv].view(n, heads, vdim), alpha)
        y = (plain.rms(o, 1e-5) * norm_w.double()).reshape(n, hv)
        want.append(y * plain.silu(r[:, offs["gate_off"]:offs["gate_off"] + hv]))
        states.append(S)
    for dtype, chunk, tol in ((torch.float32, 0, 3e-5), (torch.float32, 32, 3e-5), (torch.bfloat16, 0, 1e-2), (torch.bfloat16, 32, 1e-2),
                              (torch.bfloat16, 64, 1e-2)):
        ops = CudaOps("cuda:0", dtype)
        state = torch.randn(4, heads, dim, vdim, generator=g).cuda()       # what a slot held before must not matter
        state[slots] = 0.0
        done = [0, 0, 0]
        got = [torch.zeros(n, hv, dtype=torch.float64) for n in lengths]
        for step in range(5):
            live = [s for s in range(3) if step < len(cuts[s])]
            q_lens = [cuts[s][step] for s in live]
            ctx, starts = _step_ctx(q_lens, [done[s] + cuts[s][step] for s in live], [slots[s] for s in live])
            proj = torch.cat([rows[s][done[s]:done[s] + cuts[s][step]] for s in live]).cuda()
            out = torch.zeros(sum(q_lens), hv, dtype=dtype, device="cuda:0")
            ops.gated_linear_attention(ctx, proj, out, state, w2.cuda(), bias.cuda(), norm_w.cuda(), heads, dim, vdim, rank, tau,
                                       scale, 1e-5, chunk=chunk if max(q_lens) > 2 * chunk else 0, **offs)
            assert int(ctx.status[0]) == 0
            for j, s in enumerate(live):
                got[s][done[s]:done[s] + cuts[s][step]] = out[starts[j]:starts[j + 1]].cpu().double()
                done[s] += cuts[s][step]
        for s in range(3):
            err = float((got[s] - want[s]).abs().max()) / float(want[s].abs().max())
            assert err <= tol, (dtype, chunk, s, err)
            serr = float((state[slots[s]].cpu().double() - states[s]).abs().max()) / float(states[s].abs().max())
            assert serr <= 3e-5, (dtype, chunk, s, "state", serr)


@pytest.mark.gpu
def test_small_kernels_against_their_definitions():
    """Layer norm (with a large mean, gathered rows, every width form), the gated layer's gelu, the output gate on
    a column slice."""
    from leone_b200.ops.cuda import CudaOps
    g = torch.Generator().manual_seed(1)
    for dtype in (torch.float32, torch.bfloat16):
        ops = CudaOps("cuda:0", dtype)
        for width in (7, 70, 320, 512, 2048, 4096, 9000):
            x = torch.randn(9, width, generator=g) * 2 + 50.0
            w, b = (1 + 0.1 * torch.randn(width, generator=g)).to(dtype), torch.randn(width, generator=g).to(dtype)
            for rows in (None, torch.tensor([8, 0, 3], dtype=torch.int32)):
                for bias in (b, None):
                    for wide in (dtype, torch.float32):
                        src = x if rows is None else x[rows.long()]
                        out = torch.zeros(src.shape, dtype=wide, device="cuda:0")
                        ops.layer_norm(x.cuda(), w.cuda(), None if bias is None else bias.cuda(), out, 1e-5,
                                       None if rows is None else rows.cuda())
                        want = plain.layer_norm(src.double(), w.double(), torch.zeros(width) if bias is None else bias.double(), 1e-5)
                        tol = 1e-5 if wide == torch.float32 else 8e-3
                        assert float((out.cpu().double() - want).abs().max()) <= tol * float(want.abs().max()), (width, dtype)
        for tokens, hidden, inter in ((5, 64, 48), (70, 72, 40), (300, 128, 256), (3, 50, 13)):
            x = torch.randn(tokens, hidden, generator=g).to(dtype)
            gate, up = (torch.randn(inter, hidden, generator=g).to(dtype) * 0.3 for _ in range(2))
            out = torch.zeros(tokens, inter, dtype=dtype, device="cuda:0")
            shape = (2.0 * math.sqrt(2.0 / math.pi), float("inf"), 0.0, 0.044715)
            ops.linear_swiglu(x.cuda(), ops.prepare_gate_up(gate.cuda(), up.cuda()), out, gate_shape=shape)
            want = plain.gelu_tanh(x.double() @ gate.double().t()) * (x.double() @ up.double().t())
            tol = 1e-5 if dtype == torch.float32 else 2e-2
            assert float((out.cpu().double() - want).abs().max()) <= tol * float(want.abs().max()), (tokens, dtype)
        a, z = torch.randn(37, 72, generator=g).to(dtype), torch.randn(37, 96, generator=g).to(dtype) * 3
        y = a.clone().cuda()
        ops.gate_rows(y, z.cuda()[:, 16:88], "sigmoid")
        want = a.double() * torch.sigmoid(z[:, 16:88].double())
        assert float((y.cpu().double() - want).abs().max()) <= (1e-6 if dtype == torch.float32 else 1e-2) * float(want.abs().max())


@pytest.mark.gpu
@pytest.mark.parametrize("which", ["A", "C", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(dtype, which, tmp_path):
    """generate(): admission, prompt portions mixed with decode, captured decode steps (with the
    recurrent states in their slots), finish."""
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
    """bin/trace_run as a user runs it: a folder with config.json and model.safetensors (the decay's inner width
    in the tensors only), steps over stdin."""
    from leone_b200.weights.safetensors import write_safetensors
    folder, out = str(tmp_path / "model"), str(tmp_path / "out")
    raw = copy.deepcopy(TINY["A"])
    for entry in raw["layers"]:
        entry["mixer"].pop("decay_rank", None)
    config_from_dict(raw).write(folder)
    tensors = {k: v.to(torch.bfloat16) for k, v in tiny_tensors("A").items()}
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    reqs = _requests(97, [30, 5, 41, 17, 8])
    steps = replay.trace_mixed(reqs, seed=11)
    got = replay.run_trace_program(folder, "float32", steps, out, replay.max_live_tokens(steps), extra=("--page-tokens", "4"))
    oracle = plain.PlainKakirax(raw, {k: v.float() for k, v in tensors.items()})
    replay.compare(steps, got, oracle, reqs, what="trace program", **FP32)
