"""Defilorn (layers listed in config.json: mLSTM recurrences, latent attention with interpolated
rotation, sinks and an output gate per entry, differential attention over a sliding window; pre-norm
blocks with norm weights stored around zero, a repeated run of layers whose later passes open with the
embedding, tanh-GELU gated dense layers, softmax-routed gated experts among which some are the identity
and an always-on expert with a gate per token) against the plain float64 restatement in
tests/defilorn_ref.py.  Every test makes its own small configuration and random weights."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

from helpers import C, E, W, ROOT
import nvllm_pkg
import defilorn_ref as ref
from st_writer import write_safetensors
from test_zozonex import Engine, prompt
from test_lazovik import check

gpu = pytest.mark.gpu
BLOCK = C.KV_BLOCK_SIZE
PRECS = [C.PREC_FP32, C.PREC_BF16]


# ------------------------------------------------------------------ configurations
def ml(heads=3, dim=16, vdim=20, cap=7.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def lat(heads=5, dim=16, rot_dim=8, vdim=12, kv_rank=24, q_rank=40, base=500.0, factor=4.0, original=64, fast=8.0, slow=0.5, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "rot": {"base": base, "dims": rot_dim, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}},
                      "scale": float((dim + rot_dim) ** -0.5 if scale is None else scale)}}


def att(heads=6, kv_heads=2, dim=12, vdim=20, size=21, diff=0.35, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                                           "diff": diff, "scale": float(dim ** -0.5 if scale is None else scale)}}


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=7, top=2, identity=3, shared=36):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}, "shared": {"ff": shared}}


def layer(mix, mlp=None):
    return dict(copy.deepcopy(mix), mlp=mlp)


def model(layers, vocab=211, width=72, eps=1e-5, loop=None):
    j = {"architecture": "Defilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        j["loop"] = dict(zip(("start", "stop", "times"), loop))
    return j


def mixed_model():
    """Every mixer and feed-forward and none, sizes that differ layer to layer, a repeated run with a
    cache and a state in it."""
    return model([layer(att(), moe()),
                  layer(ml(), dense()),
                  layer(lat(), moe(experts=5, top=3, identity=1, shared=20)),
                  layer(att(heads=4, kv_heads=4, dim=16, vdim=8, size=50, diff=0.8), dense(ff=100)),
                  layer(ml(heads=2, dim=24, vdim=8, cap=20.0)),
                  layer(lat(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=16, q_rank=16, base=30.0), moe(ff=40, top=4))],
                 loop=(1, 4, 2))


def odd_model():
    """Sizes that are multiples of nothing convenient, windows of one and two tokens, one head, one
    expert, more chosen than there are real experts, a run from the first layer on."""
    return model([layer(att(heads=3, kv_heads=1, dim=5, vdim=7, size=1)),
                  layer(ml(heads=5, dim=6, vdim=10), moe(ff=20, experts=2, top=4, identity=3, shared=12)),
                  layer(lat(heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=9, q_rank=11), dense(ff=33)),
                  layer(att(heads=1, kv_heads=1, dim=10, vdim=30, size=2), dense(ff=9)),
                  layer(ml(heads=1, dim=37, vdim=41), moe(ff=9, experts=1, top=1, identity=1, shared=5))],
                 vocab=101, width=40, eps=3e-4, loop=(0, 3, 3))


def mma_model():
    """Sizes that take the tensor-core kernels in bf16; recurrences at sizes of a real model's heads."""
    return model([layer(lat(heads=8, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=64), moe(ff=64, experts=8, shared=64)),
                  layer(ml(heads=4, dim=64, vdim=128), dense(ff=256)),
                  layer(att(heads=8, kv_heads=2, dim=32, vdim=64, size=70), moe(ff=96, experts=4, top=1)),
                  layer(lat(heads=16, dim=32, rot_dim=64, vdim=72, kv_rank=128, q_rank=96), dense(ff=128)),
                  layer(ml(heads=2, dim=128, vdim=64), moe(ff=64, experts=8, top=3, shared=128)),
                  layer(att(heads=2, kv_heads=2, dim=64, vdim=128, size=200), dense(ff=136))],
                 width=128, loop=(1, 4, 2))


def random_weights(j, seed, bf16=False):
    cfg = C.defilorn_from_json(j)
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in cfg.tensor_shapes().items():
        if name.endswith((".q.norm", ".k.norm")) or name.endswith(".mix.norm"):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith((".dq.norm", ".dkv.norm")):
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name.endswith((".norm1", ".norm2", "final.norm")):
            a = 0.2 * rng.standard_normal(shape)  # stored around zero
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            a = 1.2 * rng.standard_normal(shape) / np.sqrt(np.sqrt(shape[0]) + 1.0)
        elif name.endswith(".sink"):
            a = 1.5 * rng.standard_normal(shape)
        elif name.endswith(".i.b"):
            a = rng.standard_normal(shape)
        elif name.endswith(".f.b"):
            a = rng.uniform(0.0, 4.0, shape)
        elif name.endswith(".correction"):
            a = 0.3 * rng.standard_normal(shape)  # as large as the scores: without it other experts are chosen
        elif name == "embed":
            a = rng.standard_normal(shape)
        elif name.endswith(".router"):
            a = 2.0 * rng.standard_normal(shape) / np.sqrt(shape[1])
        else:
            a = rng.standard_normal(shape) / np.sqrt(shape[1])
        a = np.asarray(a, dtype=np.float32)
        w[name] = W.bf16_round(a) if bf16 else a
    return cfg, w


def setup(j, prec, seed=7, **kw):
    cfg, w = random_weights(j, seed, bf16=prec == C.PREC_BF16)
    return cfg, w, Engine(cfg, w, prec, **kw)


def no_close_calls(j, prec):
    """With random weights, some token in a few hundred has two choice scores closer than bf16
    rounding, and a run that then picks the other expert is not comparable from that token on.  The
    bf16 runs of models with several layers therefore use ALL experts of a layer (the scores still
    weight them); the choice is tested in fp32 and, in bf16, on single layers."""
    if prec == C.PREC_FP32:
        return j
    j = copy.deepcopy(j)
    for lc in j["layers"]:
        if lc.get("mlp") and lc["mlp"]["kind"] == "moe":
            r = lc["mlp"]["router"]
            r["top"] = r["experts"] + r["identity"]
    return j


def routed(j):
    return any(lc.get("mlp") and lc["mlp"]["kind"] == "moe" for lc in j["layers"])


# ------------------------------------------------------------------ CPU: configuration, the restatement itself
def test_config_reader_takes_every_size_and_constant_from_the_file():
    j = mixed_model()
    cfg = C.ARCHITECTURES[j["architecture"]](j)
    assert cfg.arch == C.ARCH_DEFILORN and not cfg.tied_head and cfg.needs_state_slots and cfg.norm_offset == 1.0
    assert cfg.block_style == C.LBLOCK_SEQUENTIAL_PRENORM and cfg.loop_embed
    assert (cfg.vocab_size, cfg.hidden, cfg.norm_eps, cfg.loop_start, cfg.loop_stop, cfg.loop_times) == (211, 72, 1e-5, 1, 4, 2)
    assert list(cfg.runs) == [0, 1, 2, 3, 1, 2, 3, 4, 5]
    d0, m1, a2, d3, m4, a5 = cfg.layers
    assert [l.mixer for l in cfg.layers] == [C.MIXER_ATTENTION, C.MIXER_MLSTM, C.MIXER_LATENT_ATTENTION] * 2
    assert (d0.heads, d0.kv_heads, d0.dim, d0.vdim, d0.window, d0.diff_maps, d0.diff, d0.qk_norm, d0.rot_dims) == (6, 2, 12, 20, 21, 1, 0.35, 3, 0)
    assert (d3.window, d3.diff, d3.kv_heads) == (50, 0.8, 4) and abs(d3.scale - 0.25) < 1e-12
    assert (m1.heads, m1.dim, m1.vdim, m1.gate_cap, m4.gate_cap) == (3, 16, 20, 7.0, 20.0)
    assert (a2.heads, a2.dim, a2.rot_dim, a2.vdim, a2.kv_rank, a2.q_rank, a2.rot_pairs, a2.out_gate, a2.sink_learned) == (5, 16, 8, 12, 24, 40, 1, 1, 1)
    assert (a2.rot_base, a2.rot_factor, a2.rot_original, a2.rot_fast, a2.rot_slow, a5.rot_base) == (500.0, 4.0, 64.0, 8.0, 0.5, 30.0)
    assert a2.window == 0 and abs(a2.scale - 24 ** -0.5) < 1e-12
    assert (m1.mlp, m1.act, m1.ff) == (C.MLP_DENSE, C.FFN_GEGLU, 56) and m4.mlp == C.MLP_NONE
    assert (a2.mlp, a2.act, a2.ff, a2.experts, a2.top, a2.route_identity, a2.route_correction, a2.route_raw, a2.shared_ff, a2.shared_gate) == \
        (C.MLP_MOE, C.FFN_SWIGLU, 24, 5, 3, 1, 1, 1, 20, 1)
    sh = cfg.tensor_shapes()
    assert sh["head"] == (211, 72) and "loop.step" not in sh and "final.norm.b" not in sh and "l4.norm2" not in sh
    assert sh["l0.mix.q"] == (6 * 2 * 12, 72) and sh["l0.mix.k"] == (2 * 2 * 12, 72) and sh["l0.mix.v"] == (40, 72) and sh["l0.mix.lq2"] == (12,)
    assert sh["l2.mix.g"] == (60, 72) and sh["l2.mix.sink"] == (5,) and sh["l2.mix.uq"] == (120, 40) and sh["l2.mix.dkv"] == (32, 72)
    assert sh["l1.mix.norm"] == (60,) and sh["l1.mix.i"] == (3, 72) and sh["l1.mix.f.b"] == (3,) and sh["l1.mlp.gate"] == (56, 72)
    assert sh["l2.mlp.router"] == (6, 72) and sh["l2.mlp.correction"] == (6,) and sh["l2.mlp.shared.sg"] == (1, 72) and "l2.mlp.e5.up" not in sh
    c, specs = cfg.to_c(C.PREC_FP32, num_state_slots=3)
    assert (c.loop_embed, c.loop_times, c.num_state_slots) == (1, 2, 3) and specs[0].diff_maps == 1 and specs[2].route_identity == 1
    # every pass has caches and state of its own
    assert cfg.cache_bytes_per_token(2) == 2 * (2 * (24 + 20) + 2 * (32 + 4 * (32 + 8)) + 20)
    assert cfg.state_bytes_per_sequence() == 4 * (2 * 3 * (16 * 20 + 16 + 1) + 2 * (24 * 8 + 24 + 1))
    plain = C.defilorn_from_json(model([layer(lat())]))
    assert not plain.needs_state_slots and list(plain.runs) == [0]
    with pytest.raises(ValueError):
        C.defilorn_from_json(model([dict(type="conv", mixer=ml()["mixer"], mlp=None)]))
    with pytest.raises(ValueError):
        C.defilorn_from_json(model([layer(ml(), {"kind": "poly", "ff": 8})]))


def test_reference_mechanisms_against_hand_computed_values():
    """The restatement itself, on inputs small enough to check by hand."""
    assert np.allclose(ref.over_rms(np.array([[3.0, 4.0]]), 0.5), np.array([[3.0, 4.0]]) / np.sqrt(13.0))
    assert abs(ref.gelu_tanh(np.array(1.0)) - 0.841192) < 1e-6 and abs(ref.log_sigmoid(np.array(0.0)) + np.log(2.0)) < 1e-12
    # frequencies: turning fast (kept), slow (divided), cos and sin scaled
    f, mult = ref.frequencies({"dims": 4, "base": 100.0, "scaling": {"factor": 8.0, "original": 100, "fast": 10.0, "slow": 1.0}})
    at = lambda turns: 4 * np.log(100 / (2 * np.pi * turns)) / (2 * np.log(100.0))
    assert (np.floor(at(10.0)), np.ceil(at(1.0))) == (0, 2)
    assert np.allclose(f, [1.0, 0.5 * 0.1 + 0.5 * 0.1 / 8]) and abs(mult - (1 + 0.1 * np.log(8.0))) < 1e-12
    x = ref.rotate_pairs(np.array([[[1.0, 0.0, 1.0, 0.0, 5.0]]] * 2), {"dims": 4, "base": 100.0}, np.array([0.0, 1.0]))
    assert np.allclose(x[1, 0], [np.cos(1), np.sin(1), np.cos(0.1), np.sin(0.1), 5])
    p = ref.softmax_rows(np.zeros((4, 4)), 2)
    assert np.allclose(p, [[1, 0, 0, 0], [.5, .5, 0, 0], [0, .5, .5, 0], [0, 0, .5, .5]])
    assert np.allclose(ref.softmax_rows(np.zeros((3, 3)), 0, sink=np.log(2.0))[2], 0.2)
    # matrix memory, gates open (forget 1, write e^0): S = 4 then 4 + 6, n = 1 then 2; q = 1 divides by max(n, 1)
    o = ref.matrix_memory(np.ones((2, 1)), np.ones((2, 1)), np.array([[4.0], [6.0]]), np.zeros(2), np.zeros(2))
    assert np.allclose(o.ravel(), [4.0 / (1 + 1e-6), 10.0 / (2 + 1e-6)])
    # the maximum starts at 0: a first write of e^-3 is weighed against 1
    o = ref.matrix_memory(np.ones((1, 1)), np.ones((1, 1)), np.array([[4.0]]), np.array([-3.0]), np.zeros(1))
    assert np.allclose(o, 4 * np.exp(-3.0) / (1 + 1e-6))
    # ... and moves with the input gate: everything relative to e^5
    o = ref.matrix_memory(np.ones((1, 1)), np.full((1, 1), 2.0), np.array([[4.0]]), np.array([5.0]), np.array([-1.0]))
    assert np.allclose(o, 8.0 / (2 + 1e-6))
    idx, s = ref.route(np.log(np.array([1.0, 3.0, 4.0])), np.array([0.6, 0.0, 0.0]), 2)
    assert idx == [0, 2] and np.allclose(s, [1 / 8, 4 / 8])
    w = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.25]), "lq2": np.array([1.0, 0.0]), "lk2": np.array([0.5, 9.0])}
    assert abs(ref.difference_weight(w, "", 0.25) - (np.exp(1.0) - np.exp(0.5) + 0.25)) < 1e-12
    assert ref.schedule({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == \
        [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]


# ------------------------------------------------------------------ GPU: each mechanism alone
CASES = {
    "mlstm": lambda: model([layer(ml())]),
    "mlstm_one_head_one_key_entry": lambda: model([layer(ml(heads=1, dim=1, vdim=1))]),
    "mlstm_wide_state": lambda: model([layer(ml(heads=2, dim=200, vdim=48))]),
    "mlstm_wide_values": lambda: model([layer(ml(heads=1, dim=12, vdim=300))]),
    "mlstm_heads_of_64_by_128": lambda: model([layer(ml(heads=2, dim=64, vdim=128, cap=15.0))], width=128),
    "mlstm_small_cap": lambda: model([layer(ml(cap=0.7))]),
    "latent": lambda: model([layer(lat())]),
    "latent_rank_64_rot_16": lambda: model([layer(lat(heads=8, kv_rank=64, rot_dim=16, q_rank=64))], width=128),
    "latent_rank_128_rot_64": lambda: model([layer(lat(heads=8, dim=64, vdim=64, kv_rank=128, rot_dim=64, q_rank=64, base=20000.0))], width=128),
    "latent_rank_256_rot_32": lambda: model([layer(lat(heads=4, dim=32, vdim=136, kv_rank=256, rot_dim=32, q_rank=64))], width=128),
    "latent_rank_320": lambda: model([layer(lat(heads=2, dim=32, vdim=64, kv_rank=320, rot_dim=32, q_rank=24))], width=64),
    "latent_scaling_of_one": lambda: model([layer(lat(factor=1.0, original=7, fast=1.0, slow=1.0))]),
    "latent_narrow_ramp": lambda: model([layer(lat(rot_dim=16, base=20.0, factor=30.0, original=40, fast=2.0, slow=1.5))]),
    "attention": lambda: model([layer(att())]),
    "attention_groups_of_one": lambda: model([layer(att(heads=3, kv_heads=3, size=40))]),
    "attention_window_of_one": lambda: model([layer(att(size=1))]),
    "attention_window_past_the_prompt": lambda: model([layer(att(size=1000, dim=8, vdim=32, heads=10))]),
    "attention_equal_sizes": lambda: model([layer(att(dim=32, vdim=32, heads=8, kv_heads=1, size=33))], width=128),
    "attention_32_by_64": lambda: model([layer(att(dim=32, vdim=64, heads=4, kv_heads=2, size=65))], width=128),
    "attention_64_by_64": lambda: model([layer(att(dim=64, vdim=64, heads=6, kv_heads=2, size=40))], width=128),
    "attention_64_by_128": lambda: model([layer(att(dim=64, vdim=128, heads=4, kv_heads=2, size=50))], width=128),
    "attention_128_by_128": lambda: model([layer(att(dim=128, vdim=128, heads=2, kv_heads=1, size=30))], width=128),
    "attention_24_by_128_groups_of_five": lambda: model([layer(att(dim=24, vdim=128, heads=10, kv_heads=2, size=30))], width=128),
    "attention_wide_values": lambda: model([layer(att(dim=9, vdim=260, heads=2, kv_heads=2, size=30))], width=64),
    "gated_dense": lambda: model([layer(ml(), dense(ff=50))]),
    "gated_dense_wide": lambda: model([layer(ml(), dense(ff=1000))], width=128),
    "experts": lambda: model([layer(ml(), moe(ff=20, experts=12, top=3))]),
    "experts_without_identity": lambda: model([layer(lat(), moe(ff=20, experts=9, top=1, identity=0))]),
    "experts_mostly_identity": lambda: model([layer(lat(), moe(ff=64, experts=2, top=5, identity=20, shared=200))], width=128),
    "run_of_one_layer": lambda: model([layer(ml()), layer(att(), dense())], loop=(0, 1, 4)),
    "run_of_one_pass": lambda: model([layer(ml(), dense()), layer(lat())], loop=(0, 2, 1)),
    "run_of_everything": lambda: model([layer(lat(), moe()), layer(att(), moe())], loop=(0, 2, 2)),
}


@gpu
@pytest.mark.parametrize("prec", PRECS)
@pytest.mark.parametrize("case", sorted(CASES))
def test_each_mechanism_alone(case, prec):
    j = CASES[case]()
    if len(j["layers"]) > 1:
        j = no_close_calls(j, prec)
    cfg, w, eng = setup(j, prec)
    try:
        toks = prompt(j, 90, 1)
        want = ref.forward(j, w, toks)
        got, _ = eng.step([("a", toks[:78], list(range(78)))])
        rows = [eng.step([("a", [t], [0])], decode=True)[0][0] for t in toks[78:]]
        check(np.concatenate([got, np.stack(rows)]), want, prec, case, routed(j))
    finally:
        eng.close()


@gpu
def test_residual_stream_after_every_layer():
    """One layer more, one more entry of the reference's stream to meet: models of 1 .. n layers
    share their first layers' weights, the last layer's output is read through norm and head."""
    full = mixed_model()
    cfgf, wf = random_weights(full, 9)
    toks = prompt(full, 50, 2)
    for n in range(1, len(full["layers"]) + 1):
        j = dict(full, layers=full["layers"][:n], loop=full["loop"] if n >= 4 else None)
        cfg = C.defilorn_from_json(j)
        w = {k: wf[k] for k in cfg.tensor_shapes()}
        eng = Engine(cfg, w, C.PREC_FP32)
        try:
            got, _ = eng.step([("a", toks, list(range(50)))])
            check(got, ref.forward(j, w, toks), C.PREC_FP32, f"{n} layers")
        finally:
            eng.close()


MODELS = {"mixed": mixed_model, "odd": odd_model, "mma": mma_model}


# ------------------------------------------------------------------ GPU: schedules
@gpu
@pytest.mark.parametrize("prec", PRECS)
@pytest.mark.parametrize("which", sorted(MODELS))
def test_prefill_equals_token_by_token_decoding(which, prec):
    j = no_close_calls(MODELS[which](), prec)
    cfg, w, eng = setup(j, prec)
    try:
        toks = prompt(j, 70, 2)
        want = ref.forward(j, w, toks)
        got, _ = eng.step([("whole", toks, list(range(70)))])
        check(got, want, prec, "whole prompt", True)
        rows = [eng.step([("dec", toks[:9], [8])])[0][0]]
        for t in range(9, 70):
            rows.append(eng.step([("dec", [toks[t]], [0])], decode=True)[0][0])
        check(np.stack(rows), want[8:], prec, "decoded", True)
        if prec == C.PREC_FP32:  # the same arithmetic either way: far closer to each other than to float64
            assert np.abs(np.stack(rows) - got[8:]).max() <= 4e-5 * np.abs(want).max()
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
@pytest.mark.parametrize("which", sorted(MODELS))
def test_portions_of_several_sizes_down_to_two_tokens(which, prec):
    j = no_close_calls(MODELS[which](), prec)
    cfg, w, eng = setup(j, prec)
    try:
        toks = prompt(j, 331, 3)
        want = ref.forward(j, w, toks)
        got, pos = [], 0
        for n in [2, 3, 2, 16, 17, 40, 1, 5, 100, 2, 71, 2, 70]:  # (one portion crosses the page border at 256)
            out, _ = eng.step([("p", toks[pos:pos + n], list(range(n)))])
            got.append(out)
            pos += n
        assert pos == 331
        check(np.concatenate(got), want, prec, "portions", True)
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("which,prec", [("mixed", C.PREC_FP32), ("odd", C.PREC_FP32), ("mma", C.PREC_BF16)])
def test_batches_of_unequal_requests_equal_each_alone(which, prec):
    j = no_close_calls(MODELS[which](), prec)
    cfg, w, eng = setup(j, prec, num_blocks=10, slots=5)
    try:
        A, B, Cc, Dd = (prompt(j, n, s) for n, s in ((150, 4), (41, 5), (7, 6), (290, 7)))
        wa, wb, wc, wd = (ref.forward(j, w, t) for t in (A, B, Cc, Dd))
        g1, _ = eng.step([("a", A[:100], [0, 99]), ("b", B, [40]), ("c", Cc[:2], [1])])
        g2, _ = eng.step([("c", Cc[2:], [4]), ("a", A[100:], [49]), ("b", [3], [0]), ("d", Dd[:260], [255, 256, 259])])
        wb2 = ref.forward(j, w, B + [3])
        g3, _ = eng.step([("d", [Dd[260]], [0]), ("a", [9], [0]), ("c", [11], [0])], decode=True)
        # one row each, but a first row among them: a ragged step with as many rows as sequences
        g4, _ = eng.step([("d", [Dd[261]], [0]), ("e", [5], [0]), ("a", [2], [0])])
        got = np.concatenate([g1, g2, g3, g4])
        wa2 = ref.forward(j, w, A + [9, 2])
        want = np.stack([wa[0], wa[99], wb[40], wc[1], wc[6], wa[149], wb2[41], wd[255], wd[256], wd[259], wd[260],
                         wa2[150], ref.forward(j, w, Cc + [11])[7], wd[261], ref.forward(j, w, [5])[0], wa2[151]])
        check(got, want, prec, "four steps", True)
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
def test_pages_and_slots_are_freed_and_used_again(prec):
    j = no_close_calls(mixed_model(), prec)
    cfg, w, eng = setup(j, prec, num_blocks=3, slots=2)
    try:
        got, want = [], []
        for r in range(5):  # 5 pairs of requests through 2 slots and 3 pages; each leaves state and cache rows behind
            a, b = prompt(j, 200 + 20 * r, 10 + r), prompt(j, 30 + r, 20 + r)
            ga, _ = eng.step([("a", a[:120], [119]), ("b", b[:10], [9])])
            gb, _ = eng.step([("a", a[120:], [len(a) - 121]), ("b", b[10:], [len(b) - 11])])
            wa, wb = ref.forward(j, w, a), ref.forward(j, w, b)
            got += [ga, gb]
            want += [wa[119], wb[9], wa[-1], wb[-1]]
            if r % 2:
                eng.end("a"), eng.end("b")
            else:
                eng.end("b"), eng.end("a")
        check(np.concatenate(got), np.stack(want), prec, "five rounds", True)
        assert len(eng.bm.free_block_ids) == 3 and len(eng.bm.free_state_slots) == 2
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("which,prec", [("odd", C.PREC_FP32), ("mixed", C.PREC_FP32), ("mixed", C.PREC_BF16), ("mma", C.PREC_BF16)])
def test_first_tokens_of_a_sequence(which, prec):
    """Positions 0, 1, 2: shorter than the windows and any tile; state, normaliser and running maximum
    begin at zero whatever the slot held — for a first row inside a prompt and for a prompt of a
    single token."""
    j = no_close_calls(MODELS[which](), prec)
    cfg, w, eng = setup(j, prec)
    try:
        eng.step([("dirt", prompt(j, 40, 29), [])])  # leaves state and rows in slot and page
        eng.end("dirt")
        for n in (1, 2, 3):
            toks = prompt(j, n, 30 + n)
            got, _ = eng.step([("s", toks, list(range(n)))])
            nxt = [eng.step([("s", [t], [0])], decode=True)[0] for t in (4, 9, 4, 7)]
            want = ref.forward(j, w, toks + [4, 9, 4, 7])
            check(np.concatenate([got] + nxt), want, prec, f"{n} tokens + 4", True)
            eng.end("s")
    finally:
        eng.close()


@gpu
def test_long_decoding_stays_on_the_reference():
    j = mixed_model()
    cfg, w, eng = setup(j, C.PREC_FP32)
    try:
        toks = prompt(j, 460, 40)
        want = ref.forward(j, w, toks)
        eng.step([("l", toks[:20], [])])
        rows = [eng.step([("l", [toks[t]], [0])], decode=True)[0][0] for t in range(20, 460)]
        check(np.stack(rows), want[20:], C.PREC_FP32, "440 decoded tokens")
    finally:
        eng.close()


# ------------------------------------------------------------------ GPU: faults that random weights would hide
BIG = 5


def make_standout(w, rows_of=(), gain=1.0):
    """Every sublayer norms what it reads, so a token cannot stand out by the size of its embedding.
    Instead: entry 0 of every embedding is zero except token BIG's, which is nothing else, and
    column 0 of the given projection rows is multiplied by `gain` — what token BIG (and only it)
    sends through those rows is that much larger than any other token's."""
    w["embed"][:, 0] = 0.0
    w["embed"][BIG] = 0.0
    w["embed"][BIG, 0] = 8.0
    for name, rows in rows_of:
        w[name][rows, 0] *= gain
    return w


def draw_latent_queries_to_big(w, p, m):
    """One score stands out: entry 1 of every embedding but BIG's is the same large number and leads the
    query latents, BIG's key latent points along entry 0 (a latent is normed over its row, so it can stand
    out by direction only), and the two meet in W_uq and W_uk: wherever BIG is visible the softmax is its."""
    w["embed"][:, 1] = 4.0
    w["embed"][BIG, 1] = 0.0
    w[p + "dq"][0] = 0.0
    w[p + "dq"][0, 1] = 4.0
    w[p + "dkv"][1:m["kv_rank"], 0] = 0.0
    w[p + "dkv"][0] = 0.0
    w[p + "dkv"][0, 0] = 4.0
    H, d, r = m["heads"], m["dim"], m["rot_dim"]
    uq = w[p + "uq"].reshape(H, d + r, -1)[:, :d, 0]
    gain = 24.0 / (m["scale"] * np.sqrt(m["q_rank"] * m["kv_rank"]) * (uq * uq).sum(axis=1, keepdims=True))
    w[p + "uk"].reshape(H, d, -1)[:, :, 0] = W.bf16_round((uq * gain).astype(np.float32))
    w[p + "o"] *= 4.0


def draw_map_to_big(w, p, m, which):
    """The same for one of the two score maps: its queries all point along one vector (entry 1 of every
    embedding but BIG's leads them), BIG's key points along it too, other keys do not."""
    w["embed"][:, 1] = 4.0
    w["embed"][BIG, 1] = 0.0
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    u = W.bf16_round(np.random.default_rng(3).choice([-1.0, 1.0], (G, d)).astype(np.float32))
    q = w[p + "q"].reshape(H, 2, d, -1)
    k = w[p + "k"].reshape(G, 2, d, -1)
    q[:, which, :, 1] = np.repeat(u, H // G, axis=0) * 2.0
    k[:, :, :, 1] = 0.0
    k[:, which, :, 0] = u
    w[p + "q.norm"][:] = 1.0
    w[p + "k.norm"][:] = 1.0
    w[p + "v"][:, 0] *= 3.0
    w[p + "v"][:, 1] *= 0.3


def without(toks, t=BIG, other=6):
    return [other if x == t else x for x in toks]


@gpu
@pytest.mark.parametrize("prec,sizes", [(C.PREC_FP32, (12, 20)), (C.PREC_BF16, (12, 20)), (C.PREC_BF16, (32, 64)), (C.PREC_BF16, (16, 32))])
@pytest.mark.parametrize("size", [1, 2, 31, 32, 33, 64, 65, 127, 128, 129, 256, 257, 300])
def test_a_key_just_inside_and_just_outside_the_window(size, prec, sizes):
    """One attention layer.  The key of one token outweighs all others in one of the two maps wherever it
    is seen: position p0 + size - 1 still sees the token at p0, p0 + size does not.  Both sides of the
    edge in a prompt's portions (windows' ends on tile and page borders and beside them) and in decoding."""
    d, v = sizes
    j = model([layer(att(heads=4, kv_heads=2, dim=d, vdim=v, size=size, scale=14.0 / d))], width=64)
    for which in (0, 1):
        cfg, w = random_weights(j, 14, bf16=prec == C.PREC_BF16)
        make_standout(w)
        draw_map_to_big(w, "l0.mix.", j["layers"][0]["mixer"], which)
        n, p0 = size + 80, 37
        base = without(prompt(j, n, 15))
        far = list(base)
        far[p0] = BIG
        want, plain = ref.forward(j, w, far), ref.forward(j, w, base)
        moved = np.abs(want - plain).max(axis=1) / np.abs(plain).max()
        e = p0 + size
        # the test's own premise: inside the window it shows, outside it does not
        assert moved[p0:e].min() > 0.1 and moved[e:].max() < 1e-12
        eng = Engine(cfg, w, prec)
        try:
            got, pos = [], 0
            for c in (e - 2, 5, n - e - 3):
                out, _ = eng.step([("f", far[pos:pos + c], list(range(c)))])
                got.append(out)
                pos += c
            check(np.concatenate(got), want, prec, f"portions, map {which}")
            eng.step([("d", far[:e - 3], [])])
            dec = np.stack([eng.step([("d", [far[t]], [0])], decode=True)[0][0] for t in range(e - 3, e + 4)])
            check(dec, want[e - 3:e + 4], prec, f"decoded, map {which}")
        finally:
            eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
@pytest.mark.parametrize("at", [0, 3, 255, 256, 257])
def test_a_far_key_among_hundreds(at, prec):
    """Latent attention: one token's key wins the softmax over hundreds of others from hundreds of
    positions away, at and across page borders, in a prompt's portions and in decoding (where the keys are
    cut into ranges)."""
    d = 16 if prec == C.PREC_BF16 else 8
    j = model([layer(lat(heads=2, dim=d, rot_dim=d, vdim=16, kv_rank=2 * d, q_rank=16))], width=64)
    cfg, w = random_weights(j, 24, bf16=prec == C.PREC_BF16)
    make_standout(w)
    draw_latent_queries_to_big(w, "l0.mix.", j["layers"][0]["mixer"])
    n = 720
    base = without(prompt(j, n, 15))
    far = list(base)
    far[at] = BIG
    plain, want = ref.forward(j, w, base), ref.forward(j, w, far)
    moved = np.abs(want - plain).max(axis=1) / np.abs(plain).max()
    assert moved[at:].min() > 0.1  # the test's own premise
    eng = Engine(cfg, w, prec)
    try:
        got, pos = [], 0
        for c in (250, 12, 430):
            out, _ = eng.step([("f", far[pos:pos + c], list(range(c)))])
            got.append(out)
            pos += c
        rows = [eng.step([("f", [far[t]], [0])], decode=True)[0][0] for t in range(pos, n)]
        check(np.concatenate(got + [np.stack(rows)]), want, prec, "far key")
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
def test_sinks_from_nothing_to_everything(prec):
    """Sinks far below, at and far above the scores: the first takes nothing, the last all of a head's
    weight; in a prompt, in decoding without and with key ranges."""
    kw = dict(kv_rank=32, rot_dim=16, q_rank=32) if prec == C.PREC_BF16 else {}
    j = model([layer(lat(heads=6, **kw))], width=64)
    cfg, w = random_weights(j, 25, bf16=prec == C.PREC_BF16)
    w["l0.mix.sink"][:] = [-200.0, -3.0, 1.0, 4.0, 6.0, 120.0]
    w["l0.mix.o"] *= 3.0
    toks = prompt(j, 420, 26)
    want = ref.forward(j, w, toks)
    none = dict(w, **{"l0.mix.sink": np.full(6, -1e3, dtype=np.float32)})
    assert np.abs(ref.forward(j, none, toks) - want).max() > 0.1 * np.abs(want).max()
    eng = Engine(cfg, w, prec)
    try:
        got, _ = eng.step([("a", toks[:400], list(range(400)))])
        rows = [eng.step([("a", [t], [0])], decode=True)[0][0] for t in toks[400:]]
        check(np.concatenate([got, np.stack(rows)]), want, prec, "long")
        eng.step([("b", toks[:1], [])])
        rows = [eng.step([("b", [t], [0])], decode=True)[0][0] for t in toks[1:30]]
        check(np.stack(rows), want[1:30], prec, "short")
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
def test_a_far_token_reaches_through_the_recurrent_state(prec):
    """mLSTM layers only, forget gates near one: nothing but the carried state links position 600 to
    position 2.  The prompt goes in portions and then decodes."""
    j = model([layer(ml(heads=2, dim=32, vdim=16, cap=15.0)), layer(ml(heads=4, dim=16, vdim=8, cap=15.0))], width=64)
    cfg, w = random_weights(j, 12, bf16=prec == C.PREC_BF16)
    for name in w:
        if name.endswith(".f.b"):
            w[name][:] = 12.0
        if name.endswith((".mix.i", ".mix.f")):
            w[name] *= 0.5
    make_standout(w, [("l0.mix.v", slice(None))], 300.0)
    eng = Engine(cfg, w, prec)
    try:
        toks = without(prompt(j, 640, 13), other=8)
        with_far = list(toks)
        with_far[2] = BIG
        want, plain = ref.forward(j, w, with_far), ref.forward(j, w, toks)
        assert np.abs(want[600:] - plain[600:]).max() > 0.1 * np.abs(want[600:]).max()  # the test's own premise
        got, pos = [], 0
        for n in (250, 12, 200, 138):
            out, _ = eng.step([("f", with_far[pos:pos + n], [n - 1])])
            got.append(out[0])
            pos += n
        for t in range(600, 640):
            got.append(eng.step([("f", [with_far[t]], [0])], decode=True)[0][0])
        check(np.stack(got), want[[249, 261, 461, 599] + list(range(600, 640))], prec, "far token")
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("i_bias,f_bias,cap", [(-9.0, 9.0, 12.0), (9.0, 9.0, 12.0), (-9.0, -9.0, 12.0), (40.0, -40.0, 50.0),
                                               (-40.0, 40.0, 50.0), (0.0, 0.0, 0.1)])
def test_gates_at_their_ends(i_bias, f_bias, cap):
    """Input gates of e^-9 and e^9 and far beyond, forget gates shut and open, per head from one end to
    zero, projections that swing them: the running maximum keeps every exponential in range, the
    normaliser is met on both sides of e^-m, and what decoding carries is what the prompt left."""
    j = model([layer(ml(heads=4, dim=8, vdim=8, cap=cap)), layer(ml(heads=2, dim=8, vdim=8, cap=cap))], width=64)
    cfg, w = random_weights(j, 26)
    w["l0.mix.i.b"][:] = np.linspace(i_bias, 0.0, 4)
    w["l0.mix.f.b"][:] = np.linspace(f_bias, 0.0, 4)
    w["l1.mix.i.b"][:] = i_bias
    w["l1.mix.f.b"][:] = f_bias
    for n in ("l0.mix.i", "l0.mix.f"):
        w[n] *= 4.0
    eng = Engine(cfg, w, C.PREC_FP32)
    try:
        toks = prompt(j, 340, 27)
        want = ref.forward(j, w, toks)
        got, pos = [], 0
        for n in (1, 259, 60):  # (259: more than one round of 256 tokens in the gates' scan)
            got.append(eng.step([("a", toks[pos:pos + n], list(range(n)))])[0])
            pos += n
        rows = [eng.step([("a", [t], [0])], decode=True)[0][0] for t in toks[pos:]]
        check(np.concatenate(got + [np.stack(rows)]), want, C.PREC_FP32, "gates")
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
@pytest.mark.parametrize("favour", ["some", "identity", "real"])
def test_the_correction_chooses_but_does_not_weigh(favour, prec):
    """One layer whose corrections decide the choice: two real and one identity expert, identity experts
    only (no expert GEMM has a row), or real ones only; the weights are the uncorrected scores."""
    j = model([layer(ml(), moe(ff=24, experts=9, top=3, identity=4, shared=16))], width=64)
    cfg, w = random_weights(j, 20, bf16=prec == C.PREC_BF16)
    up = {"some": [2, 7, 11], "identity": [9, 10, 12], "real": [0, 4, 8]}[favour]
    w["l0.mlp.correction"][:] = 0.0
    w["l0.mlp.correction"][up] = 2.0
    toks = prompt(j, 120, 21)
    want = ref.forward(j, w, toks)
    w0 = dict(w, **{"l0.mlp.correction": np.zeros(13, dtype=np.float32)})
    assert np.abs(ref.forward(j, w0, toks) - want).max() > 0.05 * np.abs(want).max()
    eng = Engine(cfg, w, prec)
    try:
        got, _ = eng.step([("p", toks[:100], list(range(100)))])
        rows = [eng.step([("p", [t], [0])], decode=True)[0][0] for t in toks[100:]]
        check(np.concatenate([got, np.stack(rows)]), want, prec, "routing")
    finally:
        eng.close()


@gpu
def test_long_prompts_of_routed_tokens():
    """More (token, slot) pairs than the one-launch sort takes, identity pairs among them, and more than 64
    experts: the separate sort and gather."""
    for seed, m in ((1, moe(ff=16, experts=6, top=4, identity=5)), (2, moe(ff=16, experts=90, top=6, identity=10))):
        j = model([layer(ml(heads=1, dim=8, vdim=8), m)], width=64)
        for prec in PRECS:
            cfg, w, eng = setup(j, prec, seed=80 + seed, num_blocks=8)
            try:
                toks = prompt(j, 1100, 81 + seed)
                got, _ = eng.step([("p", toks, list(range(1100)))])
                check(got, ref.forward(j, w, toks), prec, "routing", True)
            finally:
                eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
@pytest.mark.parametrize("n_seqs", [13, 20])
def test_decoding_many_sequences_with_keys_cut_into_ranges(n_seqs, prec):
    """Sequences of 1200 down to 1 tokens decoding together (more than eight rows: the batch GEMMs; more than
    sixteen: the values are expanded apart from the merge of the key ranges), windows of 40 and 900: the
    tiles of a wide window are shared out to several CTAs, some of which find no key."""
    kw = dict(dim=16, rot_dim=16, vdim=16, kv_rank=64, q_rank=32)
    j = model([layer(lat(heads=8, **kw), dense(ff=64)), layer(ml(heads=2, dim=16, vdim=32), moe(experts=3, top=4, identity=1)),
               layer(att(heads=4, kv_heads=2, dim=32, vdim=64, size=900), dense(ff=64)), layer(att(heads=4, kv_heads=4, dim=32, vdim=32, size=40))],
              width=64, loop=(0, 3, 2))
    cfg, w, eng = setup(j, prec, seed=31, num_blocks=40, slots=n_seqs)
    try:
        sizes = (1200, 300, 255, 256, 129, 64, 63, 41, 40, 9, 3, 2, 1, 400, 20, 21, 22, 23, 24, 25)[:n_seqs]
        lens = {f"s{i}": n for i, n in enumerate(sizes)}
        toks = {k: prompt(j, n + 5, 32 + i) for i, (k, n) in enumerate(lens.items())}
        want = {k: ref.forward(j, w, t) for k, t in toks.items()}
        eng.step([(k, toks[k][:n], []) for k, n in lens.items()])
        rows = {k: [] for k in lens}
        for t in range(5):
            out, _ = eng.step([(k, [toks[k][n + t]], [0]) for k, n in lens.items()], decode=True)
            for i, k in enumerate(lens):
                rows[k].append(out[i])
        for k, n in lens.items():
            check(np.stack(rows[k]), want[k][n:], prec, f"sequence of {n}")
    finally:
        eng.close()


# ------------------------------------------------------------------ GPU: models drawn at random
def draw_model(rng):
    """Sizes, head counts, layer order, windows, constants, feed-forwards and the repeated run are drawn."""
    layers = []
    tc = rng.random() < 0.5  # sizes that the tensor-core kernels take in bf16
    for i in range(int(rng.integers(2, 7))):
        kind = rng.choice(["ml", "lat", "att"])
        if kind == "ml":
            mix = ml(heads=int(rng.integers(1, 7)), dim=int(rng.choice([4, 10, 16, 32, 64, 100, 128])),
                     vdim=int(rng.choice([4, 9, 16, 32, 64, 128, 140])), cap=float(rng.choice([1.0, 8.0, 15.0])))
        elif kind == "lat":
            rank = int(rng.integers(1, 9)) * (16 if tc else int(rng.choice([4, 8, 11])))
            rot = int(rng.choice([16, 32])) if tc else int(rng.integers(1, 9)) * 2
            dim = int(rng.integers(1, 5)) * (8 if tc else 5)
            mix = lat(heads=int(rng.integers(1, 11)), dim=dim, rot_dim=rot, vdim=int(rng.integers(1, 7)) * int(rng.choice([8, 3])), kv_rank=rank,
                      q_rank=int(rng.integers(1, 9)) * 8, base=float(rng.choice([30.0, 1000.0, 20000.0])), factor=float(rng.choice([1.0, 2.5, 40.0])),
                      original=int(rng.choice([16, 100, 4096])), fast=float(rng.choice([2.0, 32.0])), slow=float(rng.choice([0.5, 1.0])),
                      scale=float((dim + rot) ** -0.5 * rng.uniform(0.5, 2)))
        else:
            g = int(rng.integers(1, 4))
            dim, vdim = ((32, 32), (32, 64), (64, 64), (64, 128))[rng.integers(4)] if tc else (int(rng.integers(1, 40)), int(rng.integers(1, 50)))
            mix = att(heads=g * int(rng.integers(1, 6)), kv_heads=g, dim=dim, vdim=vdim, diff=float(rng.uniform(0.1, 0.9)),
                      size=int(rng.choice([1, 2, 7, 31, 32, 33, 64, 65, 100, 128, 200, 256, 500])), scale=float(dim ** -0.5 * rng.uniform(0.5, 2)))
        r = rng.random()
        mlp = None
        if r < 0.35:
            mlp = dense(ff=int(rng.integers(4, 200)))
        elif r < 0.85:
            e, idn = int(rng.integers(1, 14)), int(rng.integers(0, 6))
            mlp = moe(ff=int(rng.integers(4, 100)), experts=e, identity=idn, top=int(rng.integers(1, min(5, e + idn) + 1)), shared=int(rng.choice([7, 16, 50])))
        layers.append(layer(mix, mlp))
    n = len(layers)
    a = int(rng.integers(0, n))
    loop = (a, int(rng.integers(a + 1, n + 1)), int(rng.integers(1, 4))) if rng.random() < 0.8 else None
    return model(layers, vocab=int(rng.integers(50, 500)), width=int(rng.choice([64, 96, 128, 192, 256])),
                 eps=float(rng.choice([1e-5, 1e-6, 1e-4])), loop=loop)


def replay_drawn(j, prec, seed, rng):
    """Whole prompt, then the same tokens in drawn portions with the last ones decoded, beside a
    second request that comes and goes; every row."""
    cfg, w, eng = setup(j, prec, seed=50 + seed)
    try:
        n = int(rng.integers(30, 330))
        toks, other = prompt(j, n, 60 + seed), prompt(j, int(rng.integers(3, 120)), 70 + seed)
        want, want_o = ref.forward(j, w, toks), ref.forward(j, w, other)
        got, _ = eng.step([("w", toks, list(range(n)))])
        check(got, want, prec, "whole prompt", True)
        eng.end("w")
        rows, pos, po, ndec = [], 0, 0, int(rng.integers(1, 9))
        while pos < n - ndec:
            c = int(min(n - ndec - pos, rng.choice([2, 2, 3, 5, 17, 64, 100, 130])))
            entries = [("p", toks[pos:pos + c], list(range(c)))]
            if po < len(other):
                co = int(min(len(other) - po, rng.choice([1, 2, 9, 40])))
                entries.append(("o", other[po:po + co], [co - 1]))
            out, _ = eng.step(entries)
            rows.append(out[:c])
            if len(entries) > 1:
                check(out[c:], want_o[po + co - 1:po + co], prec, "second request", True)
                po += co
                if po >= len(other):
                    eng.end("o")
            pos += c
        for t in range(pos, n):
            rows.append(eng.step([("p", [toks[t]], [0])], decode=True)[0])
        check(np.concatenate(rows), want, prec, "portions and decoding", True)
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("seed", range(10))
def test_models_drawn_at_random(seed):
    rng = np.random.default_rng(6000 + seed)
    replay_drawn(draw_model(rng), C.PREC_FP32, seed, rng)


# ------------------------------------------------------------------ GPU: entry points
@gpu
def test_greedy_generation_through_the_engine_and_its_scheduler():
    """LLMEngine.generate: the scheduler admits the prompts, the block manager hands out pages
    and state slots, Run() samples greedily; three requests of unequal length at once."""
    R = nvllm_pkg.sub("runner")
    j = mixed_model()
    cfg, w = random_weights(j, 21)
    run = R.CudaModelRunner(cfg, w.items(), precision=C.PREC_FP32, num_kv_blocks=12, sampling=None, num_state_slots=8)
    eng = E.LLMEngine(E.EngineConfig(max_num_seqs=8, num_kvcache_blocks=12, max_model_len=4096), run)
    try:
        prompts = [prompt(j, n, 50 + n) for n in (5, 61, 250)]
        outs = eng.generate(prompts, E.SamplingParams(temperature=1.0, max_tokens=12, ignore_eos=True), temperature=0.0)
        for p, o in zip(prompts, outs):
            assert o == ref.greedy(j, w, p, 12)
        assert len(eng.scheduler.block_manager.free_state_slots) == 8
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_command_line_on_a_model_directory(tmp_path, dtype):
    """bin/trace_run: config.json + model.safetensors (bf16) in, logits of the wanted places out."""
    prec = C.PREC_FP32 if dtype == "float32" else C.PREC_BF16
    j = no_close_calls(mixed_model(), prec)
    cfg, w = random_weights(j, 22, bf16=True)
    mdir, out = tmp_path / "model", tmp_path / "out"
    mdir.mkdir()
    (mdir / "config.json").write_text(json.dumps(j))
    write_safetensors(str(mdir / "model.safetensors"), w, dtype="BF16")
    a, b = prompt(j, 80, 60), prompt(j, 9, 61)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [49]}, {"id": "b", "tokens": b, "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:], "want": [29]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [7], "want": [0]}, {"id": "c", "tokens": b[:4], "want": [3]}], "end": ["a", "c"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(mdir), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                       text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb, wa2 = ref.forward(j, w, a), ref.forward(j, w, b), ref.forward(j, w, a + [7])
    got = np.concatenate([np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, j["vocab"]) for s in (0, 1, 2)])
    check(got, np.stack([wa[49], wb[0], wb[8], wa[79], wa2[80], wb[3]]), prec, "three steps", True)


@gpu
def test_sizes_the_kernels_do_not_cover_are_refused_at_create():
    L = nvllm_pkg.sub("lib")
    R = nvllm_pkg.sub("runner")
    for bad in ([layer(ml(heads=1, dim=300, vdim=8))],
                [layer(lat(kv_rank=513))],
                [layer(att(heads=5, kv_heads=2))],
                [layer(att(vdim=600))],
                [layer(ml(cap=0.0))],
                [layer(ml(), moe(experts=250, identity=7))]):
        cfg, w = random_weights(model(bad), 1)
        with pytest.raises(L.NvllmError):
            R.CudaModelRunner(cfg, w.items(), precision=C.PREC_FP32, num_kv_blocks=2, sampling=None, num_state_slots=1)
