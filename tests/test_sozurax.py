"""Sozurax (layers listed in config.json: HGRN2 recurrences, latent attention over a sliding window
with neighbouring pairs rotated and borrowed cache rows; LayerNorms with weight and additive term, a
short convolution added to what every mixer and feed-forward reads, PolyNorm dense layers, softmax-
routed gated experts with a router bias and a plain always-on expert) against the plain float64
restatement in tests/sozurax_ref.py.  Every test makes its own small configuration and random weights."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

from helpers import C, E, W, ROOT
import nvllm_pkg
import sozurax_ref as ref
from st_writer import write_safetensors
from test_zozonex import Engine, prompt
from test_lazovik import check

gpu = pytest.mark.gpu
BLOCK = C.KV_BLOCK_SIZE
PRECS = [C.PREC_FP32, C.PREC_BF16]


# ------------------------------------------------------------------ configurations
def hg(heads=3, dim=16, vdim=20):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def lat(heads=4, dim=16, rot_dim=8, vdim=12, kv_rank=24, q_rank=40, size=21, base=500.0, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "rot": {"base": base, "dims": rot_dim}, "mask": {"size": size},
         "scale": float((dim + rot_dim) ** -0.5 if scale is None else scale)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=7, top=2, shared=36):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mix, mlp=None):
    return dict(copy.deepcopy(mix), mlp=mlp)


def model(layers, vocab=211, width=72, eps=1e-5, taps=3, emb=2.5):
    return {"architecture": "Sozurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": emb}, "layers": layers}


def mixed_model():
    """Both mixers, every kind of feed-forward and none, own and borrowed cache rows (two borrowers of
    one layer with windows, head counts and value sizes of their own), sizes that differ layer to layer."""
    return model([layer(lat(), dense()),
                  layer(hg(), moe()),
                  layer(lat(heads=6, dim=8, vdim=20, q_rank=12, size=50, kv_from=0), moe(experts=5, top=1, shared=0)),
                  layer(hg(heads=2, dim=24, vdim=8)),
                  layer(lat(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=16, q_rank=16, size=3, base=30.0), moe(ff=40, top=4)),
                  layer(lat(heads=3, dim=20, vdim=16, q_rank=20, size=300, kv_from=0), dense(ff=100))])


def odd_model():
    """Sizes that are multiples of nothing convenient, windows of one and two tokens, six taps, one
    head, one expert, all experts, a layer without feed-forward first."""
    return model([layer(lat(heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=9, q_rank=11, size=1)),
                  layer(hg(heads=5, dim=6, vdim=10), moe(ff=20, experts=3, top=3, shared=12)),
                  layer(lat(heads=1, dim=10, rot_dim=2, vdim=30, kv_rank=13, q_rank=7, size=2), dense(ff=33)),
                  layer(hg(heads=1, dim=37, vdim=41), moe(ff=9, experts=1, top=1, shared=5))],
                 vocab=101, width=40, eps=3e-4, taps=6, emb=0.7)


def mma_model():
    """Row sizes that take the tensor-core latent kernels in bf16 (compile-time and run-time row
    sizes, 16 / 32 / 64 / 128 rows per CTA), recurrences at sizes of a real model's heads."""
    return model([layer(lat(heads=8, dim=32, rot_dim=16, vdim=32, kv_rank=64, q_rank=64, size=70), moe(ff=64, experts=8, shared=64)),
                  layer(hg(heads=4, dim=64, vdim=128), dense(ff=256)),
                  layer(lat(heads=16, dim=32, rot_dim=64, vdim=64, kv_rank=128, q_rank=96, size=128), moe(ff=96, experts=4, top=1)),
                  layer(lat(heads=12, dim=16, rot_dim=16, vdim=16, kv_rank=64, q_rank=40, size=200, kv_from=0)),
                  layer(hg(heads=2, dim=128, vdim=64), moe(ff=64, experts=8, top=3, shared=128)),
                  layer(lat(heads=20, dim=16, rot_dim=32, vdim=24, kv_rank=80, q_rank=64, size=33), dense(ff=136))],
                 width=128, taps=4)


def random_weights(j, seed, bf16=False):
    cfg = C.sozurax_from_json(j)
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in cfg.tensor_shapes().items():
        if name.endswith((".canon1", ".canon2")):
            a = 0.7 * rng.standard_normal(shape) / np.sqrt(shape[1])
        elif name.endswith(".lower"):
            a = rng.uniform(0.0, 0.9, shape)
        elif name.endswith(".f.b"):
            a = rng.uniform(-1.0, 3.0, shape)     # with the lower bound: gates from 0.2 to 0.99
        elif name.endswith(".router.b"):
            a = 1.5 * rng.standard_normal(shape)  # as large as the logits: without it other experts are chosen
        elif name.endswith(".act"):
            a = rng.uniform(0.3, 0.9, shape) * rng.choice([-1.0, 1.0], shape)
        elif name.endswith((".norm1.b", ".norm2.b")) or name == "final.norm.b":
            a = 0.4 * rng.standard_normal(shape)
        elif len(shape) == 1:
            a = 1.0 + 0.2 * rng.standard_normal(shape)  # norm weights
        elif name == "embed":
            a = rng.standard_normal(shape) + 0.5 * rng.standard_normal((1, shape[1]))  # rows with a mean: LayerNorm takes it off
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
    """With random weights, some token in a few hundred has two router logits closer than bf16
    rounding, and a run that then picks the other expert is not comparable from that token on.  The
    bf16 runs of models with several layers therefore use ALL experts of a layer (the logits still
    weight them); the choice is tested in fp32 and, in bf16, on single layers."""
    if prec == C.PREC_FP32:
        return j
    j = copy.deepcopy(j)
    for lc in j["layers"]:
        if lc.get("mlp") and lc["mlp"]["kind"] == "moe":
            lc["mlp"]["router"]["top"] = lc["mlp"]["router"]["experts"]
    return j


def routed(j):
    return any(lc.get("mlp") and lc["mlp"]["kind"] == "moe" for lc in j["layers"])


# ------------------------------------------------------------------ CPU: configuration, the restatement itself
def test_config_reader_takes_every_size_and_constant_from_the_file():
    j = mixed_model()
    cfg = C.ARCHITECTURES[j["architecture"]](j)
    assert cfg.arch == C.ARCH_SOZURAX and not cfg.tied_head and cfg.needs_state_slots and cfg.layer_norm
    assert cfg.block_style == C.LBLOCK_SEQUENTIAL_PRENORM
    assert (cfg.mixer_conv, cfg.ffn_conv, cfg.embedding_scale, cfg.vocab_size, cfg.hidden) == (3, 3, 2.5, 211, 72)
    a0, h1, a2, h3, a4, a5 = cfg.layers
    assert [l.mixer for l in cfg.layers] == [C.MIXER_LATENT_ATTENTION, C.MIXER_HGRN2, C.MIXER_LATENT_ATTENTION, C.MIXER_HGRN2,
                                             C.MIXER_LATENT_ATTENTION, C.MIXER_LATENT_ATTENTION]
    assert (a0.heads, a0.dim, a0.rot_dim, a0.vdim, a0.kv_rank, a0.q_rank, a0.window, a0.rot_pairs, a0.head_gate) == (4, 16, 8, 12, 24, 40, 21, 1, 0)
    assert (a0.rot_base, a0.rot_dims, a0.kv_from) == (500.0, 8, -1) and abs(a0.scale - 24 ** -0.5) < 1e-12
    assert (a2.kv_from, a2.window, a2.heads) == (0, 50, 6) and (a4.kv_from, a4.window, a4.rot_base) == (-1, 3, 30.0) and a5.window == 300
    assert (h1.heads, h1.dim, h1.vdim, h3.dim, h3.vdim) == (3, 16, 20, 24, 8)
    assert (a0.mlp, a0.act, a0.ff) == (C.MLP_DENSE, C.FFN_POLYNORM, 56) and h3.mlp == C.MLP_NONE
    assert (h1.mlp, h1.act, h1.ff, h1.experts, h1.top, h1.shared_ff, h1.route_bias, h1.route_norm, h1.route_sigmoid) == \
        (C.MLP_MOE, C.FFN_SWIGLU, 24, 7, 2, 36, 1, 1, 0)
    assert (a2.experts, a2.top, a2.shared_ff) == (5, 1, 0)
    sh = cfg.tensor_shapes()
    assert sh["head"] == (211, 72) and sh["final.norm.b"] == (72,) and sh["l3.canon1"] == (72, 3) and sh["l1.canon2"] == (72, 3)
    assert "l3.canon2" not in sh and "l3.norm2" not in sh and "l3.norm2.b" not in sh and sh["l3.norm1.b"] == (72,)
    assert sh["l0.mix.dkv"] == (32, 72) and "l2.mix.dkv" not in sh and "l2.mix.dkv.norm" not in sh and "l0.mix.g" not in sh
    assert sh["l2.mix.uq"] == (6 * 16, 12) and sh["l2.mix.uv"] == (120, 24) and sh["l1.mix.lower"] == (48,) and sh["l1.mix.f.b"] == (48,)
    assert sh["l0.mlp.act"] == (4,) and sh["l1.mlp.router.b"] == (7,) and sh["l1.mlp.shared.down"] == (72, 36) and "l2.mlp.shared.up" not in sh
    c, specs = cfg.to_c(C.PREC_FP32, num_state_slots=3)
    assert (c.mixer_conv, c.ffn_conv, c.layer_norm, c.num_state_slots) == (3, 3, 1, 3)
    assert specs[2].kv_from == 0 and specs[1].route_bias == 1 and specs[4].window == 3
    # a latent cache of (24 + 8) + (16 + 4) entries per token; states and two tails per layer with a feed-forward
    assert cfg.cache_bytes_per_token(2) == 2 * (32 + 20)
    assert cfg.state_bytes_per_sequence() == 4 * (3 * 16 * 20 + 2 * 24 * 8 + (6 + 5) * 2 * 72)
    # one tap: the sublayer reads h (1 + w), nothing is kept
    one = C.sozurax_from_json(model([layer(lat(), dense())], taps=1))
    assert not one.needs_state_slots and one.tensor_shapes()["l0.canon2"] == (72, 1)
    with pytest.raises(ValueError):
        C.sozurax_from_json(model([dict(type="attention", mixer=lat()["mixer"], mlp=None)]))
    with pytest.raises(ValueError):
        C.sozurax_from_json(model([layer(hg(), {"kind": "glu", "ff": 8})]))


def test_reference_mechanisms_against_hand_computed_values():
    """The restatement itself, on inputs small enough to check by hand."""
    got = ref.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 10.0]), np.array([0.5, 0.0]), 0.0)
    assert np.allclose(got, [[-1.5, 10.0]])
    u = np.array([[1.0], [2.0], [4.0]])
    assert ref.causal_conv(u, np.array([[10.0, 1.0]])).ravel().tolist() == [1.0, 12.0, 24.0]
    # one state entry, gate 1/2 each step, values 4 then 0: S = 2 then 1, read with q = 3
    o = ref.gated_state_scan(np.full((2, 1), 3.0), np.full((2, 1), 0.5), np.array([[4.0], [0.0]]))
    assert o.ravel().tolist() == [6.0, 3.0]
    # rows of the state follow their own gate: a gate of 1 neither forgets nor writes
    o = ref.gated_state_scan(np.array([[1.0, 1.0]]), np.array([[1.0, 0.0]]), np.array([[7.0]]))
    assert o.ravel().tolist() == [7.0]
    r = ref.rotate_pairs(np.array([[[1.0, 0.0, 1.0, 0.0, 5.0]]] * 2), 4, 100.0, np.array([0.0, 1.0]))
    assert np.allclose(r[0, 0], [1, 0, 1, 0, 5]) and np.allclose(r[1, 0], [np.cos(1), np.sin(1), np.cos(0.1), np.sin(0.1), 5])
    p = ref.windowed_softmax(np.zeros((4, 4)), 2)
    assert np.allclose(p, [[1, 0, 0, 0], [.5, .5, 0, 0], [0, .5, .5, 0], [0, 0, .5, .5]])
    assert np.allclose(ref.windowed_softmax(np.zeros((3, 3)), 0)[2], 1 / 3)
    z = np.array([[1.0, -2.0]])
    got = ref.poly_norm(z, [1.0, 10.0, 100.0, 0.5], 0.0)
    n1, n2, n3 = np.sqrt(2.5), np.sqrt(8.5), np.sqrt(32.5)
    assert np.allclose(got, [[1 / n1 + 10 / n2 + 100 / n3 + 0.5, -2 / n1 + 40 / n2 - 800 / n3 + 0.5]])
    idx, p = ref.route(np.array([0.0, np.log(3.0), 5.0, 0.1]), 2)
    assert idx == [2, 1] and np.allclose(p, np.array([np.exp(5.0), 3.0]) / (np.exp(5.0) + 3.0))


# ------------------------------------------------------------------ GPU: each mechanism alone
BARE = dict(taps=1, emb=1.0)
CASES = {
    "hgrn2": lambda: model([layer(hg())], **BARE),
    "hgrn2_wide_state": lambda: model([layer(hg(heads=2, dim=200, vdim=48))], **BARE),
    "hgrn2_wide_values": lambda: model([layer(hg(heads=1, dim=12, vdim=300))], **BARE),
    "hgrn2_heads_of_64_by_128": lambda: model([layer(hg(heads=2, dim=64, vdim=128))], **dict(BARE, width=128)),
    "latent_window": lambda: model([layer(lat())], **BARE),
    "latent_window_of_one": lambda: model([layer(lat(size=1))], **BARE),
    "latent_window_past_the_prompt": lambda: model([layer(lat(size=1000))], **BARE),
    "latent_rank_64_rot_16": lambda: model([layer(lat(heads=8, kv_rank=64, rot_dim=16, q_rank=64, size=40))], **dict(BARE, width=128)),
    "latent_rank_128_rot_64": lambda: model([layer(lat(heads=8, dim=64, vdim=64, kv_rank=128, rot_dim=64, q_rank=64, size=65))], **dict(BARE, width=128)),
    "latent_rank_256_rot_32": lambda: model([layer(lat(heads=4, dim=32, vdim=64, kv_rank=256, rot_dim=32, q_rank=64, size=30))], **dict(BARE, width=128)),
    "latent_rank_320": lambda: model([layer(lat(heads=2, dim=32, vdim=64, kv_rank=320, rot_dim=32, q_rank=24, size=30))], **dict(BARE, width=64)),
    "latent_borrowed": lambda: model([layer(lat()), layer(lat(heads=5, vdim=8, q_rank=8, size=9, kv_from=0)), layer(lat(heads=1, size=64, kv_from=0))], **BARE),
    "poly_norm": lambda: model([layer(hg(), dense(ff=50))], **BARE),
    "poly_norm_wide": lambda: model([layer(hg(), dense(ff=1000))], **dict(BARE, width=128)),
    "experts": lambda: model([layer(hg(), moe(ff=20, experts=12, top=3, shared=0))], **BARE),
    "experts_one": lambda: model([layer(lat(), moe(ff=20, experts=9, top=1, shared=0))], **BARE),
    "experts_and_shared": lambda: model([layer(lat(), moe(ff=64, experts=6, top=2, shared=200))], **dict(BARE, width=128)),
    "input_convolutions": lambda: model([layer(hg(), dense()), layer(lat())], taps=5),
    "input_convolutions_two_taps": lambda: model([layer(hg(), moe()), layer(hg())], taps=2),
    "input_convolutions_eight_taps": lambda: model([layer(lat(), moe())], taps=8, width=2056),
    "embedding_scale": lambda: model([layer(hg())], taps=2, emb=0.03),
    "everything": lambda: model([layer(lat(), moe()), layer(hg(), dense()), layer(lat(kv_from=0), moe())]),
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
        j = dict(full, layers=full["layers"][:n])
        cfg = C.sozurax_from_json(j)
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
        # portions shorter than the convolutions, one token, one that crosses the page border at 256
        for n in [2, 3, 2, 16, 17, 40, 1, 5, 100, 2, 71, 2, 70]:
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
        for r in range(5):  # 5 pairs of requests through 2 slots and 3 pages; each leaves state, tails and cache rows behind
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
    """Positions 0, 1, 2: shorter than the convolutions, the windows and any tile; the convolutions
    read zeros before the start and the state begins at zero, whatever the slot held — for a
    first row inside a prompt and for a prompt of a single token."""
    j = no_close_calls(MODELS[which](), prec)
    cfg, w, eng = setup(j, prec)
    try:
        eng.step([("dirt", prompt(j, 40, 29), [])])  # leaves state, tails and rows in slot and page
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
        toks = prompt(j, 560, 40)
        want = ref.forward(j, w, toks)
        eng.step([("l", toks[:20], [])])
        rows = [eng.step([("l", [toks[t]], [0])], decode=True)[0][0] for t in range(20, 560)]
        check(np.stack(rows), want[20:], C.PREC_FP32, "540 decoded tokens")
    finally:
        eng.close()


# ------------------------------------------------------------------ GPU: faults that random weights would hide
BIG = 5


def make_standout(w, rows_of, gain):
    """Every sublayer norms what it reads, so a token cannot stand out by the size of its embedding.
    Instead: entry 0 of every embedding is zero except token BIG's, which is nothing else, and
    column 0 of the given projection rows is multiplied by `gain` — what token BIG (and only it)
    sends through those rows is that much larger than any other token's."""
    w["embed"][:, 0] = 0.0
    w["embed"][BIG] = 0.0
    w["embed"][BIG, 0] = 8.0
    for name in w:
        if name.endswith("norm1.b"):
            w[name][:] = 0.0
    for name, rows in rows_of:
        w[name][rows, 0] *= gain
    return w


def draw_every_query_to_big(w, p, m):
    """One score stands out: entry 1 of every embedding but BIG's is the same large number and leads the
    query latents, BIG's key latent points along entry 0 (a latent is normed over its row, so it can stand
    out by direction only), and the two meet in W_uq and W_uk: wherever BIG is visible the softmax is its."""
    w[p.replace("mix.", "canon1")][:2] = 0.0
    w["embed"][:, 1] = 4.0
    w["embed"][BIG, 1] = 0.0
    w[p + "dq"][0] = 0.0
    w[p + "dq"][0, 1] = 4.0
    if p + "dkv" in w:
        w[p + "dkv"][1:m["kv_rank"], 0] = 0.0
        w[p + "dkv"][0] = 0.0
        w[p + "dkv"][0, 0] = 4.0
    H, d, r = m["heads"], m["dim"], m["rot_dim"]
    uq = w[p + "uq"].reshape(H, d + r, -1)[:, :d, 0]
    gain = 24.0 / (m["scale"] * np.sqrt(m["q_rank"] * m["kv_rank"]) * (uq * uq).sum(axis=1, keepdims=True))
    w[p + "uk"].reshape(H, d, -1)[:, :, 0] = W.bf16_round((uq * gain).astype(np.float32))
    w[p + "o"] *= 4.0


def without(toks, t=BIG, other=6):
    return [other if x == t else x for x in toks]


@gpu
@pytest.mark.parametrize("prec", PRECS)
@pytest.mark.parametrize("size", [1, 2, 63, 64, 65, 127, 128, 129, 256, 257, 300])
def test_a_key_just_inside_and_just_outside_the_window(size, prec):
    """One attention layer.  The key of one token outweighs all others wherever it is seen: position
    p0 + size - 1 still sees the token at p0, p0 + size does not.  Both sides of the edge in a
    prompt's portions (windows' ends on tile and page borders and beside them) and in decoding."""
    kw = dict(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, q_rank=32) if prec == C.PREC_BF16 else {}
    j = model([layer(lat(size=size, **kw))], width=64, taps=1, emb=1.0)
    cfg, w = random_weights(j, 14, bf16=prec == C.PREC_BF16)
    make_standout(w, [], 1.0)
    draw_every_query_to_big(w, "l0.mix.", j["layers"][0]["mixer"])
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
        got, pos, rows = [], 0, []
        for c in (e - 2, 5, n - e - 3):
            out, _ = eng.step([("f", far[pos:pos + c], list(range(c)))])
            got.append(out)
            pos += c
        got = np.concatenate(got)
        check(got, want, prec, "portions")
        eng.step([("d", far[:e - 3], [])])
        dec = np.stack([eng.step([("d", [far[t]], [0])], decode=True)[0][0] for t in range(e - 3, e + 4)])
        check(dec, want[e - 3:e + 4], prec, "decoded")
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
def test_a_far_key_among_hundreds(prec):
    """A window of 700: one token's key wins the softmax over hundreds of others from hundreds of
    positions away, over page borders, in a prompt's portions and in decoding; a second layer that
    borrows the rows finds it too, with a window of its own."""
    d = 16 if prec == C.PREC_BF16 else 8
    a = lat(heads=2, dim=d, rot_dim=d, vdim=16, kv_rank=2 * d, q_rank=16, size=700)
    b = lat(heads=3, dim=d, rot_dim=d, vdim=8, kv_rank=2 * d, q_rank=24, size=640, kv_from=0)
    j = model([layer(a), layer(b)], width=64, taps=2, emb=1.0)
    cfg, w = random_weights(j, 24, bf16=prec == C.PREC_BF16)
    make_standout(w, [], 1.0)
    for k in (0, 1):
        draw_every_query_to_big(w, f"l{k}.mix.", j["layers"][k]["mixer"])
    n = 720
    base = without(prompt(j, n, 15))
    far = list(base)
    far[3] = BIG
    plain, want = ref.forward(j, w, base), ref.forward(j, w, far)
    # the test's own premise
    moved = np.abs(want - plain).max(axis=1) / np.abs(plain).max()
    assert moved[500:640].min() > 0.1 and moved[644:700].min() > 0.05
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
def test_a_far_token_reaches_through_the_recurrent_state(prec):
    """HGRN2 layers only, gates near one: nothing but the carried state links position 600 to
    position 2.  The prompt goes in portions and then decodes."""
    j = model([layer(hg(heads=2, dim=32, vdim=16)), layer(hg(heads=4, dim=16, vdim=8))], width=64, taps=2, emb=1.0)
    cfg, w = random_weights(j, 12, bf16=prec == C.PREC_BF16)
    for name in w:
        if name.endswith(".lower"):
            w[name][:] = 0.99609375
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
def test_gates_at_their_ends():
    """Gates within 1e-9 of one (what is written must not be lost to 1 - f in fp32), gates at a
    lower bound of zero, and projections large enough to saturate the sigmoid either way."""
    j = model([layer(hg(heads=2, dim=8, vdim=8)), layer(hg(heads=2, dim=8, vdim=8))], width=64, taps=1, emb=1.0)
    cfg, w = random_weights(j, 26)
    w["l0.mix.f.b"][:] = 19.0
    w["l0.mix.lower"][:] = 0.0
    w["l1.mix.f.b"][:] = np.linspace(-60.0, 60.0, 16)
    w["l1.mix.lower"][:8] = 0.0
    eng = Engine(cfg, w, C.PREC_FP32)
    try:
        toks = prompt(j, 60, 27)
        got, _ = eng.step([("a", toks[:40], list(range(40)))])
        rows = [eng.step([("a", [t], [0])], decode=True)[0][0] for t in toks[40:]]
        check(np.concatenate([got, np.stack(rows)]), ref.forward(j, w, toks), C.PREC_FP32, "gates")
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
def test_the_router_bias_chooses_and_weighs(prec):
    """One layer whose router biases are larger than its logits: a choice without them, or weights
    from the logits alone, gives other logits; experts whose bias is far below never join."""
    j = model([layer(hg(), moe(ff=24, experts=12, top=3, shared=16))], taps=4, emb=1.0)
    cfg, w = random_weights(j, 20, bf16=prec == C.PREC_BF16)
    w["l0.mlp.router.b"][:] = np.array([0, 20, 17.5, 0, 18, 0, 0, 19, 0, 0, 18.5, 0], dtype=np.float32)
    toks = prompt(j, 120, 21)
    want = ref.forward(j, w, toks)
    w0 = dict(w)
    w0["l0.mlp.router.b"] = np.zeros(12, dtype=np.float32)
    assert np.abs(ref.forward(j, w0, toks) - want).max() > 0.05 * np.abs(want).max()
    eng = Engine(cfg, w, prec)
    try:
        got, _ = eng.step([("p", toks[:100], list(range(100)))])
        rows = [eng.step([("p", [t], [0])], decode=True)[0][0] for t in toks[100:]]
        check(np.concatenate([got, np.stack(rows)]), want, prec, "routing", True)
    finally:
        eng.close()


@gpu
@pytest.mark.parametrize("prec", PRECS)
def test_decoding_many_sequences_with_keys_cut_into_ranges(prec):
    """Thirteen sequences of 900 down to 1 tokens decoding together (more than eight rows: the
    batch GEMMs), windows of 40 and 600: the tiles of a window are shared out to several CTAs, some
    of which find no key; two borrowers read the same rows."""
    kw = dict(dim=16, rot_dim=16, vdim=16, kv_rank=64, q_rank=32)
    j = model([layer(lat(heads=8, size=600, **kw), dense(ff=64)), layer(hg(heads=2, dim=16, vdim=32), moe(experts=4, top=4)),
               layer(lat(heads=4, size=40, **dict(kw, kv_from=0)), dense(ff=64)), layer(lat(heads=2, size=129, **dict(kw, kv_from=0)))],
              width=64, taps=4, emb=1.0)
    cfg, w, eng = setup(j, prec, seed=31, num_blocks=24, slots=13)
    try:
        lens = {f"s{i}": n for i, n in enumerate((900, 300, 255, 256, 129, 64, 63, 41, 40, 9, 3, 2, 1))}
        toks = {k: prompt(j, n + 6, 32 + i) for i, (k, n) in enumerate(lens.items())}
        want = {k: ref.forward(j, w, t) for k, t in toks.items()}
        eng.step([(k, toks[k][:n], []) for k, n in lens.items()])
        rows = {k: [] for k in lens}
        for t in range(6):
            out, _ = eng.step([(k, [toks[k][n + t]], [0]) for k, n in lens.items()], decode=True)
            for i, k in enumerate(lens):
                rows[k].append(out[i])
        for k, n in lens.items():
            check(np.stack(rows[k]), want[k][n:], prec, f"sequence of {n}")
    finally:
        eng.close()


# ------------------------------------------------------------------ GPU: models drawn at random
def draw_model(rng, tensor_cores=False):
    """Sizes, head counts, layer order, windows, constants and feed-forwards are drawn."""
    layers, own = [], []
    for i in range(int(rng.integers(2, 8))):
        if rng.random() < 0.45:
            mix = hg(heads=int(rng.integers(1, 7)), dim=int(rng.choice([4, 10, 16, 32, 64, 100, 128])), vdim=int(rng.choice([4, 9, 16, 32, 64, 128])))
        else:
            step = 16 if tensor_cores else 1
            src = int(rng.choice(own)) if own and rng.random() < 0.4 else None
            if src is None:
                rank, rot, base = int(rng.integers(1, 9)) * (16 if tensor_cores else int(rng.choice([4, 8, 11]))), \
                    int(rng.choice([16, 32]) if tensor_cores else rng.integers(1, 9) * 2), float(rng.choice([30.0, 1000.0, 20000.0]))
                own.append(i)
            else:
                m = layers[src]["mixer"]
                rank, rot, base = m["kv_rank"], m["rot_dim"], m["rot"]["base"]
            dim = int(rng.integers(1, 5)) * max(step // 2, 5 if not tensor_cores else 8)
            mix = lat(heads=int(rng.integers(1, 11)), dim=dim, rot_dim=rot, vdim=int(rng.integers(1, 7)) * 8, kv_rank=rank,
                      q_rank=int(rng.integers(1, 9)) * 8, size=int(rng.choice([1, 2, 7, 31, 32, 33, 64, 65, 100, 128, 200, 256, 500])),
                      base=base, scale=float((dim + rot) ** -0.5 * rng.uniform(0.5, 2)), kv_from=src)
        r = rng.random()
        mlp = None
        if r < 0.3:
            mlp = dense(ff=int(rng.integers(4, 200)))
        elif r < 0.85:
            e = int(rng.integers(1, 14))
            mlp = moe(ff=int(rng.integers(4, 100)), experts=e, top=int(rng.integers(1, min(4, e) + 1)), shared=int(rng.choice([0, 16, 50])))
        layers.append(layer(mix, mlp))
    return model(layers, vocab=int(rng.integers(50, 500)), width=int(rng.choice([64, 96, 128, 192, 256])),
                 eps=float(rng.choice([1e-5, 1e-6, 1e-4])), taps=int(rng.choice([1, 2, 3, 4, 6])), emb=float(rng.choice([0.5, 1.0, 12.0])))


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
@pytest.mark.parametrize("seed", range(8))
def test_models_drawn_at_random(seed):
    rng = np.random.default_rng(6000 + seed)
    replay_drawn(draw_model(rng, tensor_cores=seed % 2 == 1), C.PREC_FP32, seed, rng)


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
    for bad in ([layer(hg(heads=1, dim=300, vdim=8))],
                [layer(lat(kv_rank=513))],
                [layer(lat()), layer(lat(kv_rank=32, kv_from=0))],      # rows of another size cannot be borrowed
                [layer(hg()), layer(lat(kv_from=0))]):                  # that layer has no rows
        cfg, w = random_weights(model(bad), 1)
        with pytest.raises(L.NvllmError):
            R.CudaModelRunner(cfg, w.items(), precision=C.PREC_FP32, num_kv_blocks=2, sampling=None, num_state_slots=1)
