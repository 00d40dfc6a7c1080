"""The Bafilorn configuration, its model description, the residual of several streams as parts, and the plain implementation's
own mechanisms checked against what they must equal (no GPU)."""
import copy
import math

import pytest
import torch

from odin_infer_b200.cache import CacheManager
from odin_infer_b200.config import BafilornConfig, ConfigError, config_from_dict, lookup_architecture
from odin_infer_b200.engine.model import DecoderModel
from odin_infer_b200.parts.base import Biased, PartSpec, Streamed, build_part, split_update
from odin_infer_b200.parts.norm import terms_of
from tests.plain import bafilorn_plain as P

F64 = torch.float64
LATENT = {"heads": 3, "dim": 20, "rot_dim": 12, "vdim": 28, "q_rank": 24, "kv_rank": 36, "scale": 0.2, "rot": {"dims": 12, "base": 700.0}}
LIGHTNING = {"heads": 2, "dim": 16, "vdim": 24, "decay": [0.75, 0.99]}
PARALLEL = {"left": {"heads": 6, "kv_heads": 3, "dim": 20, "vdim": 20, "scale": 0.3, "mask": {"size": 50},
                     "rot": {"dims": 12, "base": 900.0, "scaling": {"factor": 3.0, "original": 300.0, "fast": 8.0, "slow": 0.5}}},
            "right": {"width": 60, "blocks": 5, "conv": 3}}
RAW = {"architecture": "Bafilorn", "vocab": 151, "width": 72, "streams": 3, "norm": {"eps": 1e-5},
       "embedding": {"scale": 1.75, "bigram": {"buckets": 83, "mul_prev": 11, "mul_cur": 5}},
       "layers": [{"type": "parallel", "mixer": PARALLEL, "mlp": {"kind": "dense", "ff": 40}},
                  {"type": "lightning", "mixer": LIGHTNING, "mlp": None},
                  {"type": "latent_attention", "mixer": LATENT, "mlp": {"kind": "dense", "ff": 56}}],
       "loop": {"start": 0, "stop": 2, "times": 3}}


def test_configuration_reads_and_writes_the_same_keys():
    cfg = config_from_dict(RAW)
    assert isinstance(cfg, BafilornConfig) and cfg.to_dict() == RAW and config_from_dict(cfg.to_dict()) == cfg
    p, g, l = cfg.layers
    assert (p.heads, p.kv_heads, p.dim, p.chunk, p.rot_dims, p.ramp, p.inner, p.blocks, p.conv, p.ff) == (
        6, 3, 20, 50, 12, (3.0, 300.0, 8.0, 0.5), 60, 5, 3, 40)
    assert (g.heads, g.dim, g.vdim, g.decay, g.ff) == (2, 16, 24, (0.75, 0.99), 0)
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.scale, l.rot_base, l.ff) == (3, 20, 12, 28, 24, 36, 0.2, 700.0, 56)
    assert cfg.bigram == (83, 11, 5) and cfg.embedding_scale == 1.75 and cfg.streams == 3
    assert cfg.layer_runs() == [0, 1, 0, 1, 0, 1, 2] == P.schedule(RAW)


def test_absent_keys_mean_absent_mechanisms():
    raw = copy.deepcopy(RAW)
    del raw["loop"], raw["embedding"], raw["layers"][0]["mixer"]["left"]["rot"]["scaling"]
    cfg = config_from_dict(raw)
    spec = lookup_architecture("Bafilorn").build_spec(cfg)
    assert cfg.layer_runs() == [0, 1, 2] and spec.embedding.args["pair"] is None and spec.embedding.args["scale"] == 1.0
    assert all(e.args["ramp"] is None for e in spec.position_encodings.values())
    assert config_from_dict(cfg.to_dict()) == cfg
    raw["loop"] = {"start": 1, "stop": 2, "times": 1}
    assert config_from_dict(raw).layer_runs() == [0, 1, 2]
    raw["loop"] = {"start": 1, "stop": 3, "times": 2}
    assert config_from_dict(raw).layer_runs() == [0, 1, 2, 1, 2]


def test_every_fault_of_a_configuration_in_one_error():
    bad = copy.deepcopy(RAW)
    bad["streams"] = 0
    bad["loop"]["stop"] = 4
    bad["layers"][0]["mixer"]["left"]["kv_heads"] = 4
    bad["layers"][0]["mixer"]["left"]["vdim"] = 24
    bad["layers"][0]["mixer"]["right"]["blocks"] = 7
    bad["layers"][0]["mixer"]["left"]["rot"]["scaling"]["slow"] = 0
    bad["layers"][1]["mixer"]["decay"] = [0.5]
    bad["layers"][2]["mixer"]["rot"]["dims"] = 8
    del bad["layers"][2]["mixer"]["q_rank"]
    bad["layers"][2]["mlp"]["kind"] = "moe"
    with pytest.raises(ConfigError) as e:
        config_from_dict(bad)
    for part in ("'streams'", "stop 4", "multiple of kv_heads", "values are keys", "multiple of blocks", "slow", "list of 2 numbers",
                 "must be rot_dim", "'q_rank'", "'dense'"):
        assert part in str(e.value), (part, str(e.value))


def test_the_model_description_names_every_tensor_once():
    model = DecoderModel(lookup_architecture("Bafilorn").build_spec(config_from_dict(RAW)))
    names = [p.name for p in model.params()]
    assert len(names) == len(set(names))
    shapes = {p.name: p.shape for p in model.params() if not p.optional}
    for n, s in (("embed", (151, 72)), ("bigram", (84, 72)), ("l0.mix.left.q", (120, 72)), ("l0.mix.left.k", (60, 72)),
                 ("l0.mix.left.k.b", (60,)), ("l0.mix.left.g", (120, 72)), ("l0.mix.left.o", (72, 120)), ("l0.mix.left.o.b", (72,)),
                 ("l0.mix.right.y", (60, 72)), ("l0.mix.right.x.b", (60,)), ("l0.mix.right.conv", (60, 3)),
                 ("l0.mix.right.ra", (5, 12, 12)), ("l0.mix.right.ri.b", (5, 12)), ("l0.mix.right.lam", (60,)),
                 ("l0.mix.right.out", (72,)), ("l0.hc1.in", (3,)), ("l0.hc2.mix", (3, 3)), ("l1.mix.q", (32, 72)),
                 ("l1.mix.v", (48, 72)), ("l1.mix.norm", (48,)), ("l2.mix.dq", (24, 72)), ("l2.mix.uq", (96, 24)),
                 ("l2.mix.dkv", (48, 72)), ("l2.mix.dkv.norm", (36,)), ("l2.mix.uk", (60, 36)), ("l2.mix.uv", (84, 36)),
                 ("l2.mix.g", (84, 72)), ("l2.mlp.up", (56, 72)), ("final.norm", (72,)), ("head", (151, 72))):
        assert shapes.get(n) == s, (n, shapes.get(n))
    assert "l0.mix.left.v" not in shapes and "l0.mix.left.v.b" not in shapes
    # a layer without feed-forward reads no second norm and no second connection
    assert {p.name for p in model.params() if p.optional} == {f"l1.{n}" for n in ("norm2", "hc2.in", "hc2.out", "hc2.mix")}
    assert model.graph_safe
    cache = CacheManager(64 * 4, 64 * 2)
    model.register_cache(cache)
    unit, light = 4 * (60 + 2 * 60), 4 * 2 * 16 * 24
    assert cache.state_bytes_of == [unit, light] * 3 + [0, 4]      # every run of a layer has a state of its own; the token before
    kept = sorted((g.request.n_kv_heads, g.request.head_dim, g.request.chunk, g.n_lines, g.request.shared_kv) for g in cache.groups.values())
    assert kept == [(1, 48, 0, 1, True), (3, 20, 50, 3, False)]


def test_an_update_of_several_streams_passes_to_whoever_applies_it():
    hc = build_part("connection", PartSpec("hyper", dict(streams=2, mix="m", out="o")))
    hc.bind({"m": torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=torch.bfloat16), "o": torch.tensor([5.0, 6.0])}, None)
    u = hc.join("update")
    assert isinstance(u, Streamed) and u.update == "update" and u.mix.dtype == torch.float32 and u.mix[0, 1] == 2.0
    assert split_update(u) == (u, None)
    b = torch.ones(4)
    (term,) = terms_of(Biased(torch.zeros(3, 4), b))
    assert term.bias is b and term.scale == 1.0


def test_parts_refuse_what_they_cannot_do():
    names = {k: k for k in ("q", "k", "v", "g", "norm", "o")}
    mixer = PartSpec("lightning", dict(width=8, n_heads=1, head_dim=8, v_head_dim=8, decay=[0.5], names=names))
    one = PartSpec("rmsnorm", dict(width=8, eps=1e-5, weight="w"))
    several = PartSpec("streams_rmsnorm", dict(width=8, eps=1e-5, weight="w", streams=2, read="r"))
    hyper = PartSpec("hyper", dict(streams=2, mix="m", out="o"))
    with pytest.raises(TypeError):      # a norm of one stream where the residual is several
        build_part("block", PartSpec("prenorm", dict(mixer=mixer, feed_forward=None, norm_mixer=one, norm_feed_forward=None, connect_mixer=hyper)))
    with pytest.raises(ValueError):     # no norm on the output of a sublayer that joins several streams
        build_part("block", PartSpec("prenorm", dict(mixer=mixer, feed_forward=None, norm_mixer=several, norm_feed_forward=None,
                                                     connect_mixer=hyper, post_norm_mixer=one)))
    ffn = PartSpec("activated", dict(width=8, inner=8, activation="relu2", names={"up": "u", "down": "d"}))
    with pytest.raises(ValueError):     # both sublayers join the streams, or neither
        build_part("block", PartSpec("prenorm", dict(mixer=mixer, feed_forward=ffn, norm_mixer=several, norm_feed_forward=several, connect_mixer=hyper)))
    blk = build_part("block", PartSpec("prenorm", dict(mixer=mixer, feed_forward=None, norm_mixer=several, norm_feed_forward=None, connect_mixer=hyper)))
    with pytest.raises(TypeError):      # a norm of one stream after an update of several
        blk._norm(build_part("norm", one), None, None, Streamed("u", None, None))
    with pytest.raises(TypeError):      # and an update of one stream before a norm of several
        build_part("norm", several).forward(None, torch.zeros(2, 3, 8), torch.zeros(3, 8))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("lightning", dict(width=8, n_heads=2, head_dim=8, v_head_dim=8, decay=[0.5], names=names)))
    with pytest.raises(ValueError):
        build_part("mixer", PartSpec("gated_linear_unit", dict(width=8, inner=10, blocks=3, taps=2, names={})))
    att = dict(width=8, n_q_heads=1, n_kv_heads=1, head_dim=8, names={k: k for k in "qko"}, qk_norm=False, values_are_keys=True)
    with pytest.raises(ValueError):     # values that are the keys have their size
        build_part("mixer", PartSpec("gqa_attention", dict(att, v_head_dim=4)))
    with pytest.raises(ValueError):     # a learned sink or a fixed one
        build_part("mixer", PartSpec("gqa_attention", dict(att, sink="s", sink_logit=0.0)))
    with pytest.raises(ValueError):
        build_part("norm", PartSpec("streams_rmsnorm", dict(width=8, eps=1e-5, weight="w", streams=17)))


# ---- the plain implementation against what it must equal ------------------------------------------------------
def test_streams_by_hand():
    X = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)
    mix, out = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64), torch.tensor([0.5, -1.0], dtype=F64)
    new = P.hyper(X, mix, out, torch.tensor([[100.0]], dtype=F64))
    # stream 0: 1*1 + 3*10 + 50, stream 1: 2*1 + 4*10 - 100, both of the old ones
    assert new[:, 0, 0].tolist() == [81.0, -58.0]
    assert float(P.read_streams(X, torch.tensor([2.0, -1.0], dtype=F64))) == -8.0


def test_pair_rows_of_the_embedding():
    w = {"embed": torch.arange(10.0, dtype=F64)[:, None], "bigram": 100.0 * torch.arange(8.0, dtype=F64)[:, None]}
    cfg = {"embedding": {"scale": 3.0, "bigram": {"buckets": 7, "mul_prev": 5, "mul_cur": 2}}}
    x = P.embed(cfg, w, [4, 9, 1])
    assert x[:, 0].tolist() == [12.0 + 700.0, 27.0 + 100.0 * ((20 + 18) % 7), 3.0 + 100.0 * ((45 + 2) % 7)]


def test_ramped_frequencies_by_hand_and_the_products_tables():
    sc = {"factor": 4.0, "original": 256.0, "fast": 8.0, "slow": 1.0}
    f, gain = P.frequencies(16, 100.0, sc)
    assert abs(gain - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    lo = math.floor(16 * math.log(256 / (8 * 2 * math.pi)) / (2 * math.log(100.0)))
    hi = math.ceil(16 * math.log(256 / (2 * math.pi)) / (2 * math.log(100.0)))
    assert 0 < lo < hi < 15
    plain, one = P.frequencies(16, 100.0)
    assert one == 1.0 and f[lo] == plain[lo]
    for i in range(8):
        r = min(max((i - lo) / (hi - lo), 0.0), 1.0)
        assert abs(f[i] - (plain[i] * (1 - r) + plain[i] / 4 * r)) < 1e-12
    pe = build_part("position_encoding", PartSpec("rope", dict(rotary_dim=16, theta=100.0, ramp=sc, precise=True, exact_angles=True)))
    pe.prepare(type("rt", (), {"device": "cpu"}), 300)
    want = torch.tensor([[math.sin(p * fi) * gain for fi in f] for p in range(300)], dtype=F64)
    assert (pe.sin.double() - want).abs().max() < 1e-6


@pytest.mark.parametrize("pairs", [True, False])
def test_rotation_by_hand_and_by_distance(pairs):
    torch.manual_seed(1)
    q, k = torch.randn(1, 1, 12, dtype=F64), torch.randn(1, 1, 12, dtype=F64)

    def score(pq, pk):
        return float((P.rotate(q, [pq], 8, 100.0, pairs)[0, 0] * P.rotate(k, [pk], 8, 100.0, pairs)[0, 0]).sum())
    assert abs(score(17, 5) - score(112, 100)) < 1e-9 and abs(score(17, 5) - score(17, 6)) > 1e-3
    r = P.rotate(q, [5], 8, 100.0, pairs)[0, 0]
    a, iu, iv = 5 * 100.0 ** (-2.0 / 8), *((2, 3) if pairs else (1, 5))   # pair 1 at position 5
    assert abs(float(r[iv]) - float(q[0, 0, iv] * math.cos(a) + q[0, 0, iu] * math.sin(a))) < 1e-12
    assert torch.equal(r[8:], q[0, 0, 8:])


def test_chunked_attention_by_hand_and_its_mask_by_perturbation():
    torch.manual_seed(2)
    n, size = 11, 4
    q, k, v = torch.randn(n, 4, 6, dtype=F64), torch.randn(n, 2, 6, dtype=F64), torch.randn(n, 2, 5, dtype=F64)
    base = P.attend(q, k, v, 0.4, size, True)
    s = 0.4 * (k[4:7, 1] @ q[6, 2])                                     # token 6, query head 2 reads key/value head 1, chunk 4..7
    e = torch.exp(s)
    assert torch.allclose(base[6, 2], (e @ v[4:7, 1]) / (1.0 + e.sum()))
    for j in range(n):
        v2 = v.clone()
        v2[j] += 1.0
        moved = (P.attend(q, k, v2, 0.4, size, True) - base).abs().amax(dim=(1, 2)) > 1e-9
        assert moved.tolist() == [i >= j and i // size == j // size for i in range(n)]
    assert torch.allclose(P.attend(q, k, v, 0.4)[0], v[0].repeat_interleave(2, dim=0))   # one key and nothing added: its value
    big = P.attend(100.0 * q, k, v, 0.4, size, True)
    assert torch.isfinite(big).all()


def test_values_are_keys_before_they_turn():
    torch.manual_seed(3)
    mx = {"heads": 2, "kv_heads": 1, "dim": 4, "scale": 0.0, "mask": {"size": 1}, "rot": {"dims": 4, "base": 50.0}}
    w = {"m." + n: torch.randn(s, dtype=F64) for n, s in (("q", (8, 5)), ("q.b", (8,)), ("k", (4, 5)), ("k.b", (4,)), ("g", (8, 5)),
                                                          ("o", (5, 8)), ("o.b", (5,)))}
    h = torch.randn(6, 5, dtype=F64)
    # chunks of one token and scores of zero: half of the token's own unrotated key
    k = h @ w["m.k"].T + w["m.k.b"]
    o = torch.cat([k, k], dim=1) / 2 * torch.sigmoid(h @ w["m.g"].T)
    assert torch.allclose(P.key_value_attention(h, w, "m.", mx), o @ w["m.o"].T + w["m.o.b"])


def test_fixed_decays_by_their_sum():
    torch.manual_seed(4)
    n, e, ev = 7, 3, 5
    q, k, v = torch.randn(n, 1, e, dtype=F64), torch.randn(n, 1, e, dtype=F64), torch.randn(n, 1, ev, dtype=F64)
    got = P.decay_walk(q, k, v, [0.7])
    want = sum(0.7 ** (6 - t) * float(q[6, 0] @ k[t, 0]) * v[t, 0] for t in range(n))
    assert torch.allclose(got[6, 0], want)
    state = [torch.zeros(e, ev, dtype=F64)]
    a = P.decay_walk(q[:2], k[:2], v[:2], [0.7], state)
    b = P.decay_walk(q[2:], k[2:], v[2:], [0.7], state)
    assert torch.allclose(torch.cat([a, b]), got)


def test_causal_convolution_meets_its_last_tap_with_the_current_token():
    x = torch.arange(1.0, 7.0, dtype=F64)[:, None]
    w, b = torch.tensor([[100.0, 10.0, 1.0]], dtype=F64), torch.tensor([0.5], dtype=F64)
    y = P.causal_conv(x, w, b)
    assert y[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5, 345.5, 456.5]
    assert torch.equal(P.causal_conv(x[4:], w, b, before=x[2:4]), y[4:])


def test_gated_unit_by_hand():
    u = torch.tensor([[2.0], [-1.0]], dtype=F64)
    r, i, lam = torch.tensor([[0.25], [0.5]], dtype=F64), torch.tensor([[0.5], [1.0]], dtype=F64), torch.tensor([-3.0], dtype=F64)
    S, last = P.gated_unit_walk(u, r, i, lam)
    sp = math.log1p(math.exp(-3.0))
    a0, a1 = math.exp(-8 * 0.25 * sp), math.exp(-8 * 0.5 * sp)
    s0 = math.sqrt(1 - a0 * a0) * 0.5 * 2.0
    s1 = a1 * s0 - math.sqrt(1 - a1 * a1)
    assert abs(float(S[0]) - s0) < 1e-12 and abs(float(S[1]) - s1) < 1e-12 and float(last) == float(S[1])
    # a block's gate reads its own part of u only, output channel before input channel
    w = torch.zeros(2, 2, 2, dtype=F64)
    w[1, 0, 1] = 3.0
    g = P.block_gate(torch.tensor([[5.0, 6.0, 7.0, 8.0]], dtype=F64), w, torch.zeros(2, 2, dtype=F64))
    assert torch.allclose(g, torch.sigmoid(torch.tensor([[0.0, 0.0, 24.0, 0.0]], dtype=F64)))
