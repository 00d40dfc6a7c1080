"""The Fugavik configuration, its model description, the updates that carry a layer norm of their own, and the plain
implementation's own mechanisms checked against what they must equal (no GPU)."""
import copy
import math

import pytest
import torch

from odin_infer_b200.cache import CacheManager
from odin_infer_b200.config import ConfigError, FugavikConfig, config_from_dict, lookup_architecture
from odin_infer_b200.engine.model import DecoderModel
from odin_infer_b200.parts.base import Normed, PartSpec, build_part, split_update
from tests.plain import fugavik_plain as P

F64 = torch.float64
ATT = {"heads": 6, "kv_heads": 3, "dim": 20, "vdim": 28, "scale": 0.3, "v_mix": True,
       "rot": {"dims": 12, "base": 700.0, "scaling": {"factor": 3.0}}}
RAW = {"architecture": "Fugavik", "vocab": 151, "width": 72, "norm": {"eps": 1e-6},
       "layers": [{"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "conv": 3},
                   "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2}}},
                  {"type": "attention", "mixer": ATT, "mlp": {"kind": "dense", "ff": 40}},
                  {"type": "latent_attention", "mixer": {"heads": 3, "dim": 16, "vdim": 24, "kv_rank": 40, "scale": 0.2}, "mlp": None},
                  {"type": "attention", "mixer": copy.deepcopy(ATT), "mlp": None}]}


def test_configuration_reads_and_writes_the_same_keys():
    cfg = config_from_dict(RAW)
    assert isinstance(cfg, FugavikConfig) and cfg.to_dict() == RAW and config_from_dict(cfg.to_dict()) == cfg
    d, a, l, _ = cfg.layers
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.conv, d.experts, d.top, d.ff) == (4, 2, 12, 20, 3, 5, 2, 24)
    assert (a.rot_dims, a.rot_base, a.rot_factor, a.v_mix, a.scale) == (12, 700.0, 3.0, True, 0.3)
    assert (l.kv_rank, l.vdim, l.scale, l.mlp_kind) == (40, 24, 0.2, None)


def test_absent_keys_mean_absent_mechanisms():
    raw = copy.deepcopy(RAW)
    mx = raw["layers"][1]["mixer"]
    del mx["rot"], mx["v_mix"]
    raw["layers"] = raw["layers"][1:2]
    cfg = config_from_dict(raw)
    spec = lookup_architecture("Fugavik").build_spec(cfg)
    block = spec.layers[0].args
    assert not spec.position_encodings and block["mixer"].args["value_mix"] is None
    raw["layers"][0]["mixer"]["rot"] = {"dims": 8, "base": 50.0}
    cfg = config_from_dict(raw)
    (pe,) = lookup_architecture("Fugavik").build_spec(cfg).position_encodings.values()
    assert pe.args["slowdown"] == 1.0 and pe.args["rotary_dim"] == 8


def test_every_fault_of_a_configuration_in_one_error():
    bad = copy.deepcopy(RAW)
    bad["layers"][0]["mixer"]["kv_heads"] = 3
    bad["layers"][0]["mlp"]["router"]["top"] = 6
    bad["layers"][1]["mixer"]["rot"]["dims"] = 22
    bad["layers"][1]["mixer"]["rot"]["scaling"]["factor"] = 0
    del bad["layers"][2]["mixer"]["kv_rank"]
    bad["layers"][3]["mixer"]["vdim"] = 30
    with pytest.raises(ConfigError) as e:
        config_from_dict(bad)
    for part in ("multiple of kv_heads", "top 6", "dims (22)", "factor", "'kv_rank'", "equal kv_heads and vdim"):
        assert part in str(e.value), (part, str(e.value))


def test_the_model_description_names_every_tensor_once():
    model = DecoderModel(lookup_architecture("Fugavik").build_spec(config_from_dict(RAW)))
    names = [p.name for p in model.params()]
    assert len(names) == len(set(names))
    shapes = {p.name: p.shape for p in model.params() if not p.optional}
    for n, s in (("l0.mix.q.conv", (24, 3)), ("l0.mix.v.conv", (80, 3)), ("l0.mix.b", (4, 72)), ("l0.mix.norm", (20,)),
                 ("l0.mlp.router", (5, 72)), ("l0.mlp.e4.down", (72, 24)), ("l0.ls2", (72,)), ("l0.norm2.b", (72,)),
                 ("l1.mix.q.norm", (20,)), ("l1.mix.sink", (6,)), ("l1.mix.v", (84, 72)), ("l1.mlp.up", (40, 72)),
                 ("l2.mix.dkv", (40, 72)), ("l2.mix.uv", (72, 40)), ("l2.mix.g", (3, 72)), ("l3.mix.vmix", ()),
                 ("final.norm.b", (72,)), ("head", (151, 72))):
        assert shapes.get(n) == s, (n, shapes.get(n))
    # the first layer that mixes values has nothing to mix with, a layer without feed-forward no second norm
    assert {p.name for p in model.params() if p.optional} == {"l1.mix.vmix"} | {f"l{i}.{n}" for i in (2, 3)
                                                                               for n in ("norm2", "norm2.b", "ls2")}
    assert model.graph_safe
    cache = CacheManager(64 * 4, 64 * 2)
    model.register_cache(cache)
    assert cache.state_bytes_of == [4 * (4 * 12 * 20 + 2 * (2 * 24 + 80)), 0, 0, 0]
    kept = sorted((g.request.n_kv_heads, g.request.head_dim, g.request.value_dim, g.n_lines, g.request.shared_kv)
                  for g in cache.groups.values())
    assert kept == [(1, 40, 40, 1, True), (3, 20, 28, 2, False)]     # the latent row, and one group for both attention layers


def test_an_update_with_a_layer_norm_passes_to_whoever_adds_it():
    u = Normed("a", torch.ones(4), 1e-5, torch.zeros(4), True)
    assert split_update(u) == (u, None) and u.center
    ln = build_part("norm", PartSpec("layernorm", dict(width=4, eps=1e-5, weight="w", bias="b", scale="s")))
    ln.bind({"w": torch.tensor([1., 2, 3, 4]), "b": torch.tensor([1., 1, 1, 1]), "s": torch.tensor([2., 0, 1, -1])}, None)
    assert ln.weight.tolist() == [2, 0, 3, -4] and ln.bias.tolist() == [2, 0, 1, -1]     # the scale multiplies both
    n = ln.as_update_norm("u")
    assert n.update == "u" and n.center and n.weight is ln.weight and n.bias is ln.bias
    none = PartSpec("none", dict(width=4))
    mixer = PartSpec("gated_delta_rule", dict(width=4, n_heads=1, n_groups=1, head_dim=4, v_head_dim=4, taps=2, names={
        k: k for k in ("q", "k", "v", "g", "b", "a", "o", "q_conv", "k_conv", "v_conv", "A_log", "dt_bias", "norm")}))
    blk = build_part("block", PartSpec("prenorm", dict(mixer=mixer, feed_forward=None, norm_mixer=none, norm_feed_forward=None,
                                                       post_norm_mixer=PartSpec("layernorm", dict(width=4, eps=1e-5, weight="w", bias="b")))))
    assert blk.post_mixer.can_norm_updates
    with pytest.raises(TypeError):      # what hands the stream on cannot stand on a sublayer's output
        build_part("block", PartSpec("prenorm", dict(mixer=mixer, feed_forward=None, norm_mixer=none, norm_feed_forward=None,
                                                     post_norm_mixer=none)))


def test_parts_refuse_what_they_cannot_do():
    names = {k: k for k in ("router", "gate", "up", "down")}
    with pytest.raises(ValueError):     # groups need a score that knows them
        build_part("feed_forward", PartSpec("routed_experts", dict(width=8, inner=8, n_experts=4, top=1, names=names,
                                                                   score="sigmoid_as_is", groups=2)))
    with pytest.raises(ValueError):     # a stretch of one kind only
        build_part("position_encoding", PartSpec("rope", dict(rotary_dim=8, theta=100.0, slowdown=2.0, stretch={
            "factor": 2.0, "low": 1.0, "high": 4.0, "original": 64})))
    with pytest.raises(ValueError):     # a mixer without values of its own
        build_part("mixer", PartSpec("gqa_attention", dict(width=8, n_q_heads=1, n_kv_heads=1, head_dim=8, kv_shared=True,
                                                           value_mix={"key": "v"}, names={k: k for k in "qo"}, qk_norm=False)))


# ---- the plain implementation against what it must equal ------------------------------------------------------
def test_slowed_rotation_by_hand_and_by_distance():
    torch.manual_seed(1)
    q, k = torch.randn(1, 1, 12, dtype=F64), torch.randn(1, 1, 12, dtype=F64)

    def score(pq, pk):
        return float((P.rotate(q, [pq], 8, 100.0, 2.5)[0, 0] * P.rotate(k, [pk], 8, 100.0, 2.5)[0, 0]).sum())
    assert abs(score(17, 5) - score(112, 100)) < 1e-9 and abs(score(17, 5) - score(17, 6)) > 1e-3
    r = P.rotate(q, [5], 8, 100.0, 2.5)[0, 0]
    a = 5 / 2.5 * 100.0 ** (-2.0 / 8)                                   # pair 1 (elements 1 and 5) at position 5
    assert abs(float(r[5]) - float(q[0, 0, 5] * math.cos(a) + q[0, 0, 1] * math.sin(a))) < 1e-12
    assert torch.equal(r[8:], q[0, 0, 8:])
    assert torch.allclose(P.rotate(q, [5], 8, 100.0, 2.5), P.rotate(q, [2], 8, 100.0, 1.0))   # positions shrink by the factor


def test_the_product_tables_turn_by_the_same_angles():
    pe = build_part("position_encoding", PartSpec("rope", dict(rotary_dim=8, theta=100.0, slowdown=2.5, precise=True, exact_angles=True)))
    pe.prepare(type("rt", (), {"device": "cpu"}), 40)
    want = torch.tensor([[math.cos(p / 2.5 * 100.0 ** (-2.0 * i / 8)) for i in range(4)] for p in range(40)], dtype=F64)
    assert (pe.cos.double() - want).abs().max() < 1e-7


def test_sink_attention_by_hand_and_its_mask_by_perturbation():
    torch.manual_seed(2)
    n = 7
    q, k, v = torch.randn(n, 4, 6, dtype=F64), torch.randn(n, 2, 6, dtype=F64), torch.randn(n, 2, 5, dtype=F64)
    sink = torch.tensor([0.5, -1.0, 2.0, 0.0], dtype=F64)
    base = P.sink_attention(q, k, v, 0.4, sink)
    s = 0.4 * (k[:4, 1] @ q[3, 2])                                      # token 3, query head 2 reads key/value head 1
    e = torch.exp(s)
    assert torch.allclose(base[3, 2], (e @ v[:4, 1]) / (e.sum() + math.exp(2.0)))
    for j in range(n):
        v2 = v.clone()
        v2[j] += 1.0
        moved = (P.sink_attention(q, k, v2, 0.4, sink) - base).abs().amax(dim=(1, 2)) > 1e-9
        assert moved.tolist() == [i >= j for i in range(n)]
    no_sink = P.sink_attention(q, k, v, 0.4, torch.full((4,), -math.inf, dtype=F64))
    assert torch.allclose(no_sink[0], v[0].repeat_interleave(2, dim=0))  # one key and no sink: its value


def test_values_are_mixed_with_the_first_layers_after_that_layer():
    torch.manual_seed(3)
    mx = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 3, "scale": 0.5, "v_mix": True}
    w = {"m." + n: torch.randn(s, dtype=F64) for n, s in (("q", (8, 5)), ("k", (4, 5)), ("v", (3, 5)), ("q.norm", (4,)), ("k.norm", (4,)),
                                                          ("sink", (2,)), ("o", (5, 6)), ("vmix", ()))}
    x = torch.randn(6, 5, dtype=F64)
    _, own = P.attention(x, w, "m.", mx, 1e-5)
    assert torch.allclose(own.view(6, 3), x @ w["m.v"].T)
    first = torch.randn(6, 1, 3, dtype=F64)
    _, mixed = P.attention(x, w, "m.", mx, 1e-5, first)
    assert torch.allclose(mixed, (1 - w["m.vmix"]) * own + w["m.vmix"] * first)
    _, plain = P.attention(x, w, "m.", {**mx, "v_mix": False}, 1e-5, first)
    assert torch.equal(plain, own)


def test_causal_convolution_meets_its_last_tap_with_the_current_token():
    x = torch.arange(1.0, 7.0, dtype=F64)[:, None]
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=F64)
    y = P.causal_conv(x, w)
    assert y[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0, 456.0]
    assert torch.equal(P.causal_conv(x[4:], w, before=x[2:4]), y[4:])


def test_the_delta_rule_is_a_product_of_corrections():
    torch.manual_seed(4)
    n, e, ev = 6, 4, 3
    q, k, v = torch.randn(n, 1, e, dtype=F64), P.unit(torch.randn(n, 1, e, dtype=F64)), torch.randn(n, 1, ev, dtype=F64)
    beta, g = torch.rand(n, 1, dtype=F64), torch.rand(n, 1, dtype=F64)
    got = P.delta_walk(q, k, v, beta, g)
    S = torch.zeros(e, ev, dtype=F64)
    for t in range(n):
        kt = k[t, 0][:, None]
        S = g[t, 0] * (torch.eye(e, dtype=F64) - beta[t, 0] * kt @ kt.T) @ S + beta[t, 0] * kt @ v[t, 0][None, :]
        assert torch.allclose(got[t, 0], S.T @ q[t, 0])
    # with full strength and no decay a key answers exactly what was last written under it, and a repeat replaces
    kk = torch.eye(e, dtype=F64)[[0, 1, 0]][:, None, :]
    vv = torch.randn(3, 1, ev, dtype=F64)
    one = torch.ones(3, 1, dtype=F64)
    o = P.delta_walk(kk, kk, vv, one, one)
    assert torch.allclose(o, vv)
    state = [torch.zeros(e, ev, dtype=F64)]
    a = P.delta_walk(q[:2], k[:2], v[:2], beta[:2], g[:2], state)
    b = P.delta_walk(q[2:], k[2:], v[2:], beta[2:], g[2:], state)
    assert torch.allclose(torch.cat([a, b]), got)


def test_layer_norm_and_unit_vectors_by_hand():
    y = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F64)
    out = P.ln(y, torch.tensor([1.0, 1, 2, 1], dtype=F64), torch.tensor([0.0, 1, 0, 0], dtype=F64), 4.0)
    assert torch.allclose(out, torch.tensor([[-1.0, 1 - 1 / 3, 2 / 3, 1.0]], dtype=F64))    # deviations -3 -1 1 3, variance 5, root 3
    u = P.unit(torch.tensor([3.0, 4.0], dtype=F64))
    assert torch.allclose(u, torch.tensor([0.6, 0.8], dtype=F64), atol=1e-7)


def test_experts_read_their_score_times_the_input():
    ident = torch.eye(3, dtype=F64)
    x = torch.tensor([[2.0, -1.0, 0.5]], dtype=F64)
    picks = P.route(x, ident, {"experts": 3, "top": 2})[0]
    sg = torch.sigmoid(x[0])
    assert [e for e, _ in picks] == [0, 2] and abs(picks[0][1] - float(sg[0])) < 1e-12 and abs(picks[1][1] - float(sg[2])) < 1e-12
    w = {"m.router": ident}
    torch.manual_seed(5)
    for e in range(3):
        w.update({f"m.e{e}.gate": torch.randn(4, 3, dtype=F64), f"m.e{e}.up": torch.randn(4, 3, dtype=F64), f"m.e{e}.down": torch.randn(3, 4, dtype=F64)})
    got = P.expert_mlp(x, w, "m.", {"router": {"experts": 3, "top": 2}})
    want = torch.zeros(3, dtype=F64)
    for e in (0, 2):
        h = sg[e] * x[0]
        want += w[f"m.e{e}.down"] @ (P.silu(w[f"m.e{e}.gate"] @ h) * (w[f"m.e{e}.up"] @ h))
    assert torch.allclose(got[0], want)
