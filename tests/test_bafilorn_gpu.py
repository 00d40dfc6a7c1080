"""The Bafilorn decoder through the engine against its plain implementation (tests/plain/bafilorn_plain.py): every mechanism
alone, whole prompts against token-by-token decoding, prompts in portions, unequal batches, slots, pages and states that are
used again, keys on either side of a chunk's edge, the first tokens of a sequence, long decoding, sizes that the fast kernels
take and sizes that they do not, and greedy generation through the engine's own entry point.  The tests write their own
weights and inputs (matrices of unit gain, decays that remember for hundreds of tokens, a key far back that one query asks
for, streams that the sublayers read and join unevenly) so that a lost state, a chunk that is one token off or a one that is
not added leaves a mark far above rounding."""
import json
import math
import os

import numpy as np
import pytest
import torch

from tests import traces
from tests.plain import bafilorn_plain as P
from tests.test_fugavik_gpu import within
from tests.test_meropel_gpu import CUTS, cache_for, close, engine_for, portions, replay, requests_for, runtime
from tests.tiny import random_tokens

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def lat(heads, dim, rot, vdim, q_rank, kv_rank, scale, base=1e4):
    return {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
            "rot": {"dims": rot, "base": base}}


def lig(heads, dim, vdim, slowest=0.998):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": [round(0.6 + (slowest - 0.6) * (i + 1) / heads, 6) for i in range(heads)]}


def par(heads, kv, dim, scale, size, rot, inner, blocks, conv, base=1e4, ramp=None):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": scale, "mask": {"size": size},
            "rot": {"dims": rot, "base": base}}
    if ramp is not None:
        left["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), ramp))
    return {"left": left, "right": {"width": inner, "blocks": blocks, "conv": conv}}


def model(vocab, width, streams, eps, *layers, loop=None, scale=1.0, pair=(61, 7, 3)):
    kinds = {"kv_rank": "latent_attention", "decay": "lightning"}
    out = {"architecture": "Bafilorn", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
           "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pair))},
           "layers": [{"type": next((t for k, t in kinds.items() if k in mx), "parallel"), "mixer": mx,
                       "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for mx, ff in layers]}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# odd sizes throughout, three streams, a loop of two layers that runs three times, layers without feed-forward, chunks
# smaller than a page, several key/value heads, frequencies with and without a ramp
MIXED = model(211, 96, 3, 1e-5,
              (par(6, 3, 20, 0.3, 50, 12, 60, 5, 3, base=900.0, ramp=(3.0, 300.0, 8.0, 0.5)), 80),
              (lig(3, 24, 40), None),
              (lat(3, 20, 12, 28, 24, 36, 0.25, base=700.0), 56),
              (par(4, 2, 24, 0.35, 130, 24, 96, 3, 5), None),
              (lig(2, 20, 12), 40), loop=(1, 3, 3), scale=1.75)
# a width that is no multiple of 8; one head; one block; a convolution of one tap and of six; channels that are no multiple
# of four; five streams; the whole model runs twice; chunks of one page
ODD = model(97, 100, 5, 1e-6,
            (lat(1, 36, 4, 12, 20, 29, 0.2), 52),
            (par(3, 1, 20, 0.25, 64, 20, 33, 1, 1, base=50.0), None),
            (lig(1, 18, 36), 28),
            (par(2, 2, 12, 0.4, 7, 4, 42, 6, 6, ramp=(16.0, 64.0, 4.0, 1.0)), 36), loop=(0, 4, 2), scale=0.3, pair=(1, 5, 2))
# head sizes the tensor-core attention kernels take, widths the tensor-core products take; gates' blocks of 64 channels
FAST = model(384, 128, 2, 1e-5,
             (lat(8, 64, 64, 32, 64, 64, 0.1), 256),
             (lig(4, 64, 128), 176),
             (par(4, 2, 64, 0.14, 96, 64, 256, 4, 4), None),
             (par(2, 2, 128, 0.1, 200, 32, 128, 2, 2, base=1e6, ramp=(2.5, 200.0, 16.0, 1.0)), 128), loop=(2, 4, 2), scale=2.0,
             pair=(503, 31, 17))
# one stream only (its mix and its factors stay), no loop
ONE = model(130, 64, 1, 1e-4, (lig(2, 16, 16), 64), (par(2, 1, 16, 0.4, 33, 8, 64, 2, 4), 48), (lat(2, 16, 8, 16, 16, 24, 0.3), None))
CONFIGS = {"mixed": (MIXED, 3), "odd": (ODD, 5), "fast": (FAST, 7), "one": (ONE, 9)}


def make_weight(name: str, shape, gen) -> torch.Tensor:
    """Weights of the tests' own making: matrices N(0, 1/in), norms around one (or around zero where the one is added), biases,
    streams that are read, mixed and joined unevenly but keep their size, gated units that remember for hundreds of tokens."""
    r = torch.randn(shape, generator=gen)
    last = name.rsplit(".", 1)[-1]
    if last in ("norm1", "norm2") or name == "final.norm":
        return 0.3 * r
    if last in ("norm", "out") and len(shape) == 1 and ".hc" not in name:
        return 1.0 + 0.3 * r
    if ".hc" in name:
        s = shape[-1]
        if last == "mix":
            return 0.8 * torch.eye(s) + 0.2 / s + 0.1 * r
        return (1.0 / s if last == "in" else 1.0) + 0.4 * r
    if last == "b":
        return 0.3 * r
    if last in ("embed", "bigram"):
        return r
    if last == "conv":
        return 0.5 * r
    if last == "lam":
        return -4.0 + 1.5 * r
    return r / math.sqrt(shape[-1])


def write_model(folder: str, raw: dict, seed: int) -> str:
    from odin_infer_b200.config import config_from_dict
    from odin_infer_b200.weights import model_param_specs
    from odin_infer_b200.weights.safetensors_io import write_safetensors
    cfg = config_from_dict(raw)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(raw, f)
    gen = torch.Generator().manual_seed(seed)
    specs = model_param_specs(cfg)
    shapes = {s.name: s.concrete_shape for s in specs}
    write_safetensors(os.path.join(folder, "model.safetensors"), [(s.name, torch.bfloat16, s.concrete_shape) for s in specs],
                      lambda name: make_weight(name, shapes[name], gen).to(torch.bfloat16))
    return folder


_folders = {}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    if not _folders:
        base = tmp_path_factory.mktemp("bafilorn")
        for name, (raw, seed) in CONFIGS.items():
            _folders[name] = write_model(os.path.join(str(base), name), raw, seed)
    return _folders


_plain = {}


def plain_logits(folder, tokens, rounded=None):
    """rounded: None (exact), "bfloat16" or "float32": what an engine of that type stores between kernels is rounded to it."""
    key = (folder, tuple(tokens), rounded)
    if key not in _plain:
        cfg, w = P.read_model_folder(folder, F64)
        rnd = {None: lambda t: t, "bfloat16": P.to_bfloat16_and_back, "float32": lambda t: t.float().double()}[rounded]
        _plain[key] = P.forward(cfg, w, tokens, rnd=rnd).numpy()
    return _plain[key]


def check_rows(got: dict, folder, requests, dtype):
    for rid, rows in got.items():
        n, toks = rows.shape[0], requests[rid]
        ok, first, text = within(rows, plain_logits(folder, toks)[:n], plain_logits(folder, toks, rounded=dtype)[:n], dtype)
        assert ok, f"{rid}: {text}, first over at {first}"


# --------------------------------------------------------------------------------------
# the whole model in every cut
# --------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_and_one_by_one(folders, name, dtype):
    """Whole prompts (across several pages and chunks, the recurrences in blocks), then the same with the last tokens one by
    one, so that states and the convolutions' last inputs pass from the prompt's kernels to the single-token ones and keys
    of a chunk are decoded over its edge; the first tokens of a sequence alone (prompts of 1 and 2)."""
    raw = CONFIGS[name][0]
    reqs = requests_for(raw, [1, 2, 131, 262])
    engine = engine_for(folders[name], dtype)
    check_rows(traces.collect(traces.whole(reqs), replay(engine, traces.whole(reqs))), folders[name], reqs, dtype)
    recs = traces.tail_one_by_one(reqs, tail=70)
    check_rows(traces.collect(recs, replay(engine, recs)), folders[name], reqs, dtype)
    engine.cache.check()
    assert all(g.pool.n_held == 0 for g in engine.cache.groups.values())
    engine.destroy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,sizes", [("mixed", (2, 35, 3, 64)), ("odd", (17, 2, 2, 90)), ("fast", (130, 2, 70, 1, 129)),
                                        ("mixed", (2,)), ("odd", (1, 3)), ("one", (33, 2))])
def test_prompts_in_portions(folders, name, sizes, dtype):
    """Portions of several sizes, down to two tokens and one: a portion starts from the states, the token before and the
    convolutions' last inputs (also when it is shorter than the convolution), and in the middle of a chunk, which is
    counted from the sequence's start."""
    raw = CONFIGS[name][0]
    reqs = requests_for(raw, [131, 41] if len(sizes) <= 2 else [260, 77], seed=0 if len(sizes) > 2 else 10)
    engine = engine_for(folders[name], dtype)
    recs = portions(reqs, sizes)
    check_rows(traces.collect(recs, replay(engine, recs)), folders[name], reqs, dtype)
    engine.destroy()


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_batches_and_reuse(folders, name, dtype, graphs):
    """Batches of unequal requests, batch after batch in a cache that holds one batch only, so that every slot, every
    page and every slot's state is used again; shorter requests end earlier."""
    raw = CONFIGS[name][0]
    reqs = requests_for(raw, [5, 180, 66, 1, 129, 40, 97, 200, 3], seed=20)
    recs = traces.batches(reqs, 3, first_part=lambda n: max(1, n - 9))
    engine = engine_for(folders[name], dtype, max_tokens=traces.max_live_tokens(recs) + 64, graphs=graphs)
    check_rows(traces.collect(recs, replay(engine, recs)), folders[name], reqs, dtype)
    engine.cache.check()
    engine.destroy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_requests_join_a_running_batch(folders, dtype):
    raw = CONFIGS["mixed"][0]
    reqs = requests_for(raw, [60, 45, 90, 30, 75], seed=30)
    recs = traces.joining(reqs)
    engine = engine_for(folders["mixed"], dtype)
    check_rows(traces.collect(recs, replay(engine, recs)), folders["mixed"], reqs, dtype)
    engine.destroy()


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_cuts_agree_in_32_bit(folders, name):
    """In 32-bit a position's logits agree to rounding whole, in portions, one by one and in a batch, and a batch is the
    same bits as each request alone in the same cut."""
    raw = CONFIGS[name][0]
    reqs = requests_for(raw, [140, 59], seed=40)
    engine = engine_for(folders[name], "float32")
    ref = traces.collect(traces.whole(reqs), replay(engine, traces.whole(reqs)))
    for recs in (portions(reqs, (3, 50, 2)), traces.tail_one_by_one(reqs, tail=25), traces.batches(reqs, 2)):
        got = traces.collect(recs, replay(engine, recs))
        for rid in reqs:
            top = np.abs(ref[rid]).max()
            assert np.abs(got[rid] - ref[rid]).max() <= 1e-5 * top, rid
    alone = traces.collect(traces.batches(reqs, 1), replay(engine, traces.batches(reqs, 1)))
    both = traces.collect(traces.batches(reqs, 2), replay(engine, traces.batches(reqs, 2)))
    for rid in reqs:
        top = np.abs(alone[rid]).max()
        assert np.abs(alone[rid] - both[rid]).max() <= 2e-6 * top, rid
    engine.destroy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "fast"])
def test_long_decoding(folders, name, dtype):
    """Two hundred and fifty tokens decoded one by one after a short prompt: every state is carried as often, the keys grow
    over page borders and chunks begin anew, their pages given back."""
    raw = CONFIGS[name][0]
    reqs = requests_for(raw, [262, 250], seed=50)
    recs = traces.batches(reqs, 2, first_part=lambda n: 12)
    engine = engine_for(folders[name], dtype)
    check_rows(traces.collect(recs, replay(engine, recs)), folders[name], reqs, dtype)
    assert all(g.pool.n_held == 0 for g in engine.cache.groups.values())
    engine.destroy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt(folders, dtype):
    """A prompt of 1,100 tokens whole, and with its last 40 tokens one by one: many blocks of the recurrences, keys many pages
    back, pages of earlier chunks given back."""
    raw = CONFIGS["fast"][0]
    reqs = requests_for(raw, [1100], seed=70)
    engine = engine_for(folders["fast"], dtype, max_tokens=2048, max_ctx=1280)
    for recs in (traces.whole(reqs), traces.tail_one_by_one(reqs, tail=40)):
        check_rows(traces.collect(recs, replay(engine, recs)), folders["fast"], reqs, dtype)
    engine.cache.check()
    engine.destroy()


def test_what_a_sequence_holds(folders):
    """Every run of a layer has a cache line or a state of its own; the latent layer keeps one row per token, the layers over
    chunks a group per chunk and head size; the embedding keeps the token before."""
    engine = engine_for(folders["mixed"], "float32")
    kept = sorted((g.request.n_kv_heads, g.request.head_dim, g.request.chunk, g.n_lines, g.request.shared_kv) for g in engine.cache.groups.values())
    assert kept == [(1, 48, 0, 3, True), (2, 24, 130, 1, False), (3, 20, 50, 1, False)], kept
    light = 4 * 3 * 24 * 40
    assert engine.cache.state_bytes_of == [4 * 60 * 3, light, 0, light, 0, light, 0, 4 * 96 * 5, 4 * 2 * 20 * 12, 4]
    engine.destroy()


@pytest.mark.parametrize("dtype,margin", [("float32", 1e-5), ("bfloat16", 6e-2)])
@pytest.mark.parametrize("name", ["mixed", "fast"])
def test_greedy_generation_through_the_entry_point(folders, name, dtype, margin):
    """`Engine.generate` (the scheduler's batches, sampling on the device, one step ahead of the host): every token it chose
    is the plain logits' maximum, or within rounding of it."""
    raw = CONFIGS[name][0]
    prompts = [random_tokens(n, raw["vocab"], 60 + i) for i, n in enumerate((4, 150, 33, 71, 9))]
    engine = engine_for(folders[name], dtype, max_tokens=0, max_ctx=256)
    outs = engine.generate(prompts, max_new_tokens=12, temperature=0.0, stop_token_ids=[])
    for p, o in zip(prompts, outs):
        assert len(o.tokens) == 12
        ref = plain_logits(folders[name], p + o.tokens)[len(p) - 1:]
        for i, tok in enumerate(o.tokens):
            assert float(ref[i].max() - ref[i][tok]) <= margin * float(np.abs(ref[i]).max()), (len(p), i)
    engine.destroy()


def test_the_command_line_generates(folders, capsys):
    from odin_infer_b200 import cli
    assert cli.main([folders["odd"], "--prompt-ids", "1,2,3,4", "-n", "5", "-t", "0", "-c", "128", "--json"]) == 0
    out = [json.loads(line) for line in capsys.readouterr().out.splitlines() if line.startswith("{")]
    assert out and len(out[0]["tokens"]) == 5


def random_config(seed: int) -> dict:
    rng = np.random.default_rng(seed)

    def pick(*xs):
        return xs[int(rng.integers(len(xs)))]

    def mixer():
        kind = pick("latent", "lightning", "parallel", "parallel")
        if kind == "latent":
            return lat(pick(1, 2, 5), pick(8, 20, 64), pick(2, 8, 16, 64), pick(8, 24, 64), pick(8, 30, 64), pick(16, 33, 64),
                       float(rng.uniform(0.1, 0.4)), base=pick(50.0, 1e4, 1e6))
        if kind == "lightning":
            return lig(pick(1, 2, 3, 5), pick(8, 18, 32, 70), pick(8, 20, 33), slowest=pick(0.9, 0.999))
        kv, dim, blocks = pick(1, 2, 3), pick(8, 24, 64, 128), pick(1, 2, 4, 7)
        return par(kv * pick(1, 2, 4), kv, dim, float(rng.uniform(0.1, 0.4)), pick(1, 9, 63, 64, 65, 128, 400), pick(2, 4, dim // 2, dim),
                   blocks * pick(8, 12, 32, 33), blocks, pick(1, 2, 3, 4, 7), base=pick(50.0, 1e4, 1e6),
                   ramp=pick(None, (2.0, 100.0, 8.0, 1.0), (16.0, 1000.0, 32.0, 1.0), (1.5, 30.0, 2.0, 0.5)))
    n = int(rng.integers(2, 5))
    start = int(rng.integers(0, n))
    stop = int(rng.integers(start + 1, n + 1))
    return model(int(rng.integers(50, 300)), pick(64, 72, 100, 128), pick(1, 2, 2, 3, 4, 6), pick(1e-5, 1e-6, 1e-3),
                 *[(mixer(), pick(None, 24, 40, 64)) for _ in range(n)], loop=pick(None, (start, stop, int(rng.integers(1, 4)))),
                 scale=float(rng.uniform(0.3, 3.0)), pair=(int(rng.integers(1, 400)), int(rng.integers(1, 90)), int(rng.integers(1, 90))))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [501, 502, 503, 504, 505, 506, 507, 508, 509, 510])
def test_configurations_drawn_at_random(tmp_path, seed, dtype):
    raw = random_config(seed)
    folder = write_model(str(tmp_path / "m"), raw, seed)
    reqs = requests_for(raw, [150, 37, 3], seed=seed)
    engine = engine_for(folder, dtype)
    for recs in (traces.whole(reqs), traces.batches(reqs, 3, first_part=lambda n: max(1, n - 20))):
        check_rows(traces.collect(recs, replay(engine, recs)), folder, reqs, dtype)
    engine.destroy()


# --------------------------------------------------------------------------------------
# every mechanism alone, with inputs that show a fault
# --------------------------------------------------------------------------------------
def bound(part, dtype, rt, seed, prepare=None):
    """The part bound to weights of the tests' making (`prepare` may change them first); returns them in float64 by name."""
    gen = torch.Generator().manual_seed(seed)
    t = {p.name: make_weight(p.name, p.concrete_shape, gen) for p in part.params()}
    if prepare is not None:
        prepare(t)
    t = {k: v.to(torch.bfloat16).to(dtype).to(DEV) for k, v in t.items()}
    ref = {k: v.double().cpu() for k, v in t.items()}
    part.bind(dict(t), rt)
    return ref


def total(o):
    """A mixer's update as one tensor: partial sums and biases added, the terms of a combined update as their kernel forms them."""
    from odin_infer_b200.parts.base import Biased, Combined
    if isinstance(o, Biased):
        return total(o.update) + o.bias.double()
    if isinstance(o, Combined):
        out = 0
        for t in o:
            v = total(t.value) + (0 if t.bias is None else t.bias.double())
            if t.norm_weight is not None:
                v = v / torch.sqrt((v * v).mean(-1, keepdim=True) + t.norm_eps) * t.norm_weight.double()
            out = out + t.scale * v
        return out
    return (o.double().sum(0) if o.dim() == 3 else o.double())


def in_steps(mixer, rt, cache, h, cuts):
    """The mixer's update for one sequence whose rows h come in steps that end at the given cuts."""
    from odin_infer_b200.engine.step import StepBatch, StepEntry
    slot, at, outs = cache.take_slot(), 0, []
    for end in cuts:
        st = cache.extend(slot, end - at)
        step = StepBatch(cache, [StepEntry(slot, [0] * (end - at), list(range(end - at)))], [st], DEV)
        outs.append(total(mixer.forward(rt, step, h[at:end].contiguous(), 0)).clone())
        cache.after_step(slot)
        at = end
    cache.give_back_slot(slot)
    return torch.cat(outs)


LATENT_GEOMETRIES = [  # heads, dim, rotated, vdim, query latent, kv latent, rows
    (3, 20, 12, 28, 44, 36, 200), (1, 36, 4, 12, 20, 29, 131), (8, 64, 64, 32, 48, 64, 330), (4, 32, 32, 64, 72, 96, 260),
    (5, 16, 16, 24, 33, 48, 70), (3, 32, 64, 40, 520, 512, 90), (2, 24, 8, 16, 184, 180, 75)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("geom", LATENT_GEOMETRIES)
def test_latent_attention_alone_with_a_key_far_back(dtype, tol, geom):
    """The last row's query is built to ask for row 2's latent, hundreds of rows back (through a query latent that carries the
    key's projection, with the input channels in another order); gates differ from element to element and token to token."""
    from odin_infer_b200.parts import PartSpec, build_part
    H, D, R, V, QR, L, n = geom
    width, scale = 80, 16.0 / D
    rt = runtime(dtype)
    perm = torch.randperm(width, generator=torch.Generator().manual_seed(1))
    names = {"dq": "m.dq", "dq_norm": "m.dq.norm", "uq": "m.uq", "dkv": "m.dkv", "dkv_norm": "m.dkv.norm", "uk": "m.uk", "uv": "m.uv", "o": "m.o"}
    mixer = build_part("mixer", PartSpec("latent_attention", dict(
        width=width, n_heads=H, head_dim=D, rot_dim=R, v_head_dim=V, q_rank=QR, kv_rank=L, names=names, position_encoding="pe",
        eps=1e-5, scale=scale, gate="m.g", gate_per_head=False)))
    mixer.pe = build_part("position_encoding", PartSpec("rope", dict(rotary_dim=R, theta=300.0, layout="pairs", precise=True, exact_angles=True)))
    mixer.pe.prepare(rt, n)

    def asks_for_the_other_order(t):
        k = min(QR, L)
        t["m.dq"][:k, perm] = t["m.dkv"][:k]
        uq, uk = t["m.uq"].view(H, D + R, QR), t["m.uk"].view(H, D, L)
        uq[:, :D, :k] = uk[:, :, :k]
        uq[:, :, k:] *= 0.1
        uq[:, D:] *= 0.3
    w = bound(mixer, dtype, rt, H * 17 + L, asks_for_the_other_order)
    torch.manual_seed(L)
    h = torch.randn(n, width, device=DEV)
    h[n - 1, perm.to(DEV)] = h[2]
    h = h.to(dtype)
    mx = lat(H, D, R, V, QR, L, scale, base=300.0)
    ref = P.latent_attention(h.double().cpu(), w, "m.", mx, 1e-5)
    moved = h.clone()
    moved[2] = moved[3]       # without row 2's own key the last row reads something else
    assert (P.latent_attention(moved.double().cpu(), w, "m.", mx, 1e-5)[n - 1] - ref[n - 1]).abs().max() > 0.1 * ref[n - 1].abs().max()
    cache = cache_for([mixer], dtype)
    for cuts in ([n], [2, 63, 64, 65, n - 3, n], list(range(n - 40, n + 1))):
        close(in_steps(mixer, rt, cache, h, cuts), ref, tol)


CHUNK_GEOMETRIES = [  # heads, kv heads, dim, rotated, chunk, ramp, rows
    (6, 3, 20, 12, 50, None, 200), (2, 2, 16, 16, 64, (3.0, 100.0, 8.0, 0.5), 131), (4, 2, 64, 32, 96, (8.0, 200.0, 16.0, 1.0), 330),
    (3, 1, 24, 8, 1, None, 20), (2, 1, 128, 128, 200, None, 405), (8, 2, 64, 64, 130, (2.0, 64.0, 4.0, 1.0), 261),
    (1, 1, 64, 2, 1000, None, 140), (16, 1, 64, 16, 63, None, 190)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("geom", CHUNK_GEOMETRIES)
def test_attention_over_chunks_whose_values_are_keys(dtype, tol, geom):
    """In every chunk the row asked for is the chunk's first and the one before it (just outside): the chunk's last row carries
    both rows' inputs in the other order, the queries being projected by the keys' matrix with its input channels permuted.
    The row outside must not be heard, the one inside must; some rows' scores are so low that the added one is most of the
    denominator.  Whole, in portions that cut chunks, and one by one over the edges."""
    from odin_infer_b200.parts import PartSpec, build_part
    H, G, D, rot, size, ramp, n = geom
    width, scale = 80, 5.0 / D
    rt = runtime(dtype)
    perm = torch.randperm(width, generator=torch.Generator().manual_seed(1))
    att = build_part("mixer", PartSpec("gqa_attention", dict(
        width=width, n_q_heads=H, n_kv_heads=G, head_dim=D, position_encoding="pe", qk_norm=False, scale=scale, chunk=size,
        values_are_keys=True, sink_logit=0.0, gate="m.g", names={s: "m." + s for s in "qko"}, biases={s: f"m.{s}.b" for s in "qko"})))
    keys = ("factor", "original", "fast", "slow")
    att.pe = build_part("position_encoding", PartSpec("rope", dict(rotary_dim=rot, theta=1e7, precise=True, exact_angles=True,
                                                                   ramp=dict(zip(keys, ramp)) if ramp else None)))
    att.pe.prepare(rt, n)

    def alike(t):
        t["m.q"] = t["m.k"].view(G, D, width).repeat_interleave(H // G, dim=0).reshape(H * D, width)[:, perm.argsort()].clone()
        t["m.q"].view(H, D, width)[:, :rot] *= 0.3
    w = bound(att, dtype, rt, H * 13 + D, alike)
    torch.manual_seed(D + size)
    h = torch.randn(n, width, device=DEV)
    h[::7] *= 0.1                                # rows with small scores
    lasts = [c + size - 1 for c in range(size, n - size + 1, size)] if size > 1 else []
    for e in lasts:
        h[e] = (h[e - size + 1] + h[e - size])[perm.argsort().to(DEV)]
    h = h.to(dtype)
    mx = par(H, G, D, scale, size, rot, 1, 1, 1, base=1e7, ramp=ramp)["left"]
    hd = h.double().cpu()
    ref = P.key_value_attention(hd, w, "m.", mx)

    def differs(**other):
        return (P.key_value_attention(hd, w, "m.", {**mx, **other}) - ref).abs().max() > 3 * tol * ref.abs().max()
    if n > size:
        assert differs(mask={"size": size + 1})
    n_added = P.attend
    try:
        P.attend = lambda q, k, v, s, c, one_added: n_added(q, k, v, s, c, False)
        assert differs()                         # without the added one
    finally:
        P.attend = n_added
    cache = cache_for([att], dtype)
    cuts_of = [[n], [2, 7, 63, 64, 65, n - 3, n] if n > 70 else [2, 7, n - 3, n], list(range(max(1, n - 75), n + 1)), list(range(1, min(n, 70))) + [n]]
    for cuts in cuts_of:
        close(in_steps(att, rt, cache, h, cuts), ref, tol)


LIGHTNING_GEOMETRIES = [  # heads, dim, vdim, rows
    (3, 24, 40, 150), (1, 18, 36, 131), (4, 64, 128, 300), (2, 128, 64, 520), (5, 33, 20, 140), (2, 200, 16, 270)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("geom", LIGHTNING_GEOMETRIES)
def test_lightning_alone_remembers_a_loud_token(dtype, tol, geom):
    """Token 5 is louder than the rest: slow heads still carry its value a hundred tokens later.  Whole, in portions down to one
    token, and the last forty tokens one by one; then in a slot that is used again."""
    from odin_infer_b200.parts import PartSpec, build_part
    H, D, V, n = geom
    width = 80
    rt = runtime(dtype)
    mx = lig(H, D, V)
    mixer = build_part("mixer", PartSpec("lightning", dict(width=width, n_heads=H, head_dim=D, v_head_dim=V, decay=mx["decay"], eps=1e-5,
                                                           names={s: "m." + s for s in ("q", "k", "v", "g", "norm", "o")})))
    w = bound(mixer, dtype, rt, H * 10 + D)
    torch.manual_seed(D)
    h = torch.randn(n, width, device=DEV)
    h[5] *= 6.0
    h = h.to(dtype)
    ref = P.lightning(h.double().cpu(), w, "m.", mx, 1e-5)
    quiet = h.clone()
    quiet[5] = quiet[6]
    other = P.lightning(quiet.double().cpu(), w, "m.", mx, 1e-5)
    assert (other[100] - ref[100]).abs().max() > 1e-2 * ref[100].abs().max()     # the loud token is still heard at row 100
    cache = cache_for([mixer], dtype)
    for cuts in CUTS(n):
        close(in_steps(mixer, rt, cache, h, cuts), ref, tol)
    close(in_steps(mixer, rt, cache, quiet, [n]), other, tol)   # the slot's state was cleared for the next sequence


UNIT_GEOMETRIES = [  # channels, blocks, taps, rows
    (60, 5, 3, 150), (33, 1, 1, 131), (42, 6, 6, 90), (256, 4, 4, 300), (128, 2, 2, 520), (512, 2, 5, 140), (700, 1, 4, 70)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("geom", UNIT_GEOMETRIES)
def test_gated_unit_alone_remembers_a_loud_token(dtype, tol, geom):
    """As for the recurrence over heads; a block's gates read their own channels only, and a convolution's memory that is lost
    (or has lost its inputs' bias) changes the rows after a cut, also where a portion is shorter than the convolution."""
    from odin_infer_b200.parts import PartSpec, build_part
    inner, blocks, taps, n = geom
    width = 80
    rt = runtime(dtype)
    names = {s + t: "m." + s + u for s in ("y", "x", "ra", "ri", "conv") for t, u in (("", ""), ("_bias", ".b"))}
    names.update(lam="m.lam", o="m.o")
    mixer = build_part("mixer", PartSpec("gated_linear_unit", dict(width=width, inner=inner, blocks=blocks, taps=taps, names=names)))

    def slow(t):
        t["m.lam"] -= 2.0
        t["m.conv"][:, -1] = 1.0
        t["m.x.b"] += 0.5
    w = bound(mixer, dtype, rt, inner + taps, slow)
    torch.manual_seed(inner)
    h = torch.randn(n, width, device=DEV)
    h[5] *= 12.0
    h = h.to(dtype)
    ref = P.gated_unit(h.double().cpu(), w, "m.")
    quiet = h.clone()
    quiet[5] /= 12.0
    other = P.gated_unit(quiet.double().cpu(), w, "m.")
    assert (other[60] - ref[60]).abs().max() > 1e-2 * ref[60].abs().max()
    cache = cache_for([mixer], dtype)
    for cuts in CUTS(n):
        close(in_steps(mixer, rt, cache, h, cuts), ref, tol)
    close(in_steps(mixer, rt, cache, quiet, [n]), other, tol)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 4e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("n,blocks,lens", [(60, 5, (200, 1, 64, 65)), (33, 1, (129, 66)), (256, 2, (300,)), (140, 7, (31, 32, 33, 97))])
def test_gated_unit_kernels(n, blocks, lens, dtype, tol):
    """The scan in blocks of several sizes, and token by token in the kernel that forms its own gates, against the recurrence:
    several sequences at once from states of zeros, then a second call that goes on; a padding sequence leaves its state, a
    channel whose decay is all but one keeps its digits."""
    from odin_infer_b200.csrc import ops
    torch.manual_seed(n)
    m, T = n // blocks, sum(lens)
    u, wide = torch.randn(T, n, device=DEV).to(dtype), torch.randn(T, n + 5, device=DEV).to(dtype)
    y, yb, gb = wide[:, 3:n + 3], torch.randn(n, device=DEV), torch.randn(blocks, 2 * m, device=DEV)
    w = (torch.randn(blocks, m, 2 * m, device=DEV) / m ** 0.5).to(dtype)
    lam = torch.randn(n, dtype=F64) - 3.0
    lam[0] = -14.0
    ld = (-8.0 * P.softplus(lam)).float().to(DEV)
    z = torch.einsum("tbi,bij->tbj", u.double().view(T, blocks, m), w.double())
    r, i = (torch.sigmoid(z + gb.double())[:, :, s * m:(s + 1) * m].reshape(T, n).cpu() for s in (0, 1))
    lam32 = torch.log(torch.expm1(ld.double().cpu() / -8.0))      # the decays as the kernels get them
    want, ends, at = [], [], 0
    for k in lens:
        S, last = P.gated_unit_walk(u[at:at + k].double().cpu(), r[at:at + k], i[at:at + k], lam32)
        want.append(S * P.gelu_tanh(y[at:at + k].double().cpu() + yb.double().cpu()))
        ends.append(last)
        at += k
    want, ends = torch.cat(want), torch.stack(ends)
    slots = torch.tensor(list(range(len(lens), 0, -1)) + [0], dtype=torch.int32, device=DEV)   # the last sequence is padding

    def scan(pieces, state, block_len):
        rows = torch.cat([torch.arange(sum(lens[:j]) + p0, sum(lens[:j]) + p1, device=DEV) for j, (p0, p1) in enumerate(pieces)])
        sizes = [p1 - p0 for p0, p1 in pieces] + [0]
        starts = torch.tensor([0] + np.cumsum(sizes).tolist(), dtype=torch.int32, device=DEV)
        o = torch.full((len(rows), n), float("nan"), dtype=dtype, device=DEV)
        ops.gated_unit_scan(u[rows].contiguous(), z.reshape(T, 2 * n)[rows].float().contiguous(), gb, ld, wide[rows][:, 3:n + 3], yb, state, o,
                            starts, slots, len(lens) + 1, max(sizes), block_len=block_len)
        close(o, want[rows.cpu()], tol)
    for block_len in (0, 16, 64, 1000):
        for cut in ([lambda k: (0, k)], [lambda k: (0, (k + 1) // 2), lambda k: ((k + 1) // 2, k)]):
            state = torch.zeros(len(lens) + 1, n + 3, device=DEV)
            state[0] = 7.0
            for piece in cut:
                if any(piece(k)[1] > piece(k)[0] for k in lens):
                    scan([piece(k) for k in lens], state, block_len)
            close(state[slots[:-1].long(), :n], ends, 4e-6)
            assert (state[0] == 7.0).all() and (state[1:, n:] == 0).all()
    # one token of every sequence at a time, a padding row among them
    state, firsts = torch.zeros(len(lens) + 1, n + 3, device=DEV), np.cumsum((0,) + lens[:-1])
    for t in range(max(lens)):
        live = [j for j, k in enumerate(lens) if t < k]
        rows = torch.tensor([int(firsts[j]) + t for j in live] + [0], device=DEV)
        tok_seq = torch.tensor(list(range(len(live))) + [-1], dtype=torch.int32, device=DEV)
        o = torch.full((len(rows), n), 5.0, dtype=dtype, device=DEV)
        ops.gated_unit_step(u[rows].contiguous(), w, gb, ld, wide[rows][:, 3:n + 3], yb, state, o, tok_seq, slots[live].contiguous())
        close(o[:-1], want[rows[:-1].cpu()], tol * 3)
        assert (o[-1] == 5.0).all()
    close(state[slots[:-1].long(), :n], ends, 4e-6)


@pytest.mark.parametrize("rows", [1, 9, 20])
def test_gated_unit_step_of_many_rows(rows):
    """More rows than a CTA takes, slots in another order."""
    from odin_infer_b200.csrc import ops
    n, blocks = 96, 2
    m = n // blocks
    torch.manual_seed(rows)
    u, y = torch.randn(rows, n, device=DEV), torch.randn(rows, n, device=DEV)
    w, gb = torch.randn(blocks, m, 2 * m, device=DEV) / m ** 0.5, torch.randn(blocks, 2 * m, device=DEV)
    lam, yb = torch.randn(n, device=DEV) - 3, torch.randn(n, device=DEV)
    ld = -8.0 * torch.nn.functional.softplus(lam)
    state = torch.randn(rows, n, device=DEV)
    before = state.double().cpu()
    slots = torch.randperm(rows, generator=torch.Generator().manual_seed(1)).int().to(DEV)
    o = torch.empty(rows, n, device=DEV)
    z = torch.sigmoid(torch.einsum("tbi,bij->tbj", u.double().view(rows, blocks, m), w.double()) + gb.double())
    r, i = (z[:, :, s * m:(s + 1) * m].reshape(rows, n).cpu() for s in (0, 1))
    ops.gated_unit_step(u, w, gb, ld, y, yb, state, o, torch.arange(rows, dtype=torch.int32, device=DEV), slots)
    for t in range(rows):
        S, _ = P.gated_unit_walk(u[t:t + 1].double().cpu(), r[t:t + 1], i[t:t + 1], lam.double().cpu(), before[int(slots[t])])
        close(o[t], S[0] * P.gelu_tanh(y[t].double().cpu() + yb.double().cpu()), 4e-6)
        close(state[int(slots[t])], S[0], 4e-6)


@pytest.mark.parametrize("blocks", [0, 32])
@pytest.mark.parametrize("H,dk,dv,lens", [(3, 24, 40, (70, 1, 33)), (2, 64, 64, (130, 64)), (1, 130, 16, (90,)), (4, 128, 128, (65, 40))])
def test_fixed_decay_recurrence_between_silus(H, dk, dv, lens, blocks):
    from odin_infer_b200.csrc import ops
    torch.manual_seed(H + dk)
    T = sum(lens)
    x = torch.randn(T, H * (2 * dk + dv) + 3, device=DEV)
    q, k, v = x[:, :H * dk], x[:, H * dk:2 * H * dk], x[:, 2 * H * dk:H * (2 * dk + dv)]
    decay = torch.linspace(0.5, 0.999, H)
    state, o = torch.zeros(len(lens), H * dk * dv, device=DEV), torch.empty(T, H * dv, device=DEV)
    starts = torch.tensor([0] + np.cumsum(lens).tolist(), dtype=torch.int32, device=DEV)
    slots = torch.arange(len(lens), dtype=torch.int32, device=DEV)
    ops.linear_recurrence("fixed_silu", q, k, None, v, decay.to(DEV), decay.to(DEV), o, state, starts, slots, len(lens), H, dk, dv,
                          block_len=blocks, max_new=max(lens))
    at = 0
    for j, n in enumerate(lens):
        st = [torch.zeros(dk, dv, dtype=F64) for _ in range(H)]
        qq, kk, vv = (P.silu(t[at:at + n].double().cpu()) for t in (q, k, v))
        want = P.decay_walk(qq.view(n, H, dk), kk.view(n, H, dk), vv.view(n, H, dv), decay.double().tolist(), st)
        close(o[at:at + n], want.reshape(n, -1), 6e-6)
        close(state[j], torch.stack(st).reshape(-1), 6e-6)
        at += n


@pytest.mark.parametrize("silu", [False, True])
@pytest.mark.parametrize("H,dk,dv,lens", [(3, 24, 40, (200, 1, 129)), (2, 64, 64, (256, 64)), (1, 130, 16, (300,)), (4, 128, 128, (140, 385)),
                                          (2, 33, 70, (128, 130)), (1, 256, 200, (190,)), (5, 8, 132, (63, 64, 65, 127))])
def test_fixed_decay_recurrence_as_products_of_tiles(H, dk, dv, lens, silu):
    """Blocks of 128 tokens: several sequences at once from states of zeros, then a second call that goes on; a padding
    sequence leaves its state.  Decays from one that forgets at once to one that keeps everything; an early row is loud."""
    from odin_infer_b200.csrc import ops
    torch.manual_seed(H + dk + dv)
    T = sum(lens)
    pad = 4 if dk % 4 == 0 else 3
    x = torch.randn(T, H * (2 * dk + dv) + pad, device=DEV)
    x[3] *= 10.0
    decay = torch.tensor([0.0, 1.0, 0.999, 0.9, 0.5][:H] if H > 1 else [0.995])
    slots = torch.tensor(list(range(len(lens), 0, -1)) + [0], dtype=torch.int32, device=DEV)   # the last sequence is padding
    want, ends, at = [], [], 0
    act = P.silu if silu else (lambda t: t)
    for n in lens:
        st = [torch.zeros(dk, dv, dtype=F64) for _ in range(H)]
        qq, kk, vv = (act(t.double().cpu()) for t in x[at:at + n, :H * (2 * dk + dv)].split([H * dk, H * dk, H * dv], dim=1))
        want.append(P.decay_walk(qq.view(n, H, dk), kk.view(n, H, dk), vv.view(n, H, dv), decay.double().tolist(), st).reshape(n, -1))
        ends.append(torch.stack(st).reshape(-1))
        at += n
    want, ends = torch.cat(want), torch.stack(ends)
    for cut in ([lambda k: (0, k)], [lambda k: (0, (2 * k + 2) // 3), lambda k: ((2 * k + 2) // 3, k)]):
        state = torch.zeros(len(lens) + 1, H * dk * dv + 3, device=DEV)
        state[0] = 7.0
        for piece in cut:
            pieces = [piece(k) for k in lens]
            rows = torch.cat([torch.arange(sum(lens[:j]) + p0, sum(lens[:j]) + p1, device=DEV) for j, (p0, p1) in enumerate(pieces)])
            if len(rows) == 0:
                continue
            sizes = [p1 - p0 for p0, p1 in pieces] + [0]
            starts = torch.tensor([0] + np.cumsum(sizes).tolist(), dtype=torch.int32, device=DEV)
            xr, o = x[rows].contiguous(), torch.full((len(rows), H * dv), float("nan"), device=DEV)
            ops.decay_blocks(xr[:, :H * dk], xr[:, H * dk:2 * H * dk], xr[:, 2 * H * dk:H * (2 * dk + dv)], decay.to(DEV), o, state, starts, slots,
                             len(lens) + 1, H, dk, dv, max(sizes), silu=silu)
            close(o, want[rows.cpu()], 4e-6)
        close(state[slots[:-1].long(), :H * dk * dv], ends, 4e-6)
        assert (state[0] == 7.0).all() and (state[1:, H * dk * dv:] == 0).all()


@pytest.mark.parametrize("T", [1, 70])
@pytest.mark.parametrize("n,pad", [(96, 0), (100, 2), (33, 1), (2048, 4), (4100, 8), (9000, 0)])
def test_norm_over_the_whole_row_then_a_sigmoid_gate(n, pad, T):
    from odin_infer_b200.csrc import ops
    torch.manual_seed(n)
    o, z, w = torch.randn(T, n, device=DEV), torch.randn(T, n + pad, device=DEV), torch.randn(n, device=DEV)
    o[0] *= 1e-3                                   # eps counts
    want = P.rms(o.double().cpu(), w.double().cpu(), 1e-6) * torch.sigmoid(z[:, pad:].double().cpu())
    for zd, od, tol in ((torch.float32, torch.float32, 2e-6), (torch.float32, torch.bfloat16, 5e-3), (torch.bfloat16, torch.bfloat16, 2e-2)):
        out = torch.empty(T, n, dtype=od, device=DEV)
        ops.skip_gate_norm(o, None, None, 1, z.to(zd)[:, pad:], w, 1, 1e-6, out, sigmoid_after=True)
        close(out, want, tol)


@pytest.mark.parametrize("T", [5, 70, 300])
@pytest.mark.parametrize("C,taps", [(60, 3), (33, 1), (300, 4), (40, 6)])
def test_convolution_with_a_bias_on_its_inputs(C, taps, T):
    """Zeros, not the bias, stand before a sequence's start; the memory holds the inputs with their bias."""
    from odin_infer_b200.csrc import ops
    torch.manual_seed(C + T)
    x, w = torch.randn(T, C + 7, device=DEV), torch.randn(C, taps, device=DEV)
    b, ib = torch.randn(C, device=DEV), torch.randn(C, device=DEV) + 3.0
    cut = max(1, T // 3)
    want = P.causal_conv((x[:, 7:].double() + ib.double()).cpu(), w.double().cpu(), b.double().cpu())
    slots, state = torch.tensor([1], dtype=torch.int32, device=DEV), torch.zeros(2, max(taps - 1, 1) * C, device=DEV)
    for r0, r1 in ((0, cut), (cut, T - 1), (T - 1, T)):
        if r1 <= r0:
            continue
        out = torch.empty(r1 - r0, C, device=DEV)
        ops.causal_conv(x[r0:r1, 7:], w, b, False, state, torch.zeros(r1 - r0, dtype=torch.int32, device=DEV),
                        torch.tensor([0, r1 - r0], dtype=torch.int32, device=DEV), slots, 1, out, single_rows=r1 - r0 == 1, in_bias=ib)
        close(out, want[r0:r1], 3e-6)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("s", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("d,rows", [(96, 9), (100, 3), (33, 4), (2048, 140), (4096, 3), (8192, 2), (8196, 2), (1028, 200)])
def test_streams_kernel(d, rows, s, dtype, tol):
    """An update of partial sums with a bias, of two normed terms with factors, and none at all; the streams in place, and left
    alone where rows are gathered; the norm of what is read."""
    from odin_infer_b200.csrc import ops
    torch.manual_seed(d + s)
    x = torch.randn(s, rows, d, device=DEV)
    mix, add, read = torch.randn(s, s, device=DEV), torch.randn(s, device=DEV), torch.randn(s, device=DEV)
    w, w1, b = torch.randn(d, device=DEV), torch.randn(d, device=DEV).to(torch.bfloat16), torch.randn(d, device=DEV)
    u, v = torch.randn(3, rows, d, device=DEV), torch.randn(rows, d, device=DEV)
    X, cp = x.double().cpu(), lambda t: t.double().cpu()  # noqa: E731
    t1 = cp(u).sum(0) + cp(b)
    updates = [([], None), ([ops.Term(u)], cp(u).sum(0)), ([ops.Term(u, bias=b)], t1),
               ([ops.Term(u, 0.5, None, w1, 1e-3, b), ops.Term(v, -0.75, None, w, 1e-5)],
                0.5 * P.rms(t1, cp(w1), 1e-3) - 0.75 * P.rms(cp(v), cp(w), 1e-5))]
    for terms, y in updates:
        new = X if y is None else P.hyper(X, cp(mix), cp(add), y)
        want = P.rms(P.read_streams(new, cp(read)), cp(w), 1e-4)
        x1, out = x.clone(), torch.empty(rows, d, dtype=dtype, device=DEV)
        ops.mix_streams(x1, terms, mix, add, read, w, 1e-4, out)
        close(out, want, tol)
        close(x1, new, 2e-6)
        if y is None:
            assert torch.equal(x1, x)
        pick = torch.tensor([rows - 1, 0, rows - 1], dtype=torch.int32, device=DEV)
        x2, got = x.clone(), torch.empty(3, d, dtype=dtype, device=DEV)
        ops.mix_streams(x2, terms, mix, add, read, w, 1e-4, got, rows=pick)
        close(got, want[pick.long().cpu()], tol)
        assert torch.equal(x2, x)


@pytest.mark.parametrize("d", [96, 100, 33, 4096])
def test_a_bias_on_a_term_of_one_stream(d):
    from odin_infer_b200.csrc import ops
    torch.manual_seed(d)
    x, u, b, w = torch.randn(5, d, device=DEV), torch.randn(2, 5, d, device=DEV), torch.randn(d, device=DEV), torch.randn(d, device=DEV)
    want = x.double() + P.rms(u.double().sum(0) + b.double(), w.double(), 1e-5) + 2.0 * (u[0].double() + b.double())
    out = torch.empty(5, d, device=DEV)
    ops.combine_add(x, [ops.Term(u, 1.0, None, w, 1e-5, b), ops.Term(u[0], 2.0, bias=b)], None, 0.0, w, 1e-5, out)
    close(x, want, 2e-6)
    close(out, P.rms(want, w.double(), 1e-5), 2e-6)


@pytest.mark.parametrize("streams", [1, 4])
@pytest.mark.parametrize("with_pair", [True, False])
def test_embedding_starts_every_stream(streams, with_pair):
    from odin_infer_b200.cache import CacheManager
    from odin_infer_b200.engine.step import StepBatch, StepEntry
    from odin_infer_b200.parts import PartSpec, build_part
    rt = runtime(torch.bfloat16)
    V, d = 40, 36
    pair = {"weight": "bigram", "buckets": 13, "mul_prev": 7, "mul_cur": 4} if with_pair else None
    part = build_part("embedding", PartSpec("token_table", dict(vocab_size=V, width=d, weight="embed", scale=1.5, pair=pair, streams=streams)))
    w = bound(part, torch.bfloat16, rt, 3)
    cache = CacheManager(64 * 4, 64 * 2)
    part.state_entry = cache.add_entry(None, part.state_bytes()) if with_pair else None
    cache.state = torch.full((cache.max_slots, max(cache.state_bytes_per_slot, 1)), 0x7f, dtype=torch.uint8, device=DEV)
    cache.zero_state = lambda slot: cache.state[slot].zero_()
    toks = random_tokens(21, V, 5)
    cfg = {"embedding": {"scale": 1.5, "bigram": pair}}
    want = P.embed(cfg, w, toks) if with_pair else 1.5 * w["embed"][toks]
    slot, at = cache.take_slot(), 0
    for end in (9, 11, 12, 13, 21):
        st = cache.extend(slot, end - at)
        x = part.forward(rt, StepBatch(cache, [StepEntry(slot, toks[at:end], [])], [st], DEV))
        assert tuple(x.shape) == (streams, end - at, d)
        for k in range(streams):
            close(x[k], want[at:end], 1e-6)
        at = end


@pytest.mark.parametrize("T", [3, 40, 200])
@pytest.mark.parametrize("splits", [1, 3])
def test_product_per_head_with_a_gate_per_element(T, splits):
    from odin_infer_b200.csrc import ops
    H, K, N = 5, 37, 70
    torch.manual_seed(T)
    wide = torch.randn(splits, T, H * K + 11 + H * N, device=DEV)
    w = torch.randn(H, K, N, device=DEV) / K ** 0.5
    a, gate = (wide[..., :H * K], wide[..., H * K + 11:]) if splits > 1 else (wide[0][:, :H * K], wide[0][:, H * K + 11:])
    summed = wide.double().sum(0)
    want = torch.einsum("thk,hkn->thn", summed[:, :H * K].view(T, H, K), w.double()) * torch.sigmoid(summed[:, H * K + 11:].view(T, H, N))
    out = torch.empty(T, H * N, device=DEV)
    ops.heads_linear(a, K, w, out, N, gate=gate)
    close(out.view(T, H, N), want, 3e-6)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("T", [128, 300])
@pytest.mark.parametrize("H,K,N,off", [(3, 64, 40, 0), (5, 128, 264, 8), (1, 192, 128, 3), (2, 64, 33, 0), (4, 64, 64, 16)])
def test_product_per_head_on_the_tensor_cores_with_a_gate_per_element(T, H, K, N, off, dtype):
    """Outputs in bfloat16 and in 32-bit, with and without gates, which lie at any offset of wider rows."""
    from odin_infer_b200.csrc import ops
    torch.manual_seed(T + K)
    a = torch.randn(T, H * K, device=DEV).to(torch.bfloat16)
    w = (torch.randn(H, N, K, device=DEV) / K ** 0.5).to(torch.bfloat16)
    want = torch.einsum("thk,hnk->thn", a.double().view(T, H, K), w.double())
    gates = [None, torch.randn(2, T, H * N + off, device=DEV)[..., off:], torch.randn(T, H * N + off, device=DEV).to(torch.bfloat16)[:, off:]]
    for g in gates:
        out = torch.full((T, H * (N + 2)), 7.0, dtype=dtype, device=DEV)
        ops.heads_linear_tc(a, K, w, out, N + 2, gate=g)
        got = out.view(T, H, N + 2)
        f = 1.0 if g is None else torch.sigmoid(g.double().sum(0) if g.dim() == 3 else g.double()).view(T, H, N)
        close(got[:, :, :N], want * f, 5e-3 if dtype == torch.bfloat16 else 3e-6)
        assert (got[:, :, N:] == 7.0).all()
    ops.moe_tc_check()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("n", [3, 150, 300])
def test_two_branches_side_by_side_with_norms_and_a_bias(dtype, tol, n):
    """Attention (whose output has a bias) beside the gated unit, through the parts, in whole prompts and one by one."""
    from odin_infer_b200.config import config_from_dict, lookup_architecture
    from odin_infer_b200.parts import build_part
    raw = model(50, 80, 2, 1e-5, (par(4, 2, 24, 0.3, 40, 8, 96, 3, 4), None))
    spec = lookup_architecture("Bafilorn").build_spec(config_from_dict(raw))
    rt = runtime(dtype)
    mixer = build_part("mixer", spec.layers[0].args["mixer"])
    (pe,) = spec.position_encodings.values()
    mixer.pe = build_part("position_encoding", pe)
    mixer.pe.prepare(rt, n)
    w = bound(mixer, dtype, rt, 77)
    torch.manual_seed(n)
    h = torch.randn(n, 80, device=DEV).to(dtype)
    ref = P.parallel(h.double().cpu(), w, "l0.mix.", raw["layers"][0]["mixer"], 1e-5)
    cache = cache_for([mixer], dtype)
    for cuts in ([n], list(range(max(1, n - 50), n + 1))):
        close(in_steps(mixer, rt, cache, h, cuts), ref, tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hd,rot,T,parts", [(24, 8, 30, 1), (64, 32, 9, 3), (128, 128, 300, 1), (64, 64, 70, 2), (33, 2, 5, 1)])
def test_head_preparation_of_values_that_are_keys(dtype, hd, rot, T, parts):
    """The value cache holds the keys with their bias before they turn, the key cache the turned ones; scrambled pages, and a
    padding row that writes nothing."""
    from odin_infer_b200.csrc import ops
    Hq, Hkv = 4, 2
    torch.manual_seed(hd + T)
    src = torch.randn(parts, T, (Hq + Hkv) * hd + 5, device=DEV) if parts > 1 else torch.randn(T, (Hq + Hkv) * hd + 5, device=DEV).to(dtype)
    bias = torch.randn((Hq + Hkv) * hd, device=DEV).to(dtype)
    x = (src.double().sum(0) if parts > 1 else src.double())[:, :(Hq + Hkv) * hd] + bias.double()
    n_pages = (T + 63) // 64
    bt = torch.arange(n_pages, dtype=torch.int32, device=DEV).flip(0).contiguous().view(1, -1)
    pos, seq = torch.arange(T, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV)
    seq[T - 1] = -1
    f, gain = P.frequencies(rot, 1e3, {"factor": 4.0, "original": 100.0, "fast": 8.0, "slow": 1.0})
    ang = torch.arange(T, dtype=F64)[:, None] * torch.tensor(f, dtype=F64)
    cos, sin = (torch.cos(ang) * gain).float().to(DEV), (torch.sin(ang) * gain).float().to(DEV)
    kc, vc = (torch.full((n_pages, Hkv, 64, hd), 3.0, dtype=dtype, device=DEV) for _ in range(2))
    q = ops.head_prep(src, Hq, Hkv, hd, None, None, 1e-5, cos, sin, rot, pos, seq, bt, kc, vc,
                      q_out=torch.empty(T, Hq * hd, dtype=dtype, device=DEV), bias=bias, values_are_keys=True)
    turned = P.rotate(x.cpu().view(T, Hq + Hkv, hd), range(T), rot, 1e3, False, {"factor": 4.0, "original": 100.0, "fast": 8.0, "slow": 1.0})
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    close(q[:T - 1].view(T - 1, Hq, hd), turned[:T - 1, :Hq], tol)
    for c, want in ((kc, turned[:, Hq:]), (vc, x.cpu().view(T, Hq + Hkv, hd)[:, Hq:])):
        close(torch.stack([c[int(bt[0, t // 64]), :, t % 64] for t in range(T - 1)]), want[:T - 1], tol)
        assert (c[int(bt[0, (T - 1) // 64]), :, (T - 1) % 64] == 3.0).all()


@pytest.mark.parametrize("engine_type", ["float32", "bfloat16"])
def test_random_weights_run(engine_type):
    """An engine from a seed (no folder) generates."""
    from odin_infer_b200 import Engine, Engine_Opts
    from odin_infer_b200.config import config_from_dict
    engine = Engine.random(config_from_dict(FAST), 3, Engine_Opts(max_ctx=256, max_batch=2, dtype=engine_type, verbose=False))
    outs = engine.generate([[1, 2, 3], [5] * 40], max_new_tokens=4, temperature=0.0, stop_token_ids=[])
    assert [len(o.tokens) for o in outs] == [4, 4]
    engine.destroy()
