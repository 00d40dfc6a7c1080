"""The Fugavik decoder through the engine against its plain implementation (tests/plain/fugavik_plain.py): every mechanism
alone, whole prompts against token-by-token decoding, prompts in portions, unequal batches, slots, pages and states that are
used again, the first tokens of a sequence, long decoding, sizes that the fast kernels take and sizes that they do not, and
greedy generation through the engine's own entry point.  The tests write their own weights and inputs (matrices of unit gain,
decays that remember for hundreds of tokens, a key far back that one query asks for, sinks and scales that differ from head to
head and channel to channel) so that a lost state, a sink that is left out or a value that is not mixed leaves a mark far above
rounding."""
import json
import math
import os

import numpy as np
import pytest
import torch

from tests import traces
from tests.plain import fugavik_plain as P
from tests.test_meropel_gpu import CUTS, cache_for, close, engine_for, portions, replay, requests_for, run_in_steps, runtime, summed
from tests.tiny import TOL, random_tokens

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def attn(heads, kv, dim, vdim, scale, rot=0, base=1e4, factor=None, v_mix=False):
    out = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if rot:
        out["rot"] = {"dims": rot, "base": base}
        if factor is not None:
            out["rot"]["scaling"] = {"factor": factor}
    return out


def lat(heads, dim, vdim, rank, scale):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale}


def dlt(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def model(vocab, width, eps, *layers):
    kinds = {"kv_rank": "latent_attention", "conv": "delta"}
    return {"architecture": "Fugavik", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": next((t for k, t in kinds.items() if k in mx), "attention"), "mixer": mx, "mlp": mlp}
                       for mx, mlp in layers]}


# odd sizes throughout; three layers that mix values around one of other sizes that does not; partial, full and no rotation;
# layers without feed-forward; one expert and several per token
MIXED = model(211, 96, 1e-5,
              (dlt(4, 2, 24, 40, 3), moe(6, 3, 40)),
              (attn(4, 2, 24, 40, 0.35, rot=8, base=300.0, factor=1.7, v_mix=True), dense(80)),
              (lat(3, 20, 28, 48, 0.3), None),
              (attn(3, 3, 16, 16, 0.4), moe(5, 1, 24)),
              (attn(6, 2, 32, 40, 0.3, rot=32, base=5e5, factor=4.0, v_mix=True), None),
              (dlt(3, 3, 20, 12, 2), dense(56)),
              (attn(2, 2, 36, 40, 0.25, rot=12, base=50.0, v_mix=True), moe(4, 4, 16)))
# a width that is no multiple of 8; one head; a convolution of one tap and of five; keys that are no multiple of four
ODD = model(97, 100, 1e-6,
            (lat(1, 36, 12, 20, 0.2), moe(3, 3, 20)),
            (dlt(1, 1, 18, 36, 1), None),
            (attn(3, 1, 20, 28, 0.22, rot=20, base=900.0, factor=0.5, v_mix=True), dense(52)),
            (dlt(6, 2, 33, 9, 5), moe(4, 1, 28)))
# head sizes the tensor-core attention kernels take, widths the tensor-core products take
FAST = model(384, 128, 1e-5,
             (dlt(4, 2, 64, 128, 4), moe(12, 2, 64)),
             (attn(4, 2, 64, 64, 0.15, rot=64, base=1e4, factor=8.0, v_mix=True), dense(256)),
             (lat(8, 64, 32, 128, 0.12), moe(9, 1, 128)),
             (attn(2, 2, 128, 64, 0.1, rot=64, base=1e6, factor=2.5, v_mix=True), dense(176)),
             (attn(8, 2, 64, 64, 0.15, rot=64, base=1e4, factor=8.0, v_mix=True), None),
             (dlt(2, 1, 128, 64, 4), dense(128)))
CONFIGS = {"mixed": (MIXED, 3), "odd": (ODD, 5), "fast": (FAST, 7)}


def make_weight(name: str, shape, gen) -> torch.Tensor:
    """Weights of the tests' own making: matrices N(0, 1/in), norm weights around one with biases, scales on the sublayers'
    outputs around a half, a router of gain 3, sinks around the scores' own size, decays that remember for tens to hundreds
    of tokens."""
    r = torch.randn(shape, generator=gen)
    last = name.rsplit(".", 1)[-1]
    if last in ("norm", "norm1", "norm2"):
        return 1.0 + 0.3 * r
    if last == "b" and len(shape) == 1:
        return 0.3 * r
    if last in ("ls1", "ls2"):
        return 0.5 + 0.25 * r
    if last == "vmix":
        return 0.5 + 0.2 * r
    if last == "sink":
        return 1.0 + 1.5 * r
    if last == "embed":
        return r
    if last == "router":
        return 3.0 * r / math.sqrt(shape[1])
    if last == "conv":
        return 0.6 * r
    if last == "dt_bias":
        return -4.0 + 1.5 * r
    if last == "A_log":
        return -0.5 + 0.8 * r
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
        base = tmp_path_factory.mktemp("fugavik")
        for name, (raw, seed) in CONFIGS.items():
            _folders[name] = write_model(os.path.join(str(base), name), raw, seed)
    return _folders


_plain = {}


def plain_logits(folder, tokens, rounded=None, swapped=()):
    """rounded: None (exact), "bfloat16" or "float32": what an engine of that type stores between kernels is rounded to it;
    swapped: (layer, token) pairs whose router takes its closest call the other way."""
    key = (folder, tuple(tokens), rounded, tuple(swapped))
    if key not in _plain:
        cfg, w = P.read_model_folder(folder, F64)
        rnd = {None: lambda t: t, "bfloat16": P.to_bfloat16_and_back, "float32": lambda t: t.float().double()}[rounded]
        _plain[key] = P.forward(cfg, w, tokens, rnd=rnd, swapped=swapped).numpy()
    return _plain[key]


def close_calls(folder, tokens, upto: int, gap: float = 0.12):
    """(layer, token) pairs up to and with token `upto` whose router decides by less than `gap`, the closest first."""
    cfg, w = P.read_model_folder(folder, F64)
    gaps: dict = {}
    P.forward(cfg, w, tokens[:upto + 1], gaps=gaps)
    found = [(float(g[t]), (layer, t)) for layer, g in gaps.items() if g is not None for t in range(len(g)) if float(g[t]) < gap]
    return [pair for _, pair in sorted(found)]


# The 32-bit engine is held to the tolerance at every position, or to five times what rounding to 32 bits alone does there
# where that is more.  In bfloat16 the yardstick is what rounding alone does to this model and these tokens (the plain
# implementation run again with what a 16-bit engine stores rounded to bfloat16): a position's limit is the tolerance or
# three times the rounding's own error there, one position in ten may be over it, and the median stays within twice the
# rounding's median.  A router's close call at one of a sequence's first tokens that falls the other way moves every later
# position (few keys and a young state share it): a request that is over its limits must then be within them against the plain
# implementation that takes one such close call, at or before the first position over its limit, the other way.
def within(rows, ref, noise_ref, dtype):
    """(whether the rows are within their limits, the first position over its own, a text)."""
    n, top = rows.shape[0], max(np.abs(ref).max(), 1e-30)
    err = np.abs(rows.astype(np.float64) - ref).max(axis=1) / top
    noise = np.abs(noise_ref - ref).max(axis=1) / top
    over = np.flatnonzero(err > np.maximum(TOL[dtype], (5.0 if dtype == "float32" else 3.0) * noise))
    text = (f"{len(over)} of {n} positions over their limit, median {np.median(err):.3e} (rounding alone {np.median(noise):.3e}), "
            f"worst {err.max():.3e} at {int(err.argmax())} (rounding alone {noise.max():.3e})")
    if dtype == "float32":
        return len(over) == 0, int(over[0]) if len(over) else n, text
    mid = max(TOL[dtype] / 4, 2.0 * float(np.median(noise)))
    ok = len(over) <= max(2, n // 10) and err.max() <= max(2.0, 3.0 * noise.max()) and np.median(err) <= mid
    return ok, int(over[0]) if len(over) else n, text


def check_rows(got: dict, folder, requests, dtype):
    for rid, rows in got.items():
        n, toks = rows.shape[0], requests[rid]
        ok, first, text = within(rows, plain_logits(folder, toks)[:n], plain_logits(folder, toks, rounded=dtype)[:n], dtype)
        if not ok and dtype == "bfloat16":
            for pair in close_calls(folder, toks, first)[:4]:
                ok = ok or within(rows, plain_logits(folder, toks, swapped=(pair,))[:n],
                                  plain_logits(folder, toks, rounded=dtype, swapped=(pair,))[:n], dtype)[0]
        assert ok, f"{rid}: {text}, first over at {first}"


# --------------------------------------------------------------------------------------
# the whole model in every cut
# --------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_and_one_by_one(folders, name, dtype):
    """Whole prompts (across several pages, and with the delta rule chunk by chunk), then the same with the last tokens one by
    one, so that states and the convolutions' last inputs pass from the prompt's kernels to the single-token ones; the first
    tokens of a sequence alone (prompts of 1 and 2)."""
    raw = CONFIGS[name][0]
    reqs = requests_for(raw, [1, 2, 131, 260])
    engine = engine_for(folders[name], dtype)
    check_rows(traces.collect(traces.whole(reqs), replay(engine, traces.whole(reqs))), folders[name], reqs, dtype)
    recs = traces.tail_one_by_one(reqs, tail=70)
    check_rows(traces.collect(recs, replay(engine, recs)), folders[name], reqs, dtype)
    engine.cache.check()
    assert all(g.pool.n_held == 0 for g in engine.cache.groups.values())
    engine.destroy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,sizes", [("mixed", (2, 35, 3, 64)), ("odd", (17, 2, 2, 90)), ("fast", (130, 2, 70, 1, 129)),
                                        ("mixed", (2,)), ("odd", (1, 3))])
def test_prompts_in_portions(folders, name, sizes, dtype):
    """Portions of several sizes, down to two tokens and one: a portion starts from the states and the convolutions' last
    inputs (also when the portion is shorter than the convolution) that the portion before it left."""
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
        assert np.array_equal(alone[rid], both[rid]), rid
    engine.destroy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "fast"])
def test_long_decoding(folders, name, dtype):
    """Two hundred and fifty tokens decoded one by one after a short prompt: every state is carried as often, the keys grow
    over page borders."""
    raw = CONFIGS[name][0]
    reqs = requests_for(raw, [262, 250], seed=50)
    recs = traces.batches(reqs, 2, first_part=lambda n: 12)
    engine = engine_for(folders[name], dtype)
    check_rows(traces.collect(recs, replay(engine, recs)), folders[name], reqs, dtype)
    assert all(g.pool.n_held == 0 for g in engine.cache.groups.values())
    engine.destroy()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt(folders, dtype):
    """A prompt of 1,100 tokens whole, and with its last 40 tokens one by one: many chunks of the delta rule, experts with
    several tiles of rows each, keys many pages back."""
    raw = CONFIGS["fast"][0]
    reqs = requests_for(raw, [1100], seed=70)
    engine = engine_for(folders["fast"], dtype, max_tokens=2048, max_ctx=1280)
    for recs in (traces.whole(reqs), traces.tail_one_by_one(reqs, tail=40)):
        check_rows(traces.collect(recs, replay(engine, recs)), folders["fast"], reqs, dtype)
    engine.cache.check()
    engine.destroy()


def test_what_a_sequence_holds(folders):
    """Attention layers with equal heads share a group of the cache, a latent layer keeps one row per token, and the state area
    holds every delta layer's state and its convolution's last inputs."""
    engine = engine_for(folders["mixed"], "float32")
    kept = sorted((g.request.n_kv_heads, g.request.head_dim, g.request.value_dim, g.n_lines) for g in engine.cache.groups.values())
    assert kept == [(1, 48, 48, 1), (2, 24, 40, 1), (2, 32, 40, 1), (2, 36, 40, 1), (3, 16, 16, 1)], kept
    assert engine.cache.state_bytes_of == [4 * (4 * 24 * 40 + 2 * (2 * 48 + 160)), 0, 0, 0, 0, 4 * (3 * 20 * 12 + 120 + 36), 0]
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
    def off(p, o, swapped=()):
        ref = plain_logits(folders[name], p + o.tokens, swapped=swapped)[len(p) - 1:]
        return [i for i, tok in enumerate(o.tokens) if float(ref[i].max() - ref[i][tok]) > margin * float(np.abs(ref[i]).max())]
    for p, o in zip(prompts, outs):
        assert len(o.tokens) == 12
        wrong = off(p, o)
        if wrong and dtype == "bfloat16":     # a router's close call that fell the other way, and nothing else
            for pair in close_calls(folders[name], p + o.tokens, len(p) - 1 + wrong[0])[:6]:
                wrong = min(wrong, off(p, o, (pair,)), key=len)
        assert len(wrong) <= (1 if dtype == "bfloat16" else 0), (len(p), wrong)
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
    mixed = (pick(1, 2, 3), pick(8, 16, 40, 64))        # kv heads and value size of the layers that mix values

    def mixer():
        kind = pick("attention", "attention", "latent", "delta")
        if kind == "latent":
            return lat(pick(1, 2, 5), pick(8, 20, 64), pick(8, 24, 64), pick(16, 33, 64), float(rng.uniform(0.1, 0.4)))
        if kind == "delta":
            kv = pick(1, 2, 3)
            return dlt(kv * pick(1, 2, 3), kv, pick(8, 18, 32, 70), pick(8, 20, 33), pick(1, 2, 3, 4, 6))
        mix = pick(True, True, False)
        kv, vdim = mixed if mix else (pick(1, 2), pick(8, 24))
        dim = pick(8, 24, 64)
        return attn(kv * pick(1, 2, 4), kv, dim, vdim, float(rng.uniform(0.1, 0.4)), rot=pick(0, 4, dim // 2, dim),
                    base=pick(50.0, 1e4, 1e6), factor=pick(None, 0.7, 3.0, 16.0), v_mix=mix)

    def mlp():
        kind = pick(None, "dense", "moe", "moe")
        if kind is None:
            return None
        if kind == "dense":
            return dense(pick(24, 40, 64))
        n = pick(1, 3, 6)
        return moe(n, int(rng.integers(1, n + 1)), pick(16, 24, 32))
    return model(int(rng.integers(50, 300)), pick(64, 72, 100, 128), pick(1e-5, 1e-6, 1e-3),
                 *[(mixer(), mlp()) for _ in range(int(rng.integers(2, 6)))])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", [401, 402, 403, 404, 405, 406, 407, 408])
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


def delta_inputs(lens, H, G, dk, dv, seed, memory=-4.0):
    torch.manual_seed(seed)
    T = sum(lens)
    q, k, v = torch.randn(T, G * dk, device=DEV), torch.randn(T, G * dk, device=DEV), torch.randn(T, H * dv, device=DEV)
    a, b = torch.randn(T, H, device=DEV), torch.randn(T, H, device=DEV)
    return q, k, v, a, b, 0.7 * torch.randn(H, device=DEV) - 0.5, torch.randn(H, device=DEV) + memory


def delta_reference(x, lens, H, G, dk, dv):
    q, k, v, a, b, A, bias = (t.double().cpu() for t in x)
    out, states, at = [], [], 0
    for n in lens:
        s = slice(at, at + n)
        at += n
        spread = lambda t: P.unit(t[s].view(n, G, dk).repeat_interleave(H // G, dim=1))  # noqa: E731
        st = [torch.zeros(dk, dv, dtype=F64) for _ in range(H)]
        o = P.delta_walk(spread(q) * dk ** -0.5, spread(k), v[s].view(n, H, dv), torch.sigmoid(b[s]),
                         torch.exp(-torch.exp(A) * P.softplus(a[s] + bias)), st)
        out.append(o.reshape(n, H * dv))
        states.append(torch.stack(st).reshape(-1))
    return torch.cat(out), torch.stack(states)


DELTA_GEOMETRIES = [  # heads, groups of q and k, key size, value size, rows per sequence
    (4, 2, 64, 64, (200, 1, 64, 65)), (2, 2, 128, 128, (300,)), (6, 2, 20, 28, (150, 7, 63)), (2, 1, 33, 17, (129, 66)),
    (2, 2, 200, 40, (140,)), (1, 1, 256, 16, (90, 128)), (3, 3, 96, 200, (70, 190)), (4, 4, 12, 8, (64, 64, 128))]


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("geom", DELTA_GEOMETRIES)
def test_delta_rule_kernels(geom, chunked):
    """The walk and the form in chunks of 64 tokens against the recurrence, several sequences at once from states of zeros,
    then a second call that goes on from the states the first one left; padding sequences (no rows) leave their state."""
    from odin_infer_b200.csrc import ops
    H, G, dk, dv, lens = geom
    x = delta_inputs(lens, H, G, dk, dv, seed=dk + dv)
    ref, states = delta_reference(x, lens, H, G, dk, dv)
    q, k, v, a, b, A, bias = x
    slots = torch.tensor(list(range(len(lens), 0, -1)) + [0], dtype=torch.int32, device=DEV)   # the last sequence is padding

    def run(pieces, state):
        """pieces: (first, end) of every sequence."""
        rows = torch.cat([torch.arange(sum(lens[:i]) + p0, sum(lens[:i]) + p1, device=DEV) for i, (p0, p1) in enumerate(pieces)])
        sizes = [p1 - p0 for p0, p1 in pieces] + [0]
        starts = torch.tensor([0] + np.cumsum(sizes).tolist(), dtype=torch.int32, device=DEV)
        o = torch.full((len(rows), H * dv), float("nan"), device=DEV)
        ops.delta_rule(*(t[rows].contiguous() for t in (q, k, v, a, b)), A, bias, o, state, starts, slots, len(lens) + 1, H, dk, dv,
                       heads_per_group=H // G, q_scale=dk ** -0.5, chunked=chunked, max_new=max(sizes))
        return rows, o
    state = torch.zeros(len(lens) + 1, H * dk * dv + 3, device=DEV)   # rows further apart than the state itself
    state[0] = 7.0
    rows, o = run([(0, n) for n in lens], state)
    close(o, ref[rows.cpu()], 6e-6)
    close(state[slots[:-1].long(), :H * dk * dv], states, 6e-6)
    assert (state[0] == 7.0).all() and (state[1:, H * dk * dv:] == 0).all()
    state = torch.zeros(len(lens) + 1, H * dk * dv + 3, device=DEV)
    for pieces in ([(0, (n + 1) // 2) for n in lens], [((n + 1) // 2, n) for n in lens]):
        rows, o = run(pieces, state)
        if len(rows):
            close(o, ref[rows.cpu()], 6e-6)
    close(state[slots[:-1].long(), :H * dk * dv], states, 6e-6)


@pytest.mark.parametrize("chunked", [False, True])
def test_delta_rule_with_repeated_keys_and_no_decay(chunked):
    """Equal keys in a row with full write strength and almost no decay: every write replaces the one before, which the chunk's
    triangular system must solve exactly; a key of zeros writes nothing; large keys count as unit vectors."""
    from odin_infer_b200.csrc import ops
    n, dk, dv = 130, 32, 24
    torch.manual_seed(9)
    k = torch.randn(1, dk, device=DEV).repeat(n, 1) * torch.linspace(0.1, 100.0, n, device=DEV)[:, None]
    k[70] = 0.0
    v = torch.randn(n, dv, device=DEV)
    q = k.clone()
    q[70] = k[0]
    a, b = torch.full((n, 1), -30.0, device=DEV), torch.full((n, 1), 30.0, device=DEV)
    zero = torch.zeros(1, device=DEV)
    o, state = torch.empty(n, dv, device=DEV), torch.zeros(1, dk * dv, device=DEV)
    starts, slots = torch.tensor([0, n], dtype=torch.int32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.delta_rule(q, k, v, a, b, zero, zero, o, state, starts, slots, 1, 1, dk, dv, chunked=chunked, max_new=n)
    want = v.clone()
    want[70] = v[69]      # the zero key wrote nothing: the last value still answers
    close(o, want, 2e-4)


DELTA_MIXERS = [(4, 2, 24, 40, 3, 150), (1, 1, 36, 12, 1, 131), (6, 3, 8, 16, 6, 90), (2, 1, 128, 64, 4, 300), (3, 1, 33, 20, 2, 140)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("geom", DELTA_MIXERS)
def test_delta_mixer_alone_remembers_a_loud_token(dtype, tol, geom):
    """Token 5 is louder than the rest: slow heads still carry its value a hundred tokens later, and a state or a
    convolution's memory that is lost between steps changes the rows after the cut.  Whole, in portions down to one token
    (shorter than the convolution), and the last forty tokens one by one; then in a slot that is used again."""
    from odin_infer_b200.parts import PartSpec, build_part
    H, G, D, V, taps, n = geom
    width = 80
    rt = runtime(dtype)
    names = {k: "m." + k for k in ("q", "k", "v", "g", "b", "a", "o", "A_log", "dt_bias", "norm")}
    names.update({s + "_conv": f"m.{s}.conv" for s in "qkv"})
    mixer = build_part("mixer", PartSpec("gated_delta_rule", dict(width=width, n_heads=H, n_groups=G, head_dim=D, v_head_dim=V,
                                                                  taps=taps, eps=1e-5, names=names)))

    def slow(t):
        t["m.dt_bias"] -= 2.0
        t["m.b"] *= 0.3
        for s in "qkv":
            t[f"m.{s}.conv"][:, -1] = 1.0
    w = bound(mixer, dtype, rt, H * 10 + D, slow)
    torch.manual_seed(D)
    h = torch.randn(n, width, device=DEV)
    h[5] *= 12.0
    h = h.to(dtype)
    mx = dlt(H, G, D, V, taps)
    ref = P.delta(h.double().cpu(), w, "m.", mx, 1e-5)
    quiet = h.clone()
    quiet[5] /= 12.0
    other = P.delta(quiet.double().cpu(), w, "m.", mx, 1e-5)
    assert (other[60] - ref[60]).abs().max() > 1e-3 * ref[60].abs().max()     # the loud token is still heard at row 60
    cache = cache_for([mixer], dtype)
    for cuts in CUTS(n):
        close(run_in_steps(mixer, rt, cache, h, cuts), ref, tol)
    close(run_in_steps(mixer, rt, cache, quiet, [n]), other, tol)   # the slot's state was cleared for the next sequence


ATTENTION_GEOMETRIES = [  # heads, kv heads, dim, vdim, rotated, slowdown, tokens
    (4, 2, 24, 40, 8, 1.7, 200), (2, 2, 16, 8, 0, 1.0, 131), (4, 2, 64, 64, 32, 3.0, 330), (3, 1, 20, 28, 20, 0.5, 140),
    (2, 1, 128, 128, 128, 8.0, 330), (8, 2, 64, 64, 64, 4.0, 260)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("role", ["plain", "first", "later"])
@pytest.mark.parametrize("geom", ATTENTION_GEOMETRIES)
def test_attention_alone_with_a_key_far_back(dtype, tol, role, geom):
    """Against the plain attention, whole, in portions and one by one, over page borders.  Keys are projected by the queries'
    matrix with its input channels permuted, and the last row's input is row 2's in the other order, so that (in the elements
    that do not turn much) row 2's key stands out among hundreds; sinks differ from head to head, one of them far above every score.  "first" hands its values on,
    "later" mixes them with values of an earlier layer."""
    from odin_infer_b200.engine.step import StepBatch, StepEntry
    from odin_infer_b200.parts import PartSpec, build_part
    H, G, D, V, rot, slow, n = geom
    width, base, scale = 80, 1e8, 14.0 / D
    rt = runtime(dtype)
    perm = torch.randperm(width, generator=torch.Generator().manual_seed(1))
    names = {k: "m." + k for k in ("q", "k", "v", "o")}
    names.update({"q_norm": "m.q.norm", "k_norm": "m.k.norm"})
    mix = {"plain": None, "first": {"key": "v"}, "later": {"key": "v", "lambda": "m.vmix"}}[role]
    att = build_part("mixer", PartSpec("gqa_attention", dict(
        width=width, n_q_heads=H, n_kv_heads=G, head_dim=D, v_head_dim=V, position_encoding="pe" if rot else None, eps=1e-5,
        scale=scale, names=names, sink="m.sink", value_mix=mix)))
    if rot:
        att.pe = build_part("position_encoding", PartSpec("rope", dict(rotary_dim=rot, theta=base, slowdown=slow, precise=True,
                                                                       exact_angles=True)))
        att.pe.prepare(rt, n)

    def alike(t):
        t["m.k"] = t["m.q"].view(H, D, width)[::H // G].reshape(G * D, width)[:, perm]
        t["m.sink"][0] = 12.0
    w = bound(att, dtype, rt, H * 13 + D, alike)
    torch.manual_seed(D + V)
    h = torch.randn(n, width, device=DEV)
    h[n - 1, perm.to(DEV)] = h[2]
    h = h.to(dtype)
    first = torch.randn(n, G * V, device=DEV).to(dtype)
    mx = attn(H, G, D, V, scale, rot=rot, base=base, factor=slow, v_mix=role != "plain")
    early = first.double().cpu().view(n, G, V) if role == "later" else None
    ref, values = P.attention(h.double().cpu(), w, "m.", mx, 1e-5, early)
    moved = h.clone()
    moved[2] = moved[3]       # without row 2's own key and value the last row reads something else
    last = P.attention(moved.double().cpu(), w, "m.", mx, 1e-5, early)[0][n - 1]
    assert (last - ref[n - 1]).abs().max() > 0.1 * ref[n - 1].abs().max()
    cache = cache_for([att], dtype)
    for cuts in ([n], [2, 63, 64, 65, n - 3, n], list(range(n - 40, n + 1))):
        slot, at, outs = cache.take_slot(), 0, []
        for end in cuts:
            st = cache.extend(slot, end - at)
            step = StepBatch(cache, [StepEntry(slot, [0] * (end - at), list(range(end - at)))], [st], DEV)
            if role == "later":
                step.carried["v"] = first[at:end].contiguous()
            outs.append(summed(att.forward(rt, step, h[at:end].contiguous(), 0)).clone())
            if role == "first":
                close(step.carried["v"].float().view(end - at, G, V), values[at:end], 1e-5 if dtype == torch.float32 else 1e-2)
            cache.after_step(slot)
            at = end
        cache.give_back_slot(slot)
        close(torch.cat(outs), ref, tol)


LATENT_GEOMETRIES = [  # heads, dim, vdim, latent, rows
    (3, 20, 28, 48, 200), (1, 36, 12, 20, 131), (8, 64, 32, 128, 330), (4, 32, 64, 64, 260), (5, 16, 24, 33, 70)]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("geom", LATENT_GEOMETRIES)
def test_latent_attention_alone_with_a_key_far_back(dtype, tol, geom):
    """No positions: the last row's query is built to ask for row 2's latent, hundreds of rows back; a sink far above every
    score silences head 0 (but for what little is left), gates differ from head to head and token to token."""
    from odin_infer_b200.parts import PartSpec, build_part
    H, D, V, L, n = geom
    width, scale = 80, 20.0 / D
    rt = runtime(dtype)
    perm = torch.randperm(width, generator=torch.Generator().manual_seed(1))
    names = {"q": "m.q", "dkv": "m.dkv", "dkv_norm": "m.dkv.norm", "uk": "m.uk", "uv": "m.uv", "o": "m.o"}
    mixer = build_part("mixer", PartSpec("latent_attention", dict(
        width=width, n_heads=H, head_dim=D, rot_dim=0, v_head_dim=V, q_rank=0, kv_rank=L, names=names, position_encoding=None,
        eps=1e-5, scale=scale, sink="m.sink", gate="m.g")))

    def asks_for_the_other_order(t):   # the query of an input is (up to the norm) the key of that input in another order
        t["m.q"] = torch.zeros_like(t["m.q"])
        t["m.q"][:, perm] = t["m.uk"] @ t["m.dkv"]
        t["m.sink"][0] = 12.0
    w = bound(mixer, dtype, rt, H * 17 + L, asks_for_the_other_order)
    torch.manual_seed(L)
    h = torch.randn(n, width, device=DEV)
    h[n - 1, perm.to(DEV)] = h[2]
    h = h.to(dtype)
    mx = lat(H, D, V, L, scale)
    ref = P.latent_attention(h.double().cpu(), w, "m.", mx, 1e-5)
    moved = h.clone()
    moved[2] = moved[3]       # without row 2's own key the last row reads something else
    assert (P.latent_attention(moved.double().cpu(), w, "m.", mx, 1e-5)[n - 1] - ref[n - 1]).abs().max() > 0.1 * ref[n - 1].abs().max()
    cache = cache_for([mixer], dtype)
    for cuts in ([n], [2, 63, 64, 65, n - 3, n], list(range(n - 40, n + 1))):
        close(run_in_steps(mixer, rt, cache, h, cuts), ref, tol)


@pytest.mark.parametrize("T", [3, 40, 200])
@pytest.mark.parametrize("splits", [1, 3])
def test_product_per_head_with_partial_sums_and_a_gate(T, splits):
    """The product per head from partial sums of a split product (a view of wider rows), each head times the sigmoid of its
    gate, which are partial sums as well."""
    from odin_infer_b200.csrc import ops
    H, K, N = 5, 37, 70
    torch.manual_seed(T)
    wide = torch.randn(splits, T, H * K + 11 + H, device=DEV)
    w = torch.randn(H, K, N, device=DEV) / K ** 0.5
    a, gate = (wide[..., :H * K], wide[..., H * K + 11:]) if splits > 1 else (wide[0][:, :H * K], wide[0][:, H * K + 11:])
    total = wide.double().sum(0)
    want = torch.einsum("thk,hkn->thn", total[:, :H * K].view(T, H, K), w.double())
    out = torch.empty(T, H * N, device=DEV)
    ops.heads_linear(a, K, w, out, N)
    close(out.view(T, H, N), want, 3e-6)
    ops.heads_linear(a, K, w, out, N, gate=gate)
    close(out.view(T, H, N), want * torch.sigmoid(total[:, H * K + 11:])[:, :, None], 3e-6)


@pytest.mark.parametrize("T", [128, 300])
@pytest.mark.parametrize("H,K,N,pad", [(3, 64, 40, 0), (5, 128, 264, 24), (1, 192, 128, 8)])
def test_product_per_head_on_the_tensor_cores(T, H, K, N, pad):
    """Heads further apart than they are wide, output columns that are no whole tile, token counts that are none either, a
    gate; the columns between the heads stay as they were."""
    from odin_infer_b200.csrc import ops
    torch.manual_seed(T + K)
    a = torch.randn(T, H * (K + pad), device=DEV).to(torch.bfloat16)
    w = (torch.randn(H, N, K, device=DEV) / K ** 0.5).to(torch.bfloat16)
    gate = torch.randn(2, T, H + 3, device=DEV)
    want = torch.einsum("thk,hnk->thn", a.double().view(T, H, K + pad)[:, :, :K], w.double())
    for g in (None, gate[..., 3:]):
        out = torch.full((T, H * (N + 2)), 7.0, dtype=torch.bfloat16, device=DEV)
        ops.heads_linear_tc(a, K + pad, w, out, N + 2, gate=g)
        got = out.view(T, H, N + 2)
        close(got[:, :, :N], want if g is None else want * torch.sigmoid(gate.double().sum(0)[:, 3:])[:, :, None], 5e-3)
        assert (got[:, :, N:] == 7.0).all()
    ops.moe_tc_check()


@pytest.mark.parametrize("T", [5, 300])
@pytest.mark.parametrize("given_logits", [False, True])
@pytest.mark.parametrize("E,top", [(8, 1), (5, 5), (1, 1), (40, 7)])
def test_router_with_scores_as_they_are(E, top, T, given_logits):
    from odin_infer_b200.csrc import ops
    d = 48
    torch.manual_seed(E * 100 + top)
    h = torch.randn(T, d, device=DEV)
    wr = 3.0 * torch.randn(E, d, device=DEV) / math.sqrt(d)
    ids, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.moe_router(h, wr, None, top, 0, None, ids, wts, (h @ wr.T).contiguous() if given_logits else None, score="sigmoid_as_is")
    picks = P.route(h.double().cpu(), wr.double().cpu(), {"experts": E, "top": top})
    for t in range(T):
        assert ids[t].tolist() == [e for e, _ in picks[t]]
        assert max(abs(a - b) for a, (_, b) in zip(wts[t].tolist(), picks[t])) <= 1e-5


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 2.5e-2)])
@pytest.mark.parametrize("T", [7, 200])
@pytest.mark.parametrize("E,top,ff", [(6, 3, 40), (8, 1, 32), (4, 4, 24)])
def test_experts_that_read_their_weight_times_the_input(dtype, tol, T, E, top, ff):
    """Row by row and as grouped products: the gate's activation sees the weighted input, which a weight on the answer alone
    would miss (checked: the two differ)."""
    from odin_infer_b200.cache import CacheManager
    from odin_infer_b200.engine.step import StepBatch, StepEntry
    from odin_infer_b200.parts import PartSpec, build_part
    width = 64
    rt = runtime(dtype)
    part = build_part("feed_forward", PartSpec("routed_experts", dict(
        width=width, inner=ff, n_experts=E, top=top, score="sigmoid_as_is", weigh_input=True,
        names={"router": "m.router", "gate": "m.e{e}.gate", "up": "m.e{e}.up", "down": "m.e{e}.down"})))
    w = bound(part, dtype, rt, E * 31 + T)
    torch.manual_seed(T)
    h = torch.randn(T, width, device=DEV).to(dtype)
    mlp, hd = moe(E, top, ff), h.double().cpu()
    ref = P.expert_mlp(hd, w, "m.", mlp)
    after = torch.zeros_like(ref)
    for t, picks in enumerate(P.route(hd, w["m.router"], mlp["router"])):
        for e, wt in picks:
            after[t] += wt * (w[f"m.e{e}.down"] @ (P.silu(w[f"m.e{e}.gate"] @ hd[t]) * (w[f"m.e{e}.up"] @ hd[t])))
    assert (after - ref).abs().max() > 0.1 * ref.abs().max()
    cache = CacheManager(64 * 8, 64 * 8)
    slot = cache.take_slot()
    cache.extend(slot, T)
    got = summed(part.forward(rt, StepBatch(cache, [StepEntry(slot, [0] * T, [])], [0], DEV), h))
    if dtype == torch.float32:
        close(got, ref, tol)
    else:   # a close call of the router may fall the other way for a token or two
        err = (got.double().cpu() - ref).abs().max(dim=1).values / ref.abs().max()
        assert int((err > tol).sum()) <= max(1, T // 20), err.max()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("T", [6, 150, 400, 1100])
@pytest.mark.parametrize("width,ff", [(64, 96), (100, 36), (256, 520)])
def test_dense_feed_forward_with_relu_squared(dtype, tol, T, width, ff):
    from odin_infer_b200.parts import PartSpec, build_part
    rt = runtime(dtype)
    part = build_part("feed_forward", PartSpec("activated", dict(width=width, inner=ff, activation="relu2", names={"up": "m.up", "down": "m.down"})))
    w = bound(part, dtype, rt, ff)
    torch.manual_seed(T)
    h = torch.randn(T, width, device=DEV).to(dtype)
    close(summed(part.forward(rt, None, h)), P.relu2_mlp(h.double().cpu(), w["m.up"], w["m.down"]), tol)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("d,rows", [(96, 9), (100, 3), (1028, 4), (2048, 5), (33, 4), (4096, 2), (4100, 2)])
def test_layer_norm_of_an_update_the_add_and_what_follows(dtype, tol, d, rows):
    """The kernel behind the blocks: partial sums far from zero mean, the update's layer norm with its scale, the add, and then
    the stream converted, a layer norm of it (also with gathered rows, which leave the stream alone) or nothing."""
    from odin_infer_b200.parts import PartSpec, build_part
    rt = runtime(dtype)
    torch.manual_seed(d)
    x = torch.randn(rows, d, device=DEV)
    u = torch.randn(3, rows, d, device=DEV) + 5.0
    post = build_part("norm", PartSpec("layernorm", dict(width=d, eps=1e-5, weight="a.norm1", bias="a.norm1.b", scale="a.ls1")))
    final = build_part("norm", PartSpec("layernorm", dict(width=d, eps=1e-3, weight="f.norm", bias="f.norm.b")))
    none = build_part("norm", PartSpec("none", dict(width=d)))
    wp, wf = bound(post, dtype, rt, 1), bound(final, dtype, rt, 2)
    want = x.double().cpu() + wp["a.ls1"] * P.ln(u.double().cpu().sum(0), wp["a.norm1"], wp["a.norm1.b"], 1e-5)
    x1 = x.clone()
    out = none.forward(rt, x1, post.as_update_norm(u))
    close(x1, want, 2e-6)
    close(out, want, tol)
    assert (out is x1) == (dtype == torch.float32)
    x2 = x.clone()
    close(final.forward(rt, x2, post.as_update_norm(u)), P.ln(want, wf["f.norm"], wf["f.norm.b"], 1e-3), tol)
    close(x2, want, 2e-6)
    pick = torch.tensor([rows - 1, 0], dtype=torch.int32, device=DEV)
    x3 = x.clone()
    close(final.forward(rt, x3, post.as_update_norm(u), rows=pick), P.ln(want, wf["f.norm"], wf["f.norm.b"], 1e-3)[[rows - 1, 0]], tol)
    assert torch.equal(x3, x)
    close(final.forward(rt, x3, None), P.ln(x.double().cpu(), wf["f.norm"], wf["f.norm.b"], 1e-3), tol)   # nothing pending
    close(none.forward(rt, x3, None), x, tol)
    assert torch.equal(x3, x)
    close(none.forward(rt, x3, u), x.double() + u.double().sum(0), tol)                                   # an update as it is


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hd,vd,T", [(64, 64, 9), (128, 128, 9), (128, 128, 300), (64, 64, 300), (24, 40, 30)])
def test_head_preparation_keeps_and_mixes_values(dtype, hd, vd, T):
    """The general kernel and the two fast ones: the cache holds (1 - lambda) v + lambda v_first, the kept copy the
    projection's own values, also from partial sums."""
    from odin_infer_b200.csrc import ops
    Hq, Hkv, lam = 4, 2, 0.3125
    torch.manual_seed(hd + T)
    parts = 2 if dtype == torch.bfloat16 else 1
    qkv = torch.randn(parts, T, Hq * hd + Hkv * (hd + vd), device=DEV)
    v = qkv.double().sum(0)[:, (Hq + Hkv) * hd:]
    first = torch.randn(T, Hkv * vd, device=DEV).to(dtype)
    n_pages = (T + 63) // 64
    bt = torch.arange(n_pages, dtype=torch.int32, device=DEV).flip(0).contiguous().view(1, -1)
    pos, seq = torch.arange(T, dtype=torch.int32, device=DEV), torch.zeros(T, dtype=torch.int32, device=DEV)
    seq[T - 1] = -1       # a padding row writes nothing
    ang = torch.randn(T, hd // 2, device=DEV)
    ones = torch.ones(hd, dtype=dtype, device=DEV)
    for kw in ("keep", "mix"):
        kc, vc = torch.full((n_pages, Hkv, 64, hd), 3.0, dtype=dtype, device=DEV), torch.full((n_pages, Hkv, 64, vd), 3.0, dtype=dtype, device=DEV)
        kept = torch.full((T, Hkv * vd), 3.0, dtype=dtype, device=DEV)
        ops.head_prep(qkv if parts > 1 else qkv[0], Hq, Hkv, hd, ones, ones, 1e-5, torch.cos(ang), torch.sin(ang), hd, pos, seq, bt, kc, vc,
                      q_out=torch.empty(T, Hq * hd, dtype=dtype, device=DEV), v_head_dim=vd,
                      **({"v_keep": kept} if kw == "keep" else {"v_first": first, "v_lambda": lam}))
        want = v if kw == "keep" else (1 - lam) * v + lam * first.double()
        got = torch.stack([vc[int(bt[0, t // 64]), :, t % 64].reshape(-1) for t in range(T - 1)])
        close(got, want[:T - 1], 1e-6 if dtype == torch.float32 else 6e-3)
        assert (vc[int(bt[0, (T - 1) // 64]), :, (T - 1) % 64] == 3.0).all()
        if kw == "keep":
            close(kept[:T - 1], v[:T - 1], 1e-6 if dtype == torch.float32 else 6e-3)
