"""The bf16-weight hybrid kernels and the Fezopel design on the GPU against the plain CPU implementation: every
mechanism alone, then whole models: prompts, token-by-token decoding, portions, reuse, greedy generation."""

import pytest
import torch

from oracle import fezopel_oracle as O
from quickdraw_b200 import synthetic
from quickdraw_b200.engine import Engine
from quickdraw_b200.loader import save_hybrid_checkpoint
from quickdraw_b200.state import HybridState, LayerHistory
from quickdraw_b200.weights import ChannelDeltaWeights, GLAWeights, WindowAttnWeights
from tests import hybrid_cases as cases

pytestmark = pytest.mark.gpu
BF16, F32, F64 = torch.bfloat16, torch.float32, torch.float64
TOLERANCE = {F32: 3e-5, BF16: 2e-2}


def rnd(*shape, seed=0, std=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std


def bf(*shape, seed=0, std=1.0):
    return rnd(*shape, seed=seed, std=std).to(BF16)


def error(got, want):
    got, want = got.detach().to("cpu", F64), want.to(F64)
    return float((got - want).norm() / want.norm().clamp(min=1e-30))


@pytest.fixture(scope="module")
def M(cuda_device):
    from quickdraw_b200 import mixers
    return mixers


def status():
    return torch.zeros(1, dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------------------- products
SHAPES = [(1, 200, 256), (2, 33, 1032), (3, 8, 4104), (7, 5000, 64), (8, 77, 24), (9, 80, 64), (130, 72, 200), (300, 264, 72), (513, 1000, 128),
          (64, 24, 2056), (1100, 4104, 136), (40, 37, 50), (5, 19, 7), (70, 128, 9), (2600, 4160, 40)]


@pytest.mark.parametrize("tokens,rows,width", SHAPES)
@pytest.mark.parametrize("x_type,y_type", [(BF16, BF16), (BF16, F32), (F32, F32)])
def test_linear(M, tokens, rows, width, x_type, y_type):
    """Few-row, tensor-core and any-shape forms; the input is a slice of wider rows, the first outputs pass the GELU."""
    if x_type == F32 and tokens > 600:
        tokens = 600
    offset = 16
    wide = rnd(tokens, width + offset + (-width) % 8, seed=1).to(x_type)
    w = bf(rows, width, seed=2, std=width ** -0.5)
    stat, out = status(), torch.full((tokens, rows), 7.0, dtype=y_type, device="cuda")
    gelu = rows // 3
    x_dev = wide.cuda()
    M.linear(x_dev, offset, x_dev.shape[1], w.cuda(), out, tokens=tokens, status=stat, gelu_columns=gelu)
    want = wide[:, offset:offset + width].double() @ w.double().T
    want[:, :gelu] = O.gelu_erf(want[:, :gelu])
    assert int(stat.item()) == 0
    assert error(out, want) < (1e-5 if y_type == F32 else 5e-3)


# ------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("width", [64, 256, 320, 100, 33, 2048, 1280])
@pytest.mark.parametrize("older,following", [(-1, True), (0, True), (1, False), (7, True)])
@pytest.mark.parametrize("dtype", [BF16, F32])
def test_end_of_a_sublayer(M, width, older, following, dtype):
    from quickdraw_b200._lib import call_hybrid, ptr, stream_of
    tokens, ld = 5, width + (-width) % 8 + 8
    y, gate = rnd(tokens, width, seed=1).to(dtype), rnd(tokens, ld, seed=2).to(dtype)
    vec = {n: bf(width, seed=10 + i) for i, n in enumerate(("gb", "pw", "pb", "nw", "nb"))}
    x = rnd(tokens, width, seed=3) + 50.0 * (width == 320)          # a mean far from zero must not cost the variance its digits
    results, depth = rnd(older + 2, tokens, width, seed=4), bf(older + 2, seed=5)
    dev = {n: t.cuda() for n, t in vec.items()}
    y_d, gate_d, x_d, r_d, depth_d = y.cuda(), gate.cuda(), x.cuda(), results.cuda(), depth.cuda()
    out, normed = torch.empty_like(x_d), torch.empty(tokens, width, dtype=dtype, device="cuda")
    eps = 1e-4
    call_hybrid("qd_sublayer_close", ptr(y_d), ptr(gate_d), ld, ptr(dev["gb"]), ptr(dev["pw"]), ptr(dev["pb"]), ptr(x_d), ptr(out), ptr(r_d),
                r_d.stride(0), ptr(depth_d), older, ptr(dev["nw"]) if following else None, ptr(dev["nb"]) if following else None, ptr(normed),
                tokens, width, eps, M.DTYPE_CODE[dtype], stream_of(y_d))
    v64 = {n: t.double() for n, t in vec.items()}
    v = x.double() + O.layer_norm(y.double() * torch.sigmoid(gate[:, :width].double() + v64["gb"]), v64["pw"], v64["pb"], eps)
    if older >= 0:
        assert error(r_d[older], v) < 1e-6 and torch.equal(r_d[:older].cpu(), results[:older])
        v = O.depth_average([*results[:older].double(), v], depth.double()[:older + 1])
    assert error(out, v) < 1e-6
    if following:
        assert error(normed, O.layer_norm(v, v64["nw"], v64["nb"], eps)) < (1e-5 if dtype == F32 else 4e-3)


def test_embedding_rows_and_norm(M):
    from quickdraw_b200._lib import call_hybrid, ptr, stream_of
    table, w, b = bf(50, 36), bf(36, seed=1), bf(36, seed=2)
    ids = torch.tensor([3, 49, 0, 3])
    x, normed = torch.empty(4, 36, device="cuda"), torch.empty(4, 36, device="cuda")
    dev = [t.cuda() for t in (ids, table, w, b)]
    call_hybrid("qd_embed_norm", ptr(dev[0]), ptr(dev[1]), 50, ptr(x), ptr(dev[2]), ptr(dev[3]), ptr(normed), 4, 36, 1e-5, 1, stream_of(x))
    assert torch.equal(x.cpu(), table[ids].float())
    assert error(normed, O.layer_norm(table[ids].double(), w.double(), b.double(), 1e-5)) < 1e-6


@pytest.mark.parametrize("count", [1, 203, 40000])
def test_greedy_choice_takes_the_lowest_of_equals(M, count):
    from quickdraw_b200._lib import call_hybrid, ptr, stream_of
    keys, counter, token = torch.empty(128, dtype=torch.int64, device="cuda"), status(), torch.zeros((), dtype=torch.long, device="cuda")
    for seed in range(3):
        logits = rnd(count, seed=seed) - 5.0
        logits[torch.randint(0, count, (3,), generator=torch.Generator().manual_seed(seed))] = 2.5 - 5.0 * (seed == 2)
        dev = logits.cuda()
        call_hybrid("qd_greedy", ptr(dev), count, ptr(keys), ptr(counter), ptr(token), stream_of(dev))
        assert int(token) == int((logits == logits.max()).nonzero()[0])


# ------------------------------------------------------------------------------- mixers alone
def stacked(parts, tokens, dtype, seed=0):
    """Random projection rows laid out as the model does, and each part as float64."""
    at, total = {}, 0
    for name, width in parts.items():
        at[name] = total
        total += width + (-width) % 8
    proj = rnd(tokens, total, seed=seed).to(dtype)
    return proj, at, {name: proj[:, at[name]:at[name] + width].double() for name, width in parts.items()}


def drive(mixer, proj, at, history, cuts, start=0):
    """The mixer over the rows in portions of the given sizes (1: the one-token form)."""
    out, done, stat = [], 0, status()
    for cut in cuts:
        rows = proj[done:done + cut]
        if cut == 1:
            out.append(mixer.step(rows, at, history, torch.tensor(start + done, dtype=torch.int32, device="cuda"), stat))
        else:
            out.append(mixer.chunk(rows, at, history, start + done, stat))
        done += cut
    assert done == proj.shape[0] and int(stat.item()) == 0
    return torch.cat(out)


CUTS = {"whole": lambda n: [n], "one by one": lambda n: [1] * n, "pairs": lambda n: [2] * (n // 2) + [1] * (n % 2),
        "portions": lambda n: [3, 17, 2, 1, 1, 20] + [n - 44]}


def attention_case(m, tokens, dtype, sharp, seed=0):
    """Projections, weights, and the oracle as a function of the window and of the sink."""
    parts = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim, "g": m.heads}
    proj, at, p = stacked(parts, tokens, dtype, seed)
    w = WindowAttnWeights(q=None, k=None, v=None, g=None, o=None, q_norm=bf(parts["q"], seed=seed + 1, std=0.3) + sharp,
                          k_norm=bf(parts["k"], seed=seed + 2, std=0.3) + 1, sink=bf(m.heads, seed=seed + 3, std=2.0) + sharp)
    eps = 1e-3

    def want(window=m.window, sink=1.0):
        positions = torch.arange(tokens)
        q = O.rms_norm(p["q"], w.q_norm.double(), eps).view(tokens, m.heads, m.dim)
        k = O.rms_norm(p["k"], w.k_norm.double(), eps).view(tokens, m.kv_heads, m.dim)
        q, k = (O.rotate_interleaved(x, positions, m.rotary_base, m.rotary_dims) for x in (q, k))
        out = O.window_sink_attention(q, k, p["v"].view(tokens, m.kv_heads, m.vdim), w.sink.double() if sink else w.sink.double() * 0 - 1e9,
                                      m.scale, window)
        return (out * torch.sigmoid(p["g"])[:, :, None]).reshape(tokens, -1)
    return w, eps, proj, at, want


ATTENTIONS = {
    "shared heads": cases.attention(), "one kv head": cases.attention(heads=5, kv_heads=1, dim=32, vdim=16, window=33, rotary_dims=32),
    "own heads": cases.attention(heads=3, kv_heads=3, dim=16, vdim=64, window=7, rotary_dims=4), "window of one": cases.attention(window=1),
    "window beyond the prompt": cases.attention(window=1000, scale=-0.2), "wide": cases.attention(heads=2, kv_heads=1, dim=136, vdim=200, window=64),
    "widest": cases.attention(heads=3, kv_heads=1, dim=256, vdim=256, window=200, rotary_dims=256),
    "no vectors": cases.attention(heads=3, kv_heads=3, dim=14, vdim=9, window=11, rotary_dims=6), "tile edges": cases.attention(window=64, heads=4, kv_heads=4),
}


@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("name", ATTENTIONS)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_window_attention(M, name, cut, dtype):
    """Scores stand out (large query norm weights), so a key too many or too few at the window's edge, or a sink left
    out, moves the result far beyond the tolerance; the ring is smaller than the prompt and wraps."""
    m, tokens = ATTENTIONS[name], 150
    w, eps, proj, at, want = attention_case(m, tokens, dtype, sharp=3.0)
    exact = want()
    if m.window < tokens:
        assert error(want(window=m.window + 1), exact) > 0.07 and (m.window == 1 or error(want(window=m.window - 1), exact) > 0.07)
    assert error(want(sink=0.0), exact) > 0.07
    weights = WindowAttnWeights(**{k: None if v is None else v.cuda() for k, v in vars(w).items()})
    mixer = M.WindowAttention(weights, m, eps, torch.device("cuda"))
    cuts = CUTS[cut](tokens)
    capacity = min(tokens, m.window - 1 + max(cuts))
    history = LayerHistory(k=torch.full((capacity, m.kv_heads, m.dim), float("nan"), dtype=dtype, device="cuda"),
                           v=torch.full((capacity, m.kv_heads, m.vdim), float("nan"), dtype=dtype, device="cuda"))
    got = drive(mixer, proj.cuda(), at, history, cuts)
    assert error(got, exact) < (5e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("splits", [1, 2, 5])
@pytest.mark.parametrize("name", ["widest", "wide", "window beyond the prompt", "no vectors"])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_decoding_with_long_splits(M, name, splits, dtype):
    """Splits of several key tiles (a large window has them), with one and with two tile buffers in shared memory."""
    m, tokens = ATTENTIONS[name], 230
    w, eps, proj, at, want = attention_case(m, tokens, dtype, sharp=3.0)
    weights = WindowAttnWeights(**{k: None if v is None else v.cuda() for k, v in vars(w).items()})
    mixer = M.WindowAttention(weights, m, eps, torch.device("cuda"))
    mixer.splits = min(splits, mixer.splits)
    capacity = min(tokens, m.window - 1 + 60)
    history = LayerHistory(k=torch.empty(capacity, m.kv_heads, m.dim, dtype=dtype, device="cuda"),
                           v=torch.empty(capacity, m.kv_heads, m.vdim, dtype=dtype, device="cuda"))
    got = drive(mixer, proj.cuda(), at, history, [60, 60, 60] + [1] * 50)
    assert error(got[180:], want()[180:]) < (5e-5 if dtype == F32 else 2e-2)


@pytest.mark.parametrize("inside", [True, False])
@pytest.mark.parametrize("decoded", [True, False])
def test_a_single_far_key_at_the_edge_of_a_long_window(M, inside, decoded):
    """One query equals one key at the far end of a window of 300 (or one position beyond it), all others are small."""
    m = cases.attention(heads=2, kv_heads=1, dim=32, vdim=16, window=300, rotary_dims=2, base=1e9, scale=1.0)
    tokens = 420
    w, eps, proj, at, want = attention_case(m, tokens, BF16, sharp=1.0, seed=5)
    special, query = bf(32, seed=9, std=4.0), 417
    key = query - (m.window - 1) - (0 if inside else 1)
    proj[:, at["k"]:at["k"] + 32] *= 0.05
    proj[key, at["k"]:at["k"] + 32] = special
    proj[query, at["q"]:at["q"] + 32] = special
    p64 = {n: proj[:, at[n]:at[n] + c].double() for n, c in (("q", 64), ("k", 32), ("v", 16), ("g", 2))}
    q = O.rms_norm(p64["q"], w.q_norm.double(), eps).view(tokens, 2, 32)
    k = O.rms_norm(p64["k"], w.k_norm.double(), eps).view(tokens, 1, 32)
    q, k = (O.rotate_interleaved(x, torch.arange(tokens), 1e9, 2) for x in (q, k))
    exact = O.window_sink_attention(q[:query + 1], k[:query + 1], p64["v"][:query + 1].view(-1, 1, 16), w.sink.double(), 1.0, m.window)[query]
    exact = exact * torch.sigmoid(p64["g"][query])[:, None]
    weights = WindowAttnWeights(**{n: None if v is None else v.cuda() for n, v in vars(w).items()})
    mixer = M.WindowAttention(weights, m, eps, torch.device("cuda"))
    history = LayerHistory(k=torch.empty(m.window - 1 + 128, 1, 32, dtype=BF16, device="cuda"), v=torch.empty(m.window - 1 + 128, 1, 16, dtype=BF16, device="cuda"))
    cuts = [128, 128, 128, 33] + ([1] * 3 if decoded else [3])
    got = drive(mixer, proj.cuda(), at, history, cuts)[query].view(2, 16)
    assert error(got, exact) < 2e-2


def gla_case(m, tokens, dtype, rank, seed=0):
    keys, values = m.heads * m.dim, m.heads * m.vdim
    proj, at, p = stacked({"q": keys, "k": keys, "v": values, "g": values, "a1": rank}, tokens, dtype, seed)
    w = GLAWeights(q=None, k=None, v=None, g=None, o=None, a1=None, a2=bf(keys, rank, seed=seed + 1, std=rank ** -0.5),
                   a2_b=bf(keys, seed=seed + 2, std=4.0) + 2, norm=bf(m.vdim, seed=seed + 3) + 1)
    eps = 1e-3
    heads = lambda t, d: t.view(tokens, m.heads, d)
    z = p["a1"] @ w.a2.double().T + w.a2_b.double()
    raw, state = O.gla_recurrence(heads(p["q"] * m.dim ** -0.5, m.dim), heads(p["k"], m.dim), heads(p["v"], m.vdim), heads(O.gla_decay(z, m.tau), m.dim))
    want = O.rms_norm(raw, w.norm.double(), eps).reshape(tokens, values) * O.silu(p["g"])
    return w, eps, proj, at, want, state


def delta_case(m, tokens, dtype, rank, seed=0):
    kv_keys, keys, values = m.kv_heads * m.dim, m.heads * m.dim, m.heads * m.vdim
    proj, at, p = stacked({"q": kv_keys, "k": kv_keys, "v": values, "b": m.heads, "a1": rank, "g1": rank + 3}, tokens, dtype, seed)
    conv = lambda n, i: bf(n, m.conv, seed=seed + i, std=1.0)
    w = ChannelDeltaWeights(q=None, k=None, v=None, b=None, o=None, a1=None, g1=None, q_conv=conv(kv_keys, 1), k_conv=conv(kv_keys, 2),
                            v_conv=conv(values, 3), A_log=bf(m.heads, seed=seed + 4), dt_bias=bf(keys, seed=seed + 5, std=3.0) - 2,
                            a2=bf(keys, rank, seed=seed + 6, std=rank ** -0.5), g2=bf(values, rank + 3, seed=seed + 7, std=0.3), norm=bf(m.vdim, seed=seed + 8) + 1)
    eps, share = 1e-3, m.heads // m.kv_heads
    q, k, v = (O.silu(O.causal_conv(p[n], getattr(w, n + "_conv").double())) for n in "qkv")
    q, k = (O.unit(x.view(tokens, m.kv_heads, m.dim)).repeat_interleave(share, 1) for x in (q, k))
    z = (p["a1"] @ w.a2.double().T + w.dt_bias.double()).view(tokens, m.heads, m.dim)
    raw, state = O.channel_delta_recurrence(q * m.dim ** -0.5, k, v.view(tokens, m.heads, m.vdim), O.channel_delta_decay(z, w.A_log.double()),
                                            torch.sigmoid(p["b"]))
    want = O.rms_norm(raw, w.norm.double(), eps).reshape(tokens, values) * torch.sigmoid(p["g1"] @ w.g2.double().T)
    return w, eps, proj, at, want, state


RECURRENCES = {
    "gla": (cases.gla(), 12), "gla 128": (cases.gla(heads=2, dim=128, vdim=96, tau=16.0), 24), "gla wide": (cases.gla(heads=1, dim=200, vdim=256, tau=1.0), 16),
    "gla odd": (cases.gla(heads=2, dim=21, vdim=13, tau=2.5), 5), "gla 64": (cases.gla(heads=4, dim=64, vdim=32), 8),
    "delta": (cases.delta(), 12), "delta 128": (cases.delta(heads=4, kv_heads=2, dim=128, vdim=64, conv=4), 16), "delta taps 1": (cases.delta(conv=1), 8),
    "delta taps 2": (cases.delta(heads=2, kv_heads=2, dim=64, vdim=32, conv=2), 8), "delta taps 5": (cases.delta(heads=3, kv_heads=1, dim=40, vdim=40, conv=5), 40),
    "delta wide": (cases.delta(heads=2, kv_heads=1, dim=256, vdim=136, conv=3), 8), "delta odd": (cases.delta(heads=2, kv_heads=2, dim=19, vdim=11, conv=3), 7),
    "delta values 300": (cases.delta(heads=2, kv_heads=1, dim=32, vdim=300, conv=3), 8),
}


@pytest.mark.parametrize("cut", CUTS)
@pytest.mark.parametrize("name", RECURRENCES)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_recurrent_mixers(M, name, cut, dtype):
    m, rank = RECURRENCES[name]
    tokens = 75
    is_delta = hasattr(m, "conv")
    w, eps, proj, at, want, state = (delta_case if is_delta else gla_case)(m, tokens, dtype, rank)
    weights = type(w)(**{n: None if t is None else t.cuda() for n, t in vars(w).items()})
    mixer = (M.ChannelDelta if is_delta else M.GatedLinearAttention)(weights, m, eps, torch.device("cuda"))
    history = LayerHistory(rec=torch.zeros(m.heads, m.dim, m.vdim, device="cuda"))
    if is_delta:        # nothing before position 0 is read
        history.conv = torch.full((m.conv, 2 * m.kv_heads * m.dim + m.heads * m.vdim), float("nan"), dtype=dtype, device="cuda")
    got = drive(mixer, proj.cuda(), at, history, CUTS[cut](tokens))
    assert error(got, want) < TOLERANCE[dtype]
    # the state is fp32 in both types: only the projections' rounding (part of the inputs here) differs
    assert error(history.rec, state) < (2e-5 if dtype == F32 else 2e-3)


def test_slow_decays_over_a_long_sequence(M):
    """Channels that forget one part in a hundred thousand per token: a decay rounded to fp32 would be off by its last
    bit at every token."""
    m = cases.gla(heads=1, dim=32, vdim=32, tau=16.0)
    tokens = 3000
    w, eps, proj, at, *_ = gla_case(m, tokens, F32, 8)
    w.a2_b = torch.full_like(w.a2_b, 9.0)
    w.a2 = w.a2 * 0
    p = {n: proj[:, at[n]:at[n] + 32].double() for n in ("q", "k", "v", "g")}
    decay = O.gla_decay(w.a2_b.double(), 16.0).expand(tokens, 32).view(tokens, 1, 32)
    _, state = O.gla_recurrence(*(p[n].view(tokens, 1, 32) for n in ("q", "k", "v")), decay)
    mixer = M.GatedLinearAttention(GLAWeights(**{n: None if t is None else t.cuda() for n, t in vars(w).items()}), m, eps, torch.device("cuda"))
    history = LayerHistory(rec=torch.zeros(1, 32, 32, device="cuda"))
    drive(mixer, proj.cuda(), at, history, [1000, 1990] + [1] * 10)
    assert error(history.rec, state) < 3e-6


# -------------------------------------------------------------------------------- whole models
def build(name, seed=3):
    cfg = cases.MODELS[name]()
    tensors = cases.tensors(cfg, seed)
    from quickdraw_b200.loader import assemble_hybrid
    return cfg, tensors, assemble_hybrid(cfg, lambda n: tensors[n].cuda())


def engine_of(ckpt, dtype, max_context=256, chunk=64, graph=True):
    return Engine(ckpt, max_context=max_context, device="cuda", dtype=dtype, prefill_chunk_size=chunk, cuda_graph=graph)


def run_portions(engine, tokens, cuts):
    rows, done = [], 0
    for cut in cuts:
        rows.append(engine.extend(tokens[done:done + cut], list(range(cut))))
        done += cut
    assert done == len(tokens) and engine.fused.check() == 0
    return torch.cat(rows)


LOGITS = {F32: 2e-4, BF16: 6e-2}


@pytest.mark.parametrize("name", cases.MODELS)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompts_portions_and_decoding_give_the_oracle_s_logits(cuda_device, name, dtype):
    """One prompt whole (longer than a chunk), token by token, in portions down to two tokens: the same logits; every
    run follows another request on the same engine."""
    cfg, tensors, ckpt = build(name)
    tokens = cases.prompt(cfg, 90)
    want, _ = O.forward(cfg.to_dict(), tensors, tokens)
    engine = engine_of(ckpt, dtype)
    scale = float(want.std())
    runs = {}
    for cut, sizes in (("whole", [90]), ("one by one", [1] * 90), ("portions", [2, 3, 31, 1, 2, 1, 1, 47, 2]), ("prompt and decoding", [70] + [1] * 20)):
        engine.reset()
        engine.extend(cases.prompt(cfg, 40, seed=9))           # another request leaves its rows and states behind
        engine.reset()
        runs[cut] = run_portions(engine, tokens, sizes).cpu().double()
        worst = float((runs[cut] - want).pow(2).mean(1).sqrt().max()) / scale
        assert worst < LOGITS[dtype], (cut, worst)
    for cut, got in runs.items():
        assert float((got - runs["whole"]).pow(2).mean(1).sqrt().max()) / scale < LOGITS[dtype], cut


def test_the_stream_after_every_layer(cuda_device):
    from quickdraw_b200.hybrid import FezopelModel
    cfg, tensors, ckpt = build("mixed")
    tokens = cases.prompt(cfg, 30)
    _, want = O.forward(cfg.to_dict(), tensors, tokens)
    record = []
    FezopelModel(ckpt, F32).run(torch.tensor(tokens, device="cuda"), 0, HybridState(cfg, 64, "cuda", dtype=F32), [29], record)
    for got, layer in zip(record, want):
        assert error(got, layer) < 1e-5


def test_long_decoding_wraps_the_rings(cuda_device):
    """300 tokens through a ring of 12 rows, decoded one by one and in the graph; the last logits follow the oracle."""
    cfg = cases.config([(cases.attention(window=9), 64), (cases.delta(), None)])
    tensors = cases.tensors(cfg)
    from quickdraw_b200.loader import assemble_hybrid
    engine = engine_of(assemble_hybrid(cfg, lambda n: tensors[n].cuda()), F32, max_context=512, chunk=4)
    assert engine.state.layers[0].k.shape[0] == 12
    tokens = cases.prompt(cfg, 300)
    want, _ = O.forward(cfg.to_dict(), tensors, tokens)
    got = run_portions(engine, tokens, [20] + [1] * 280).cpu().double()
    assert float((got - want).pow(2).mean(1).sqrt().max() / want.std()) < 2e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_graph_replay_and_eager_step_agree(cuda_device, dtype):
    cfg, tensors, ckpt = build("mixed")
    tokens = cases.prompt(cfg, 25)
    eager, graph = engine_of(ckpt, dtype, graph=False), engine_of(ckpt, dtype)
    assert eager.graph is None and graph.graph is not None
    a, b = (run_portions(e, tokens, [20] + [1] * 5) for e in (eager, graph))
    assert torch.equal(a, b)


@pytest.mark.parametrize("name", ["mixed", "attention first"])
def test_greedy_generation_follows_the_oracle(cuda_device, name):
    cfg, tensors, ckpt = build(name)
    prompt = cases.prompt(cfg, 17)
    want, gap = O.greedy(cfg.to_dict(), tensors, prompt, 12)
    engine = engine_of(ckpt, F32)
    assert gap > 1e-3 and engine.generate(prompt, 12) == want
    assert engine.generate(prompt, 12) == want                    # and again after its own request
    engine.eos_token_ids = {want[4]}
    stop = want.index(want[4])
    assert engine.generate(prompt, 12) == want[:stop + 1]


def test_snapshots_and_prefix_reuse(cuda_device):
    cfg, tensors, ckpt = build("mixed")
    prompt = cases.prompt(cfg, 60)
    engine = engine_of(ckpt, F32)
    engine.prefill_reuse(prompt[:40])
    snap = engine.snapshot()
    engine.prefill(cases.prompt(cfg, 50, seed=4))
    engine.restore(snap)
    got = engine.extend(prompt[40:], [19])[0]
    fresh = engine.prefill(prompt)
    torch.testing.assert_close(got, fresh, rtol=1e-4, atol=1e-4)
    engine.prefill_reuse(prompt[:40])
    again = engine.prefill_reuse(prompt)
    assert engine.reused_tokens == 40
    torch.testing.assert_close(again, fresh, rtol=1e-4, atol=1e-4)


def test_from_pretrained_reads_the_directory(cuda_device, tmp_path):
    cfg, tensors, ckpt = build("odd sizes")
    save_hybrid_checkpoint(cfg, tensors, tmp_path)
    engine = Engine.from_pretrained(str(tmp_path), max_context=64, dtype=F32)
    prompt = cases.prompt(cfg, 9)
    want, _ = O.forward(cfg.to_dict(), tensors, prompt)
    assert error(engine.prefill(prompt), want[-1]) < 2e-4


def test_sizes_of_a_real_layer(cuda_device):
    """Widths of a real model's layers (tensor-core tiles, vectorised epilogues, clusters of four blocks): a chunk
    against token-by-token decoding in fp32, and bf16 against fp32."""
    cfg = synthetic.fezopel_config(3, 512, hidden=512, heads=4, kv_heads=2, window=70)
    ckpt = synthetic.make_fezopel(cfg, 1, "cuda")
    tokens = cases.prompt(cfg, 140)
    exact = run_portions(engine_of(ckpt, F32), tokens, [140])
    steps = run_portions(engine_of(ckpt, F32), tokens, [1] * 140)
    half = run_portions(engine_of(ckpt, BF16, chunk=140), tokens, [140])
    assert error(steps, exact.cpu()) < 1e-4 and error(half, exact.cpu()) < 6e-2
