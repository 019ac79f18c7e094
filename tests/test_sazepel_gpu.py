"""The Sazepel decoder against its plain implementation (``plain_sazepel``): every mechanism alone at the level of its
kernels, whole models of several shapes in both precisions, every way of cutting requests into steps and batches under page
pools and state slots that are used again, keys far back and at page edges in prompts and in decoding, long decoding through
captured steps, and greedy generation through the engine's own entry point.

The models are tiny, with sizes chosen so that nothing is equal by accident: head counts, key and value sizes differ, the two
sides of a pair have sizes of their own, a rotation covers part of a head or is absent, a layer has no feed-forward, a router
chooses one expert or all.  Attention is made sharp through the score scale (queries and keys have unit norm), the mixtures of
heads are far from the identity and have negative entries, and every scalar norm has a weight of its own.
"""
import json
import types

import numpy as np
import pytest
import torch

import plain_sazepel as plain

DEV = torch.device("cuda:0")
F64 = torch.float64


# --------------------------------------------------------------------------- model folders

def retention(heads, dim, vdim, decay, rot=None):
    out = {"decay": list(decay), "dim": dim, "heads": heads, "vdim": vdim}
    if rot:
        out["rot"] = {"base": rot[0], "dims": rot[1]}
    return out


def talking(heads, kv_heads, dim, vdim, scale):
    return {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}


def moe(ff, experts, top):
    return {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}


def alone(right, mlp):
    return {"type": "retention", "mixer": json.loads(json.dumps(right)), "mlp": mlp}


def pair(left, right, mlp):
    return {"type": "parallel", "mixer": json.loads(json.dumps({"left": left, "right": right})), "mlp": mlp}


def model(vocab, width, eps, scale, *layers):
    out = {"architecture": "Sazepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": list(layers)}
    if scale is not None:
        out["logit_scale"] = scale
    return out


def configs():
    return {
        # 6 heads on 3 key/value heads of 24 with values of 40, beside retention heads of 20 (14 of them rotated) with values
        # of 12; retention alone, with values wider than keys; no feed-forward in one layer
        "A": model(150, 72, 1e-5, 1.7,
                   pair(talking(6, 3, 24, 40, 0.35), retention(3, 20, 12, (0.5, 0.97, 0.999), (500.0, 14)), moe(24, 5, 2)),
                   alone(retention(2, 24, 40, (0.9, 0.998), (10000.0, 24)), None),
                   pair(talking(4, 1, 16, 16, 0.5), retention(1, 8, 8, (0.99,)), moe(40, 3, 1))),
        # heads of the sizes the tcgen05 attention kernels take, two heads on two and five on one key/value head; retention
        # heads of 136 (more than 128); every expert chosen; no scale on the logits
        "B": model(131, 96, 1e-6, None,
                   alone(retention(1, 136, 8, (0.99,), (300.0, 136)), moe(32, 4, 1)),
                   pair(talking(4, 2, 64, 64, 0.2), retention(2, 32, 64, (0.8, 0.995), (20000.0, 32)), moe(48, 6, 3)),
                   pair(talking(5, 1, 128, 128, 0.1), retention(4, 16, 16, (0.3, 0.9, 0.99, 0.9995), (50.0, 8)), moe(16, 2, 2))),
        # sizes off every 16-byte path: odd key and value sizes, a width of 70; a key/value head per head (4 of them)
        "C": model(96, 70, 1e-6, 0.4,
                   pair(talking(4, 4, 15, 9, 0.6), retention(2, 7, 33, (0.95, 0.6), (100.0, 6)), moe(18, 4, 2)),
                   alone(retention(5, 9, 5, (1.0, 0.8, 0.95, 0.99, 0.0)), moe(13, 7, 4))),
        # pairs with key/value heads enough that the blocks of different pairs matter (8 heads on 4), heads of 64 whose
        # values are narrower; experts of 64 (the fused gate/up epilogues) at a width in steps of 16
        "D": model(120, 64, 1e-6, 0.5,
                   pair(talking(8, 4, 64, 48, 0.15), retention(2, 64, 64, (0.9, 0.999), (1.0e6, 64)), moe(64, 3, 2)),
                   alone(retention(3, 64, 32, (0.97, 0.99, 0.995), (1.0e4, 32)), moe(64, 3, 1)),
                   pair(talking(2, 2, 128, 128, 0.1), retention(1, 128, 128, (0.998,), (1.0e5, 128)), None)),
    }


def write_model(folder, config, seed, edit=None):
    """Random weights of this test's own making, stored in bfloat16 so that every precision reads the same values."""
    from safetensors.torch import save_file
    g = torch.Generator().manual_seed(seed)

    def normal(*shape, std=1.0, mean=0.0):
        return (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16).contiguous()

    lin = lambda rows, cols, gain=1.0: normal(rows, cols, std=gain * cols ** -0.5)  # noqa: E731
    one = lambda: normal(std=0.25, mean=1.1)  # noqa: E731  (a number without axes)
    w, width = {}, config["width"]
    w["embed"], w["embed.norm"] = normal(config["vocab"], width, std=0.3), one()

    def fill_retention(p, m):
        hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        w[f"{p}.q"], w[f"{p}.k"], w[f"{p}.v"] = lin(hd, width, 1.3), lin(hd, width, 1.3), lin(hv, width)
        w[f"{p}.g"], w[f"{p}.o"] = lin(hv, width, 1.5), lin(width, hv)

    for i, entry in enumerate(config["layers"]):
        m, p = entry["mixer"], f"l{i}"
        for name in ("norm1", "norm1b") + (("norm2", "norm2b") if entry["mlp"] else ()):
            w[f"{p}.{name}"] = one()
        if entry["type"] == "retention":
            fill_retention(f"{p}.mix", m)
        else:
            a = m["left"]
            h, kv, d, v = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            w[f"{p}.mix.left.q"], w[f"{p}.mix.left.k"], w[f"{p}.mix.left.v"] = lin(h * d, width), lin(kv * d, width), lin(kv * v, width)
            w[f"{p}.mix.left.talk"] = (torch.eye(h) + 0.6 * torch.randn(h, h, generator=g)).to(torch.bfloat16)
            w[f"{p}.mix.left.g"], w[f"{p}.mix.left.o"] = lin(h * v, width, 1.5), lin(width, h * v)
            fill_retention(f"{p}.mix.right", m["right"])
            w[f"{p}.mix.left.out"], w[f"{p}.mix.right.out"] = normal(width, std=0.3, mean=1.0), normal(width, std=0.3, mean=0.8)
        if entry["mlp"]:
            f, e = entry["mlp"]["expert"]["ff"], entry["mlp"]["router"]["experts"]
            w[f"{p}.mlp.router"], w[f"{p}.mlp.router.b"] = lin(e, width, 2.0), normal(e, std=1.0)
            for k in range(e):
                w[f"{p}.mlp.e{k}.gate"], w[f"{p}.mlp.e{k}.up"] = lin(f, width, 1.5), lin(f, width)
                w[f"{p}.mlp.e{k}.down"] = lin(width, f)
    w["final.norm"] = one()
    w["head"] = normal(config["vocab"], width, std=2.0 * width ** -0.5)
    if edit:
        edit(w)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    save_file(w, str(folder / "model.safetensors"))
    return {k: v.to(F64) for k, v in w.items()}


def cooled(config):
    """The same model for the bfloat16 runs: a router that chooses every expert it has, since a choice between two experts
    whose logits are a rounding apart may fall either way in bfloat16 and then changes a whole request, and scores less
    sharp.  The choice itself is tested in float32 and kernel by kernel."""
    out = json.loads(json.dumps(config))
    for entry in out["layers"]:
        if entry["mlp"]:
            entry["mlp"]["router"]["top"] = entry["mlp"]["router"]["experts"]
        if entry["type"] == "parallel":
            entry["mixer"]["left"]["scale"] = round(entry["mixer"]["left"]["scale"] * 0.5, 4)
    return out


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for k, (name, config) in enumerate(configs().items()):
        for suffix, cfg in (("", config), ("+", cooled(config))):
            folder = tmp_path_factory.mktemp(f"sazepel{name}")
            out[name + suffix] = (str(folder), cfg, write_model(folder, cfg, 700 + k))
    return out


def model_for(models, name, dtype):
    key = name if dtype == "float32" else name + "+"
    return (*models[key], key)


def tokens_of(vocab, n, seed):
    g = torch.Generator().manual_seed(seed)
    return [int(t) for t in torch.randint(0, vocab, (n,), generator=g)]


_plain_cache = {}


def plain_logits(name, config, weights, tokens):
    key = (name, tuple(tokens))
    if key not in _plain_cache:
        _plain_cache[key] = plain.forward(config, weights, tokens)
    return _plain_cache[key]


def make_runner(folder, dtype, pages, page=16, seqs=4, graphs=True):
    from slipstream_b200.engine.runner import ModelRunner
    return ModelRunner(folder, dtype=dtype, page_size=page, num_pages=pages, max_num_seqs=seqs, max_model_len=1024,
                       use_cuda_graphs=graphs)


def replay(runner, requests, schedule):
    """``schedule``: steps, each a list of (request, number of tokens).  Logits of every position, per request."""
    from slipstream_b200.engine.runner import StepEntry
    at = {k: 0 for k in requests}
    got = {k: [] for k in requests}
    for step in schedule:
        entries = [StepEntry(k, requests[k][at[k]: at[k] + n], list(range(n))) for k, n in step]
        logits = runner.step(entries).cpu()
        runner.check()
        row = 0
        for k, n in step:
            got[k].append(logits[row: row + n])
            row += n
            at[k] += n
            if at[k] == len(requests[k]):
                runner.release(k)
    runner.cache.check_invariants()
    return {k: torch.cat(v) for k, v in got.items() if v}


def distances(got, want):
    """Root mean square of the difference (means taken off) over that of the plain logits, per position."""
    d = got.double() - want
    d = d - d.mean(dim=-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def distance(got, want):
    return float(distances(got, want).max())


# float32: norms behind every branch carry a rounding through unchanged in size; a fault of the kind these tests look for (a
# key, a state, a head, a row off by one) moves the logits by 1e-2 to 1.  bfloat16: at single positions a branch's output is
# small, and the norm behind it magnifies its rounding (the plain implementation with its products rounded to bfloat16 is
# off there by up to 0.26), so most positions have a bound and all of them another
BOUND = {"float32": 2e-4, "bfloat16": 6e-2}


def close(got, want, dtype):
    each = distances(got, want)
    if dtype == "float32":
        return float(each.max()) < BOUND[dtype]
    return float(each.quantile(0.9)) < BOUND[dtype] and float(each.max()) < 8 * BOUND[dtype]


def rel(got, want):
    return float((got.double().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-12))


# --------------------------------------------------------------------------- configuration and structure (no GPU)

def test_configuration_reads_every_branch_and_refuses_what_it_does_not_know():
    from slipstream_b200.config.reader import ConfigError
    from slipstream_b200.config.sazepel_config import SazepelConfig
    from slipstream_b200.registry import resolve_architecture
    c = configs()
    a = SazepelConfig.from_dict(c["A"])
    assert resolve_architecture(c["A"]).name == "Sazepel"
    assert (a.vocab_size, a.hidden_size, a.norm_eps, a.logit_scale) == (150, 72, 1e-5, 1.7)
    both, single, last = (entry.mixer for entry in a.layers)
    assert (both.left.heads, both.left.kv_heads, both.left.dim, both.left.vdim, both.left.scale) == (6, 3, 24, 40, 0.35)
    assert (both.right.heads, both.right.dim, both.right.vdim, both.right.decay) == (3, 20, 12, (0.5, 0.97, 0.999))
    assert (both.right.rot.base, both.right.rot.dims, last.right.rot, a.layers[1].mlp) == (500.0, 14, None, None)
    assert (single.heads, single.vdim, a.layers[0].mlp.ff, a.layers[0].mlp.experts, a.layers[0].mlp.top) == (2, 40, 24, 5, 2)
    b = SazepelConfig.from_dict(c["B"])
    assert b.logit_scale == 1.0
    assert SazepelConfig.from_dict(a.to_dict()) == a and SazepelConfig.from_dict(b.to_dict()) == b
    for spoil, text in ((lambda d: d["layers"][0].update(type="attention"), "not a mixer"),
                        (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "kind"),
                        (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=4), "kv_heads"),
                        (lambda d: d["layers"][0]["mixer"].pop("right"), "right"),
                        (lambda d: d["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
                        (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=26), "rot.dims"),
                        (lambda d: d["layers"][0]["mlp"]["router"].update(top=6), "top"),
                        (lambda d: d["layers"][2].pop("mixer"), "mixer"),
                        (lambda d: d.pop("width"), "width")):
        bad = json.loads(json.dumps(c["A"]))
        spoil(bad)
        with pytest.raises(ConfigError, match=text):
            SazepelConfig.from_dict(bad)


def test_model_structure_follows_the_configuration():
    from slipstream_b200.config.sazepel_config import SazepelConfig
    from slipstream_b200.models.sazepel import build_sazepel
    built = build_sazepel(SazepelConfig.from_dict(configs()["A"]))
    names = {s.name: tuple(s.shape) for s in built.weight_specs()}
    assert names["embed.norm"] == () and names["final.norm"] == () and names["l0.norm1b"] == () and names["l2.norm2"] == ()
    assert names["l0.mix.left.q"] == (144, 72) and names["l0.mix.left.v"] == (120, 72) and names["l0.mix.left.g"] == (240, 72)
    assert names["l0.mix.left.talk"] == (6, 6) and names["l0.mix.left.out"] == (72,) and names["l0.mix.right.out"] == (72,)
    assert names["l0.mix.right.v"] == (36, 72) and names["l0.mix.right.o"] == (72, 36) and "l0.mix.right.norm" not in names
    assert names["l0.mlp.router"] == (5, 72) and names["l0.mlp.router.b"] == (5,) and names["l0.mlp.e4.gate"] == (24, 72)
    assert names["l1.mix.g"] == (80, 72) and "l1.norm2" not in names and "l1.mlp.router" not in names
    # pages hold one size for keys and values, a multiple of 16; each layer's heads make a group of its own here
    assert [(g.spec.num_kv_heads, g.spec.head_dim, g.num_entries) for g in built.group_layouts] == [(3, 48, 1), (1, 16, 1)]
    assert [[(s.name, tuple(s.shape)) for s in entry] for entry in built.entry_state] == [
        [("right.memory", (3, 20, 12))], [("memory", (2, 24, 40))], [("right.memory", (1, 8, 8))]]


# --------------------------------------------------------------------------- every mechanism alone

def step_ctx(q_lens, seq_lens, slots):
    """What the state kernels read of a step: row ranges, positions, lengths after the step and state slots."""
    starts = [0]
    for n in q_lens:
        starts.append(starts[-1] + n)
    as_dev = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)  # noqa: E731
    positions = [p for n, s in zip(q_lens, seq_lens) for p in range(s - n, s)]
    return types.SimpleNamespace(q_start=as_dev(starts), seq_lens=as_dev(seq_lens), state_slots=as_dev(slots),
                                 positions=as_dev(positions), num_requests=len(q_lens), max_q_len=max(q_lens),
                                 is_decode_only=all(n == 1 for n in q_lens))


PLANS = [  # two requests of 200 and 37 rows: whole; portions down to two tokens and single ones; at the edges of tiles
    [[("a", 200), ("b", 37)]],
    [[("a", 33)], [("a", 2), ("b", 17)], [("a", 1), ("b", 1)], [("a", 34), ("b", 2)], [("b", 16)], [("b", 1)], [("a", 120)]]
    + [[("a", 1)] for _ in range(10)],
    [[("b", 37)], [("a", 16)], [("a", 64)], [("a", 63)], [("a", 57)]],
]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim,dims", [(3, 24, 40, 24), (1, 136, 8, 128), (2, 5, 33, 4), (4, 64, 64, 64), (4, 64, 32, 32),
                                                 (2, 128, 128, 128), (1, 256, 70, 0), (2, 48, 96, 20), (2, 64, 128, 0), (3, 32, 16, 16)])
def test_retention_whole_and_cut_with_slots_used_again(heads, dim, vdim, dims, dtype):
    from slipstream_b200 import ops
    g = torch.Generator().manual_seed(heads * 1000 + dim)
    lens, slots = {"a": 200, "b": 37}, {"a": 2, "b": 0}
    width = heads * (2 * dim + 2 * vdim)
    width += -width % 8
    rows = {k: (torch.randn(n, width, generator=g) * 0.8).to(dtype) for k, n in lens.items()}
    decay = [0.999, 0.5, 0.9, 0.97][:heads]
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": 700.0, "dims": dims} if dims else None}
    inv = (700.0 ** (-torch.arange(0, dims, 2, dtype=F64) / dims)).float().to(DEV) if dims else None
    eye = torch.eye(width, dtype=F64)
    at = np.cumsum([0, heads * dim, heads * dim, heads * vdim, heads * vdim])
    w = {f"p.{role}": eye[at[i]: at[i + 1]] for i, role in enumerate("qkvg")}
    w["p.o"] = torch.eye(heads * vdim, dtype=F64)
    # the plain mixer with identity projections: its input is the projected row itself
    want = {k: plain.retention(m, w, "p", r.double(), 1e-6) for k, r in rows.items()}
    for plan in PLANS:
        state = torch.randn(3, heads, dim, vdim, device=DEV)  # what a slot's last owner left
        state[[0, 2]] = 0.0  # the engine clears a slot at admission
        done = {k: 0 for k in lens}
        got = {k: [] for k in lens}
        for step in plan:
            ctx = step_ctx([n for _, n in step], [done[k] + n for k, n in step], [slots[k] for k, _ in step])
            x = torch.cat([rows[k][done[k]: done[k] + n] for k, n in step]).to(DEV)
            out = ops.retention(x, torch.tensor(decay, device=DEV), state, ctx, heads, dim, vdim, 1e-6, inv_freq=inv, k_scale=dim ** -0.5)
            row = 0
            for k, n in step:
                got[k].append(out[row: row + n].double().cpu())
                row += n
                done[k] += n
        for k in lens:
            assert rel(torch.cat(got[k]), want[k]) < (3e-5 if dtype == torch.float32 else 1e-2), (plan, k)
    ops.check_errors(DEV)


@pytest.mark.gpu
def test_retention_forgets_and_remembers_exactly():
    """Decays of 0 (the newest token alone) and 1 (every token alike), and a key 190 tokens back that alone matches."""
    from slipstream_b200 import ops
    heads, d, n = 2, 64, 200
    g = torch.Generator().manual_seed(1)
    x = torch.randn(n, heads * 3 * d, generator=g) * 0.05
    x[7, heads * d: 2 * heads * d] += 4.0 * torch.randn(heads * d, generator=g)
    x[199, : heads * d] = x[7, heads * d: 2 * heads * d]
    for dtype in (torch.float32, torch.bfloat16):
        rows = x.to(dtype)
        q, k, v = (rows[:, i * heads * d: (i + 1) * heads * d].double().reshape(n, heads, d) for i in range(3))
        for decay in ([0.0, 1.0], [1.0, 0.999]):
            want = plain.retention_heads(q, k * d ** -0.5, v, decay).reshape(n, -1)
            for cut in ([n], [64, 8, 1, 127]):
                state, at, got = torch.zeros(1, heads, d, d, device=DEV), 0, []
                for m in cut:
                    ctx = step_ctx([m], [at + m], [0])
                    got.append(ops.decay_attention(rows[at: at + m].contiguous().to(DEV), torch.tensor(decay, device=DEV), state, ctx, heads, d, d,
                                                   silu=False, k_scale=d ** -0.5))
                    at += m
                got = torch.cat(got)
                assert rel(got, want) < 2e-5, (dtype, decay, cut)
                assert rel(got[199:], want[199:]) < 2e-5


def attention_case(seed, lens, q_lens, n_q, n_kv, d, page, dtype):
    g = torch.Generator().manual_seed(seed)
    blocks = [-(-n // page) for n in lens]
    pages = sum(blocks) + 3
    perm = torch.randperm(pages, generator=g).tolist()
    table = torch.full((len(lens), max(blocks)), -1, dtype=torch.int32)
    for r in range(len(lens)):
        for b in range(blocks[r]):
            table[r, b] = perm.pop()
    kv = torch.randn(pages, 2, n_kv, page, d, generator=g)
    q = torch.randn(sum(q_lens), n_q, d, generator=g)
    starts = torch.tensor(np.concatenate([[0], np.cumsum(q_lens)]), dtype=torch.int32)
    return q.to(dtype), kv.to(dtype), table, starts, torch.tensor(lens, dtype=torch.int32)


def across_reference(q, kv, table, starts, lens, n_kv, page, scale):
    """[N, keys' head, values' head, head of the group, D]: every query head's weights over the values of every head."""
    n, n_q, d = q.shape
    group = n_q // n_kv
    out = torch.zeros(n, n_kv, n_kv, group, d, dtype=F64)
    for r in range(len(lens)):
        a, b, s = int(starts[r]), int(starts[r + 1]), int(lens[r])
        slot = torch.arange(s)
        where = table[r].long()[slot // page]
        k, v = kv.double()[where, 0, :, slot % page], kv.double()[where, 1, :, slot % page]  # [s, n_kv, d]
        seen = slot[None, :] <= torch.arange(s - (b - a), s)[:, None]
        scores = torch.einsum("ihd,jhd->hij", q[a:b].double(), k.repeat_interleave(group, dim=1)) * scale
        p = torch.softmax(scores.masked_fill(~seen, -float("inf")), -1)
        out[a:b] = torch.einsum("agij,jcd->iacgd", p.reshape(n_kv, group, b - a, s), v)
    return out


@pytest.mark.gpu
@pytest.mark.parametrize("n_q,n_kv,d,page", [(6, 3, 64, 16), (8, 1, 128, 16), (6, 3, 48, 8), (2, 2, 64, 8), (28, 4, 128, 64), (4, 1, 32, 5),
                                             (2, 2, 256, 16), (4, 2, 64, 32), (20, 1, 64, 16), (34, 2, 80, 16), (16, 8, 128, 16),
                                             (10, 5, 64, 8), (3, 3, 128, 64), (32, 2, 128, 8), (7, 7, 64, 64), (36, 6, 128, 32)])
def test_every_head_over_all_values_in_every_attention_kernel_and_the_mixture_behind(n_q, n_kv, d, page):
    from slipstream_b200 import ops
    from slipstream_b200.engine.context import query_tiles_host
    group, scale = n_q // n_kv, 2.0 * d ** -0.5
    g = torch.Generator().manual_seed(n_q)
    mix = torch.eye(n_q) + 0.5 * torch.randn(n_q, n_q, generator=g)
    for dtype, lens, q_lens in ((torch.float32, [70, 5, 330], [70, 5, 17]), (torch.bfloat16, [70, 5, 330, 200], [70, 5, 17, 1]),
                                (torch.bfloat16, [1, 63, 64, 65, 700, 129, 333], [1] * 7)):
        q, kv, table, starts, seq = attention_case(d + page, lens, q_lens, n_q, n_kv, d, page, dtype)
        n = q.shape[0]
        ref = across_reference(q, kv, table, starts, seq, n_kv, page, scale)
        flat = ref.reshape(n, -1)
        dev = [t.to(DEV) for t in (q.reshape(n, -1), kv, table, starts, seq)]
        ql = np.asarray(q_lens, dtype=np.int32)
        tiles = lambda lengths, rows: [torch.from_numpy(t).to(DEV) for t in query_tiles_host(lengths, rows)]  # noqa: E731
        tol = 5e-6 if dtype == torch.float32 else 1.2e-2
        fresh = lambda: torch.full((n, n_kv * n_q * d), float("nan"), device=DEV)  # noqa: E731
        args = (dev[0], n_q * d)
        if dtype == torch.float32:
            req, q0 = tiles(ql, 16)
            out = fresh()
            ops.paged_attention_simt(*args, out, dev[1], dev[2], req, q0, dev[3], dev[4], n_q, n_kv, d, scale, across=True)
            assert rel(out, flat) < tol, "simt"
        elif max(q_lens) > 1:
            req, r0 = tiles(ql * group, 64)
            out = fresh()
            ops.paged_attention_prefill(*args, out, dev[1], dev[2], req, r0, dev[3], dev[4], n_q, n_kv, d, scale, across=True)
            assert rel(out, flat) < tol, "mma"
            if ops.tcgen05_prefill_fits(d, n_q, n_kv, page):
                req, t0 = tiles(ql, 128 // group)
                for parts in (1, 2, 8):
                    out = fresh()
                    ops.paged_attention_prefill_tcgen05(*args, out, dev[1], dev[2], req, t0, dev[3], dev[4], n_q, n_kv, d, scale, parts, across=True)
                    assert rel(out, flat) < tol, ("tcgen05", parts)
        else:
            for tma, stages in [(False, 2)] + ([(True, 2), (True, 3)] if ops.tcgen05_attention_fits(d, n_q, n_kv, page, 0) else []):
                for slices in (1, 2, 5, 8, 16):
                    out = fresh()
                    ops.paged_attention_decode(*args, out, dev[1], dev[2], dev[3], dev[4], n, n_q, n_kv, d, scale, n_slices=slices, tma=tma,
                                               stages=stages, across=True)
                    assert rel(out, flat) < tol, ("decode", tma, stages, slices)
        # the mixture: heads' outputs per values' head, weighed by the row of the table, under the gate of the row
        gate = torch.randn(n, n_q * d + 8, generator=g).to(dtype)
        by_head = ref.permute(0, 2, 1, 3, 4).reshape(n, n_kv, n_q, d)  # [N, values' head, query head, D]
        want = torch.stack([torch.einsum("g,ngd->nd", mix[h].double(), by_head[:, h // group]) for h in range(n_q)], dim=1).reshape(n, -1)
        table_t = mix.t().contiguous().to(DEV)
        got = ops.talk_heads(flat.float().to(DEV), table_t, n_kv, dtype)
        assert rel(got, want) < (5e-6 if dtype == torch.float32 else 6e-3)
        got = ops.talk_heads(flat.float().to(DEV), table_t, n_kv, dtype, gate.to(DEV)[:, 8:])
        gated = want * torch.sigmoid(gate[:, 8:].double())
        assert rel(got, gated) < (5e-6 if dtype == torch.float32 else 8e-3)
        if dtype == torch.bfloat16 and max(q_lens) == 1 and ops.across_decode_sets(d, n_q, n_kv, page)[0]:
            for slices in (1, 2, 5, 18, 64):  # all kv heads in one walk, mixture and gate behind it
                got = ops.talking_attention_decode(*args, dev[1], dev[2], dev[3], dev[4], n, n_q, n_kv, d, scale, table_t, gate.to(DEV)[:, 8:], slices)
                assert rel(got, gated) < 1.5e-2, slices
                got = ops.talking_attention_decode(*args, dev[1], dev[2], dev[3], dev[4], n, n_q, n_kv, d, scale, table_t, None, slices)
                assert rel(got, want) < 1.5e-2, slices
    ops.check_errors(DEV)


@pytest.mark.gpu
@pytest.mark.parametrize("target", [0, 7, 8, 15, 16, 63, 64, 255, 256, 298, 299, 300])
def test_one_key_that_stands_out_is_found_wherever_it_lies(target):
    """A query at position 299: one key matches it far better than all others and its values (another one per key/value
    head) stand out.  Found at every place up to its own, at page and tile edges, never behind it; by prompt portions and
    by single tokens."""
    from slipstream_b200 import ops
    from slipstream_b200.engine.context import query_tiles_host
    n_q, n_kv, d, page, n = 4, 2, 64, 8, 300
    for dtype in (torch.float32, torch.bfloat16):
        q, kv, table, starts, seq = attention_case(5, [n + 1], [2], n_q, n_kv, d, page, dtype)
        direction = torch.randn(d, generator=torch.Generator().manual_seed(1))
        direction = direction / direction.norm() * d ** 0.5
        q[0] = direction.to(dtype)
        at = (int(table[0, target // page]), target % page)
        kv[at[0], 0, :, at[1]] = direction.to(dtype)
        kv[at[0], 1, :, at[1]] = torch.tensor([30.0, -50.0])[:, None].to(dtype)
        ref = across_reference(q, kv, table, starts, seq, n_kv, page, 1.0)
        assert (float(ref[0].abs().min()) > 20.0) == (target <= 299)
        dev = [t.to(DEV) for t in (q.reshape(2, -1), kv, table, starts, seq)]
        out = torch.empty(2, n_kv * n_q * d, device=DEV)
        ql = np.asarray([2], dtype=np.int32)
        tiles = lambda lengths, rows: [torch.from_numpy(t).to(DEV) for t in query_tiles_host(lengths, rows)]  # noqa: E731
        if dtype == torch.float32:
            req, q0 = tiles(ql, 16)
            ops.paged_attention_simt(dev[0], n_q * d, out, dev[1], dev[2], req, q0, dev[3], dev[4], n_q, n_kv, d, 1.0, across=True)
            assert rel(out, ref.reshape(2, -1)) < 1e-5
            continue
        req, t0 = tiles(ql, 64)
        ops.paged_attention_prefill_tcgen05(dev[0], n_q * d, out, dev[1], dev[2], req, t0, dev[3], dev[4], n_q, n_kv, d, 1.0, across=True)
        assert rel(out, ref.reshape(2, -1)) < 1e-2
        req, r0 = tiles(ql * 2, 64)
        ops.paged_attention_prefill(dev[0], n_q * d, out, dev[1], dev[2], req, r0, dev[3], dev[4], n_q, n_kv, d, 1.0, across=True)
        assert rel(out, ref.reshape(2, -1)) < 1e-2
        one, length = torch.tensor([0, 1], dtype=torch.int32, device=DEV), torch.tensor([n], dtype=torch.int32, device=DEV)
        for tma in (False, True):
            for slices in (1, 4):
                ops.paged_attention_decode(dev[0][:1].contiguous(), n_q * d, out, dev[1], dev[2], one, length, 1, n_q, n_kv, d, 1.0, n_slices=slices,
                                           tma=tma, across=True)
                assert rel(out[:1], ref[:1].reshape(1, -1)) < 1e-2, (tma, slices)
        behind = (int(table[0, 37]), n % page)  # what a page's last owner left behind the newest token reaches nobody
        kv[behind[0], :, :, behind[1]:] = float("inf")
        eye = torch.eye(n_q, device=DEV)
        want = torch.stack([ref[0, h // 2, h // 2, h % 2] for h in range(n_q)]).reshape(1, -1)
        for slices in (1, 7):
            got = ops.talking_attention_decode(dev[0][:1].contiguous(), n_q * d, kv.to(DEV), dev[2], one, length, 1, n_q, n_kv, d, 1.0, eye, None, slices)
            assert target > 299 or rel(got, want) < 1e-2, slices
            assert bool(torch.isfinite(got).all())


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n_q,n_kv,d,dv,D", [(6, 3, 24, 40, 48), (4, 4, 15, 9, 16), (4, 2, 64, 64, 64), (3, 1, 128, 100, 128), (2, 2, 200, 256, 256)])
def test_unit_norms_of_queries_keys_and_values_on_their_way_to_the_pages(n_q, n_kv, d, dv, D, dtype):
    from slipstream_b200 import ops
    g = torch.Generator().manual_seed(d)
    n, page, eps = 7, 5, 1e-3
    heads = torch.zeros(n, n_q + 2 * n_kv, D)
    heads[:, : n_q + n_kv, :d] = torch.randn(n, n_q + n_kv, d, generator=g)
    heads[:, n_q + n_kv:, :dv] = torch.randn(n, n_kv, dv, generator=g) * 3.0
    heads = heads.to(dtype)
    rows = torch.cat([heads.reshape(n, -1), torch.randn(n, 16, generator=g).to(dtype)], dim=1).contiguous().to(DEV)
    kv = torch.full((4, 2, n_kv, page, D), 7.0, dtype=dtype, device=DEV)
    slots = torch.tensor([3, 4, 5, 19, 0, -1, 11], dtype=torch.int32)
    ops.rope_norm_cache(rows, torch.arange(n, dtype=torch.int32, device=DEV), slots.to(DEV), None, kv, n_q, n_kv, D, 0, norm_dim=d, eps=eps,
                        value_norm_dim=dv)
    x = heads.double()
    over = torch.tensor([d] * (n_q + n_kv) + [dv] * n_kv, dtype=F64)[None, :, None]
    want = x / torch.sqrt((x * x).sum(-1, keepdim=True) / over + eps)
    tol = 1e-6 if dtype == torch.float32 else 6e-3
    assert rel(rows[:, : n_q * D].reshape(n, n_q, D), want[:, :n_q]) < tol
    for t, slot in enumerate(slots.tolist()):
        if slot >= 0:
            assert rel(kv[slot // page, 0, :, slot % page], want[t, n_q: n_q + n_kv]) < tol
            assert rel(kv[slot // page, 1, :, slot % page], want[t, n_q + n_kv:]) < tol
    assert int((kv != 7.0).any(-1).sum()) == 2 * n_kv * 6  # the token without a slot went nowhere
    ops.check_errors(DEV)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top", [(5, 2), (4, 1), (12, 3), (3, 3), (37, 6)])
def test_router_bias_and_softmax_over_the_chosen(experts, top, dtype):
    from slipstream_b200 import ops
    g = torch.Generator().manual_seed(experts)
    hidden, n = 72, 50
    x, w = torch.randn(n, hidden, generator=g).to(dtype), (torch.randn(experts, hidden, generator=g) * 0.3).to(dtype)
    for bias in (torch.randn(experts, generator=g), torch.arange(experts) * 17.0, torch.where(torch.arange(experts) % 2 == 0, 16.0, 0.0)):
        mlp = {"router": {"experts": experts, "top": top}}
        ids_want, w_want = plain.route(mlp, {"p.router": w.double(), "p.router.b": bias.double()}, "p", x.double())
        ids, weights = ops.router(x.to(DEV), w.to(DEV), top, True, softmax=True, bias=bias.to(DEV))
        assert torch.equal(ids.cpu().long(), ids_want), "another choice"
        assert rel(weights, w_want) < 2e-5


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,n,hidden,ff,experts,top", [
    (torch.float32, 37, 72, 24, 5, 2), (torch.bfloat16, 37, 72, 24, 5, 2), (torch.bfloat16, 9, 70, 13, 4, 3), (torch.bfloat16, 3, 64, 64, 8, 1),
    (torch.bfloat16, 300, 64, 40, 3, 2), (torch.bfloat16, 600, 128, 128, 6, 2), (torch.bfloat16, 1, 128, 64, 6, 6)])
def test_gated_experts_weighed_on_their_outputs(dtype, n, hidden, ff, experts, top):
    """All routes of the grouped products (CUDA cores; mma.sync tiles of 32 and 128 rows; from 1,024 pairs the grouped
    tcgen05 kernel) through the part, router included, against the plain sum."""
    from slipstream_b200.parts import RoutedExperts, Runtime
    g = torch.Generator().manual_seed(n)
    part = RoutedExperts("m", hidden, ff, experts, top, renormalize=True, weight_on_input=False, scores="softmax", router_tensor="m.router",
                         router_bias="m.router.b", expert_names="m.e{e}.{role}")
    w = {s.name: (torch.randn(s.shape, generator=g) * (s.shape[-1] ** -0.5 if len(s.shape) > 1 else 1.0)).to(dtype) for s in part.weight_specs()}
    part.bind({k: v.to(DEV) for k, v in w.items()}, Runtime(DEV, dtype))
    x = torch.randn(n, hidden, generator=g).to(dtype)
    want = plain.routed_experts({"router": {"experts": experts, "top": top}}, {k: v.double() for k, v in w.items()}, "m", x.double())
    got = part.forward(x.to(DEV), None)
    each = (got.double().cpu() - want).abs().amax(-1) / want.abs().max()
    # (in bfloat16 a choice between two logits a rounding apart could fall either way: none does at these seeds)
    assert float(each.max()) < (1e-5 if dtype == torch.float32 else 2e-2)
    from slipstream_b200.ops import check_errors
    check_errors(DEV)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 70, 3584, 5000])
def test_norms_with_one_number_normed_embedding_and_normed_pair(width, dtype):
    from slipstream_b200 import ops
    from slipstream_b200.parts import JoiningNorm, Runtime, TokenEmbedding
    g = torch.Generator().manual_seed(width)
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    n, eps, vocab = 9, 1e-3, 40
    runtime = Runtime(DEV, dtype)
    norm_in, norm_out = JoiningNorm("n.in", width, eps, scalar=True), JoiningNorm("n.out", width, eps, scalar=True)
    embed = TokenEmbedding("e", vocab, width, scale=0.7, tensor="e", norm=JoiningNorm("e.norm", width, eps, scalar=True))
    w = {"n.in": torch.tensor(1.25), "n.out": torch.tensor(-0.75), "e.norm": torch.tensor(0.8125), "e": torch.randn(vocab, width, generator=g) * 0.1}
    w = {k: v.to(dtype) for k, v in w.items()}
    dev = {k: v.to(DEV) for k, v in w.items()}
    for part in (norm_in, norm_out, embed):
        assert [s.shape for s in part.weight_specs()][-1] == ()
        part.bind(dev, runtime)
    ids = torch.tensor([0, 39, 7, 7, 20, 1, 2, 3, 4], dtype=torch.int32)
    stream = embed.forward_step(ids.to(DEV), None, {})
    x = plain.norm(w["e"].double()[ids.long()] * 0.7, w["e.norm"].double(), eps)
    assert stream.dtype == torch.float32 and rel(stream, x) < 3e-6
    y = torch.randn(n, width, generator=g).to(dtype)
    got = norm_in.add_norm(stream, norm_out.branch(y.to(DEV)))
    x = x + plain.norm(y.double(), w["n.out"].double(), eps)
    assert rel(stream, x) < 3e-6 and rel(got, plain.norm(x, w["n.in"].double(), eps)) < tol
    a, b = (torch.randn(n, width, generator=g).to(dtype) for _ in range(2))
    wa, wb = torch.randn(width, generator=g), torch.randn(width, generator=g)
    want = 0.5 * (plain.norm(a.double(), wa.double(), eps) + plain.norm(b.double() * 1.0, wb.double(), eps))
    unformed = ops.PairedOutput(a.to(DEV), wa.to(DEV), b.to(DEV), wb.to(DEV), eps, 0.5)
    assert rel(unformed.materialize(), want) < tol
    # the pair's output formed where it joins the stream, and chosen experts' outputs summed there, in both their forms
    got = norm_in.add_norm(stream, norm_out.branch(unformed))
    x = x + plain.norm(want, w["n.out"].double(), eps)
    assert rel(stream, x) < 3e-6 and rel(got, plain.norm(x, w["n.in"].double(), eps)) < tol
    terms, weights = torch.randn(n, 3, width, generator=g), torch.rand(n, 3, generator=g)
    place = torch.randperm(3 * n, generator=g).to(torch.int32)
    in_order = torch.empty(3 * n, width)
    in_order[place.long()] = terms.reshape(3 * n, width)
    for y, value in ((ops.WeighedTerms(terms.to(DEV), None, weights.to(DEV)), terms.double()),
                     (ops.WeighedTerms(in_order.to(dtype).to(DEV), place.to(DEV), weights.to(DEV)), terms.to(dtype).double())):
        chosen = norm_in.add_norm(stream, norm_out.branch(y), rows=torch.tensor([7, 2], dtype=torch.int32, device=DEV))
        got = norm_in.add_norm(stream, norm_out.branch(y))
        x = x + plain.norm((weights.double()[:, :, None] * value).sum(1), w["n.out"].double(), eps)
        want = plain.norm(x, w["n.in"].double(), eps)
        assert rel(stream, x) < 3e-6 and rel(got, want) < tol and rel(chosen, want[[7, 2]]) < tol
    ops.check_errors(DEV)
    out_of_range = torch.tensor([3, vocab], dtype=torch.int32, device=DEV)  # flagged by the kernel, nothing is read there
    embed.forward_step(out_of_range, None, {})
    with pytest.raises(ops.KernelError, match="vocabulary"):
        ops.check_errors(DEV)


# --------------------------------------------------------------------------- whole models

@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_every_cut_and_batch_gives_the_plain_logits(models, name, dtype):
    """Whole prompts; token by token; portions of several sizes down to two tokens; three unequal requests mixed, in a
    pool smaller than their sum, with two state slots, so that pages and slots are used again."""
    folder, config, weights, key = model_for(models, name, dtype)
    vocab = config["vocab"]
    reqs = {"a": tokens_of(vocab, 70, 1), "b": tokens_of(vocab, 37, 2), "c": tokens_of(vocab, 45, 3)}
    want = {k: plain_logits(key, config, weights, t) for k, t in reqs.items()}
    plans = {
        "whole": [[("a", 70)], [("b", 37)], [("c", 45)]],
        "token by token": [[("b", 1)] for _ in range(37)],
        "portions": [[("a", n)] for n in (16, 1, 2, 13, 3, 2, 17, 16)],
        "mixed": [[("a", 20), ("b", 2)], [("a", 1), ("b", 30)], [("a", 17), ("b", 1)], [("a", 2), ("b", 4)],
                  [("a", 30), ("c", 9)], [("c", 2)], [("c", 34)]],
    }
    for what, plan in plans.items():
        runner = make_runner(folder, dtype, pages=7, seqs=2)  # 112 tokens of cache for up to 115 tokens of requests
        got = replay(runner, reqs, plan)
        for k, logits in got.items():
            assert close(logits, want[k][: logits.shape[0]], dtype), (what, k, distance(logits, want[k][: logits.shape[0]]))


def drawn_config(seed):
    """A model of this design drawn at random: sizes, head counts, the order of the layers and constants follow the seed."""
    import random
    rnd = random.Random(seed)
    layers = []

    def draw_retention():
        heads, dim = rnd.randint(1, 4), rnd.randint(3, 80)
        rot = (rnd.choice([100.0, 10000.0, 5.0e5]), 2 * rnd.randint(1, dim // 2)) if rnd.random() < 0.8 else None
        return retention(heads, dim, rnd.randint(3, 80), [round(rnd.uniform(0.3, 0.9995), 4) for _ in range(heads)], rot)

    for _ in range(rnd.randint(2, 5)):
        mlp = None
        if rnd.random() < 0.8:
            experts = rnd.randint(1, 9)
            mlp = moe(rnd.randint(4, 70), experts, rnd.randint(1, experts))
        if rnd.random() < 0.4:
            layers.append(alone(draw_retention(), mlp))
        else:
            kv, dim = rnd.randint(1, 4), rnd.randint(4, 80)
            left = talking(kv * rnd.randint(1, 4), kv, dim, rnd.randint(3, 80), round(rnd.uniform(2.0, 7.0) / dim, 4))
            layers.append(pair(left, draw_retention(), mlp))
    return model(rnd.randint(60, 200), rnd.choice([40, 48, 57, 72, 88, 104, 136]), rnd.choice([1e-6, 1e-5]),
                 rnd.choice([None, round(rnd.uniform(0.3, 2.5), 2)]), *layers)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(1, 9))
def test_models_drawn_at_random(tmp_path, seed, dtype):
    """Eight models whose every size, constant and option follows a seed: whole prompts, and portions beside decoded tokens
    under a pool smaller than the requests with two state slots."""
    config = drawn_config(seed)
    if dtype == "bfloat16":
        config = cooled(config)
    weights = write_model(tmp_path / "m", config, 40 + seed)
    vocab = config["vocab"]
    reqs = {"a": tokens_of(vocab, 90, seed), "b": tokens_of(vocab, 23, seed + 100), "c": tokens_of(vocab, 41, seed + 200)}
    want = {k: plain.forward(config, weights, t) for k, t in reqs.items()}
    plans = {"whole": [[("a", 90)], [("b", 23)], [("c", 41)]],
             "mixed": [[("a", 19), ("b", 2)], [("a", 1), ("b", 20)], [("a", 68), ("b", 1)], [("a", 2), ("c", 3)], [("c", 1)], [("c", 37)]]}
    for what, plan in plans.items():
        runner = make_runner(str(tmp_path / "m"), dtype, pages=8, seqs=2)
        got = replay(runner, reqs, plan)
        for k, logits in got.items():
            assert close(logits, want[k][: logits.shape[0]], dtype), (seed, what, k, distance(logits, want[k][: logits.shape[0]]))


@pytest.mark.gpu
def test_the_stream_after_every_layer(models):
    from slipstream_b200.engine.context import plan_step, to_device
    from slipstream_b200.engine.runner import StepEntry
    for name in ("A", "C"):
        folder, config, weights = models[name]
        toks = tokens_of(config["vocab"], 40, 9)
        _, want = plain.forward(config, weights, toks, want_layers=True)
        runner = make_runner(folder, "float32", pages=4, seqs=1, graphs=False)
        seen = []

        def tap(pos, stream, pending):
            if pending is not None:  # the branch whose norm and sum the next norm's kernel would do
                stream = stream.clone()
                pending.norm.add_norm(stream, pending)
            seen.append(stream.double().cpu())

        runner.admit("a")
        ctx = to_device(plan_step([StepEntry("a", toks, [39])], runner.cache, runner.config.vocab_size), runner.device)
        ctx.extras["layer_observer"] = tap
        with torch.inference_mode():
            runner.run(ctx)
        runner.check()
        assert len(seen) == len(config["layers"])
        for i, total in enumerate(seen):
            assert float((total - want[i]).abs().max() / want[i].abs().max()) < 2e-5, (name, i)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "D"])
def test_long_decoding_through_captured_steps_across_pages(models, name, dtype):
    """A prompt of 21 tokens, then 150 tokens one by one (captured decode steps), beside a second request."""
    folder, config, weights, key = model_for(models, name, dtype)
    reqs = {"a": tokens_of(config["vocab"], 171, 5), "b": tokens_of(config["vocab"], 160, 6)}
    want = {k: plain_logits(key, config, weights, t) for k, t in reqs.items()}
    plan = [[("a", 21), ("b", 10)]] + [[("a", 1), ("b", 1)] for _ in range(150)]
    runner = make_runner(folder, dtype, pages=24, seqs=2)
    got = replay(runner, reqs, plan)
    for k, logits in got.items():
        assert close(logits, want[k][: logits.shape[0]], dtype), (k, distance(logits, want[k][: logits.shape[0]]))


def remembering(config):
    """The same model with one retention head per layer that hardly decays, and attention sharp enough to single out a key."""
    out = json.loads(json.dumps(config))
    for entry in out["layers"]:
        m = entry["mixer"]
        r = m if entry["type"] == "retention" else m["right"]
        r["decay"] = [0.9995] + r["decay"][1:]
        if entry["type"] == "parallel":
            m["left"]["scale"] = round(12.0 / m["left"]["dim"], 4)
    return out


@pytest.mark.gpu
def test_tokens_far_back_decide(tmp_path):
    """What the plain model says when ten tokens some 380 positions back change (retention heads that hardly forget, sharp
    attention over every key) moves its logits by many times the bound; the engine follows in prompts cut at odd places and
    in decoding."""
    config = remembering(configs()["A"])
    weights = write_model(tmp_path / "m", config, 5)
    vocab = config["vocab"]
    base = tokens_of(vocab, 400, 21)
    other, first = list(base), list(base)
    for i in range(10, 20):
        other[i] = (base[i] + 1) % vocab
    first[0] = (base[0] + 1) % vocab
    want = {k: plain.forward(config, weights, t) for k, t in (("base", base), ("other", other), ("first", first))}
    assert distance(want["other"][-33:], want["base"][-33:]) > 20 * BOUND["float32"]
    assert distance(want["first"][-33:], want["base"][-33:]) > 5 * BOUND["float32"]
    plan = [[("x", 100)], [("x", 3)], [("x", 64)], [("x", 201)]] + [[("x", 1)] for _ in range(32)]
    for k, toks in (("base", base), ("other", other), ("first", first)):
        got = replay(make_runner(str(tmp_path / "m"), "float32", pages=26, seqs=1), {"x": toks}, plan)["x"]
        assert distance(got, want[k]) < BOUND["float32"], (k, distance(got, want[k]))


def test_a_mistake_in_a_mechanism_would_show():
    """Mistakes planted in the plain implementation move its logits by many times the float32 bound (no GPU)."""
    g = torch.Generator().manual_seed(0)
    import pathlib
    import tempfile
    config = configs()["A"]
    with tempfile.TemporaryDirectory() as folder:
        weights = write_model(pathlib.Path(folder) / "m", config, 700)
    toks = [int(t) for t in torch.randint(0, config["vocab"], (60,), generator=g)]
    right = plain.forward(config, weights, toks)

    def with_(changes):
        kept = {k: getattr(plain, k) for k in changes}
        try:
            for k, v in changes.items():
                setattr(plain, k, v)
            return plain.forward(config, weights, toks)
        finally:
            for k, v in kept.items():
                setattr(plain, k, v)

    talk, heads, rotate, route = plain.talk, plain.retention_heads, plain.rotate, plain.route
    wrong = {
        "mixture transposed": with_({"talk": lambda p, t: talk(p, t.T)}),
        "no mixture": with_({"talk": lambda p, t: p}),
        "a decay short": with_({"retention_heads": lambda q, k, v, d: heads(q, k, v, d) - (q * k).sum(-1, keepdim=True) * v}),
        "state not carried over a cut": with_({"retention_heads": lambda q, k, v, d: torch.cat([heads(q[:50], k[:50], v[:50], d), heads(q[50:], k[50:], v[50:], d)])}),
        "rotation off by one": with_({"rotate": lambda x, rot: rotate(torch.cat([x[1:], x[:1]]), rot)}),
        "values not normed": with_({"talking_attention": lambda m, w, p, h, eps: _unnormed_values(m, w, p, h, eps)}),
        "no router bias": with_({"route": lambda mlp, w, p, h: route(mlp, {**w, f"{p}.router.b": torch.zeros_like(w[f"{p}.router.b"])}, p, h)}),
        "chosen experts weighed alike": with_({"route": lambda mlp, w, p, h: (route(mlp, w, p, h)[0], torch.full_like(route(mlp, w, p, h)[1], 0.5))}),
    }
    for what, logits in wrong.items():
        assert distance(logits, right) > 50 * BOUND["float32"], (what, distance(logits, right))


def _unnormed_values(m, w, p, h, eps):
    t = h.shape[0]
    q = plain.unit((h @ w[f"{p}.q"].T).reshape(t, m["heads"], m["dim"]), eps)
    k = plain.unit((h @ w[f"{p}.k"].T).reshape(t, m["kv_heads"], m["dim"]), eps)
    v = (h @ w[f"{p}.v"].T).reshape(t, m["kv_heads"], m["vdim"]).repeat_interleave(m["heads"] // m["kv_heads"], dim=1)
    o = torch.einsum("hij,jhv->ihv", plain.talk(plain.head_weights(q, k, m["scale"]), w[f"{p}.talk"]), v).reshape(t, -1)
    return (o * torch.sigmoid(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T


@pytest.mark.gpu
def test_a_state_slot_that_is_not_cleared_shows(models):
    """Negative control: when a slot's last owner's state is left in place, the next request's logits are far off."""
    folder, config, weights = models["C"]
    reqs = {"a": tokens_of(config["vocab"], 30, 1), "b": tokens_of(config["vocab"], 30, 2)}
    want = plain_logits("C", config, weights, reqs["b"])
    runner = make_runner(folder, "float32", pages=8, seqs=1)
    replay(runner, {"a": reqs["a"]}, [[("a", 30)]])
    runner.store.zero_state = lambda slot: None
    got = replay(runner, {"b": reqs["b"]}, [[("b", 30)]])["b"]
    assert distance(got, want) > 20 * BOUND["float32"]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B", "D"])
def test_long_portions_and_steps_that_keep_coming_up(models, name, dtype):
    """600-token portions (the tensor-core paths of attention, retention and experts), then portions of one size until
    their step is replayed from a graph, then single tokens."""
    folder, config, weights, key = model_for(models, name, dtype)
    toks = tokens_of(config["vocab"], 800, 77)
    want = plain_logits(key, config, weights, toks)
    runner = make_runner(folder, dtype, pages=54, seqs=1)
    got = replay(runner, {"x": toks}, [[("x", 600)]] + [[("x", 19)] for _ in range(10)] + [[("x", 8)], [("x", 1)], [("x", 1)]])["x"]
    assert close(got, want, dtype), distance(got, want)


@pytest.mark.gpu
def test_greedy_generation_through_the_engine_and_its_scheduler(models):
    """Five prompts of unequal length through `LLMEngine.generate_batch` with prompt portions of 16 tokens and room for
    two requests at a time, so that pages and state slots come back: every generated token is the plain model's
    arg-max (or within a hair of it)."""
    from slipstream_b200 import CacheConfig, EngineConfig, SamplingParams, SchedulerConfig
    from slipstream_b200.engine.llm_engine import LLMEngine, Request
    for name, dtype, slack in (("A", "float32", 1e-4), ("D+", "bfloat16", 5e-2)):
        folder, config, weights = models[name]
        engine = LLMEngine(EngineConfig.for_model(folder, dtype=dtype, max_model_len=512,
                                                  cache=CacheConfig(block_size=16, num_gpu_blocks=14),
                                                  scheduler=SchedulerConfig(prefill_chunk_size=16, max_num_seqs=2)))
        prompts = [tokens_of(config["vocab"], n, 40 + n) for n in (1, 5, 37, 50, 18)]
        params = SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True)
        outs = engine.generate_batch([Request(f"r{i}", None, p, params, float(i)) for i, p in enumerate(prompts)])
        for prompt, out in zip(prompts, outs):
            assert len(out) == 12
            toks = list(prompt)
            for tok in out:
                logits = plain.forward(config, weights, toks)[-1]
                assert logits[tok] >= logits.max() - slack * logits.abs().max(), (name, len(toks))
                toks.append(tok)
        assert engine.runner.cache.all_pages_free()
        engine.runner.check()
