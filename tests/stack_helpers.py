"""What the GPU tests of layer stacks share: step inputs, portions of sequences, a paged key / value store on scattered pages."""
import torch

DEV = "cuda:0"
DEPTH = 8


def rel(got, want):
    return float((got.float().cpu() - want).norm() / want.norm())


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def status_word():
    return torch.zeros(4, dtype=torch.int32, device=DEV)


def meta(runs, slots, cache_slots=None):
    """Device inputs of a step: runs = [(first position, rows)] of the sequences in `slots`."""
    starts = [sum(n for _, n in runs[:i]) for i in range(len(runs))]
    return {"q_start": i32(starts), "q_len": i32([n for _, n in runs]), "kv_len": i32([p + n for p, n in runs]), "state_slot": i32(slots),
            "slot_map": i32(cache_slots if cache_slots is not None else list(range(sum(n for _, n in runs))))}


# portions of three sequences in one batch: long runs with ragged ends, runs around the depth of a state slot, single tokens; then single
# steps that take tokens back
STEPS = [[(0, 37), (0, 1), (0, 9)], [(37, 1), (1, 2), (9, 8)], [(38, 150), (3, 1), (17, 1)], [(188, 3), (4, 64), (18, 65)], [(191, 8), (68, 7), (83, 2)],
         [(192, 1), (70, 8), (84, 8)], [(193, 1), (78, 1), (92, 129)]]


class Paged:
    """A paged key / value store with sequences on scattered pages; slots nobody owns hold large finite noise."""

    def __init__(self, lens, G, dim, vdim, dt, seed=0):
        g = torch.Generator().manual_seed(seed)
        up = lambda n: -(-n // 64) * 64
        self.dp, self.dvp = up(dim), up(vdim)
        need = [-(-n // 64) for n in lens]
        total = sum(need) + 3
        ids = (torch.randperm(total - 1, generator=g) + 1).tolist()
        pages = [[ids.pop() for _ in range(n)] for n in need]
        store = torch.randn(total * 64, G * (self.dp + self.dvp) + 64, generator=g) * 40
        self.k, self.v = [], []
        for n, pg in zip(lens, pages):
            k, v = torch.randn(n, G, dim, generator=g).to(dt).float(), torch.randn(n, G, vdim, generator=g).to(dt).float()
            self.k.append(k); self.v.append(v)
            for j in range(n):
                s = pg[j // 64] * 64 + j % 64
                for h in range(G):
                    store[s, h * self.dp:h * self.dp + dim] = k[j, h]
                    store[s, G * self.dp + h * self.dvp:G * self.dp + h * self.dvp + vdim] = v[j, h]
        self.store = store.to(dt).to(DEV)
        self.table = torch.zeros(len(lens), max(need), dtype=torch.int32)
        for i, pg in enumerate(pages):
            self.table[i, :len(pg)] = torch.tensor(pg)
        self.table = self.table.to(DEV)
