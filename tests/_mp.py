"""Spawn helper: run ``fn(rank, world, *args)`` in ``world`` processes (gloo on CPU, or NCCL with one GPU each)."""
import os
import socket
import traceback

import torch
import torch.distributed as dist
import torch.multiprocessing as mp


def _free_port():
    s = socket.socket()
    s.bind(("127.0.0.1", 0))
    p = s.getsockname()[1]
    s.close()
    return p


def _entry(rank, world, port, fn, args, q, backend="gloo", received=None):
    os.environ["MASTER_ADDR"] = "127.0.0.1"
    os.environ["MASTER_PORT"] = str(port)
    torch.set_num_threads(1)
    try:
        if backend == "nccl":
            torch.cuda.set_device(rank)
            dist.init_process_group("nccl", rank=rank, world_size=world, device_id=torch.device("cuda", rank))
        else:
            dist.init_process_group("gloo", rank=rank, world_size=world)
        out = fn(rank, world, *args)
        q.put((rank, "ok", out))
    except Exception:  # noqa: BLE001
        q.put((rank, "err", traceback.format_exc()))
    finally:
        if dist.is_initialized():
            dist.destroy_process_group()
    if received is not None:
        received.wait(60)      # tensors in the result are fetched from this process: it must not leave before


def run_distributed(fn, world, *args, timeout=300, backend="gloo"):
    ctx = mp.get_context("spawn")
    q, received = ctx.Queue(), ctx.Event()
    port = _free_port()
    procs = [ctx.Process(target=_entry, args=(r, world, port, fn, args, q, backend, received)) for r in range(world)]
    for p in procs:
        p.start()
    res = {}
    for _ in range(world):
        rank, st, out = q.get(timeout=timeout)
        if st == "err":
            for p in procs:
                p.kill()
            raise RuntimeError(f"rank {rank} failed:\n{out}")
        res[rank] = out
    received.set()
    for p in procs:
        p.join(timeout=30)
    return [res[r] for r in range(world)]
