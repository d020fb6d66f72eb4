"""Work of one layer that does not depend on each other, side by side on the device.

A layer whose sublayers read one input is a few chains of small kernels; in a step of single tokens each of them leaves
most of the device idle. Inside a captured step (where forking a stream costs the host nothing) `run_branches` puts
every chain but the first on a stream of its own, forked off the current stream and joined to it again by events, so
that the graph holds them as parallel branches. Elsewhere the chains run one after the other."""

from __future__ import annotations

import os

import torch

ENABLED = os.environ.get("PULSARLM_B200_BRANCHES", "1") != "0"  # (0: always one after the other, for comparison)

_STREAMS: dict[tuple, torch.cuda.Stream] = {}


def _stream(device: torch.device, name: str) -> torch.cuda.Stream:
    """One stream per device and name: the allocator keeps freed blocks per stream."""
    key = (device, name)
    if key not in _STREAMS:
        _STREAMS[key] = torch.cuda.Stream(device)
    return _STREAMS[key]


def run_branches(batch, device: torch.device, first, **others):
    """The results of `first()` and of every other call, in order. In a captured step each other call runs on the
    stream named like its keyword; names must differ from those of a `run_branches` that may be open around this one.
    What the calls read must stay referenced by the caller until they return (memory is handed out again in stream
    order, and everything is joined to the current stream before that)."""
    if not ENABLED or batch is None or not batch.extras.get("graph"):
        return (first(), *(call() for call in others.values()))
    main = torch.cuda.current_stream(device)
    fork = torch.cuda.Event()
    fork.record(main)
    results, joins = [], []
    for name, call in others.items():
        side = _stream(device, name)
        side.wait_event(fork)
        with torch.cuda.stream(side):
            results.append(call())
        joins.append(torch.cuda.Event())
        joins[-1].record(side)
    mine = first()
    for join in joins:
        main.wait_event(join)
    return (mine, *results)
