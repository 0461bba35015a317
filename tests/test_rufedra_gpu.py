import json,glob
for f in glob.glob('/root/.claude/projects/-root-repo/*.jsonl'):
    n=0
    for l in open(f):
        if 'test_rufedra_gpu.py <<' in l:
            n+=1
            d=json.loads(l)
            for c in d['message']['content']:
                if c.get('type')=='tool_use' and 'cat > tests/test_rufedra_gpu.py' in c['input'].get('command',''):
                    s=c['input']['command']
                    body=s.split("<<'E'\n",1)[1].split("\nE\n",1)[0]+"\n"
                    open('tests/test_rufedra_gpu.py','w').write(body); print(f,len(body.splitlines()))
    print(f,n)
